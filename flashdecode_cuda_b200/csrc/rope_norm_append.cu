// What stands between an attention mixer's packed projection and its attention kernel when q and k are both normed and
// rotated (dimension i paired with i + rot / 2):
//
//   * by option q and k are RMS-normed over their WHOLE projections (weights q_w, k_w) before the rotation;
//   * the first `rot` dimensions of every head are turned at the token's position;
//   * by option every head of q and k is then divided by its own root mean square (no weight);
//   * by option the values are mixed with the same token's values of another layer, v <- (1 - lam) v + lam v_first, or
//     left in v_first for later layers;
//   * q goes to its buffer, k and v to the paged cache.
//
// proj [T, ld] from its first column on: q (n_q * d), k (n_kv * d), v (n_kv * dv).  d and dv may be padded with zero columns;
// q_count, k_count and head_count say over how many values the means run.  A CTA per token: the row's q and k wait in shared
// memory as floats, a warp takes a head at a time.  Sums, norms, angles' use and the mixing are float, rounded once.
#include "common.cuh"

namespace fd {

struct RopeNorm {
    const void* proj; int ld;
    void* q_out; void* k_pool; void* v_pool; void* v_first;     // v_first [T, n_kv dv] or null
    const float* q_w; const float* k_w;
    float eps;
    const float* cos_t; const float* sin_t; int table_len, rot;
    int head_norm;                       // 1: divide every head of q and k by its root mean square after the rotation
    int v_mode; const float* lam;        // 0: values as they are; 1: also to v_first; 2: mixed with v_first by *lam
    const int* tok_row; const int* tok_pos; const int* row_slot; const int* block_table;
    int max_blocks, num_blocks, block_size, n_q, n_kv, d, dv, q_count, k_count, head_count, write_kv;
    int* status;
};

template <typename T>
__global__ void __launch_bounds__(256)
rope_norm_append_kernel(const RopeNorm p) {
    extern __shared__ __align__(16) float s_row[];           // q and k of the token
    __shared__ float red[33];
    const int t = blockIdx.x;
    const int slot = p.row_slot[p.tok_row[t]];
    if (slot < 0) return;                                    // padding row of a fixed-size batch
    const T* row = static_cast<const T*>(p.proj) + (size_t)t * p.ld;
    const int nq = p.n_q * p.d, nk = p.n_kv * p.d, nv = p.n_kv * p.dv;
    const int pos = p.tok_pos[t];
    const int bcol = pos / p.block_size;
    const int blk = p.write_kv && pos >= 0 && bcol < p.max_blocks ? p.block_table[(size_t)slot * p.max_blocks + bcol] : -1;
    const bool stored = p.write_kv && blk >= 0 && blk < p.num_blocks;
    if (threadIdx.x == 0) {
        if (p.write_kv && !stored) set_status(p.status, STATUS_BAD_BLOCK);
        if (p.rot > 0 && (pos < 0 || pos >= p.table_len)) set_status(p.status, STATUS_BAD_POSITION);
    }
    const bool turned = p.rot > 0 && pos >= 0 && pos < p.table_len;
    float sq = 0.f, sk = 0.f;
    for (int i = threadIdx.x; i < nq + nk; i += blockDim.x) {
        const float v = to_float(row[i]);
        s_row[i] = v;
        if (i < nq) sq = fmaf(v, v, sq); else sk = fmaf(v, v, sk);
    }
    float rq = 1.f, rk = 1.f;
    if (p.q_w != nullptr) {
        rq = 1.f / sqrtf(block_sum(sq, red) / (float)p.q_count + p.eps);
        rk = 1.f / sqrtf(block_sum(sk, red) / (float)p.k_count + p.eps);
    } else {
        __syncthreads();
    }
    // values: to the pool, mixed with or left for the other layers
    T* vf = static_cast<T*>(p.v_first);
    const float lam = p.v_mode == 2 ? *p.lam : 0.f;
    for (int i = threadIdx.x; i < nv; i += blockDim.x) {
        const int h = i / p.dv, j = i - h * p.dv;
        T v = row[nq + nk + i];
        if (p.v_mode == 1) vf[(size_t)t * nv + i] = v;
        else if (p.v_mode == 2) v = from_float<T>((1.f - lam) * to_float(v) + lam * to_float(vf[(size_t)t * nv + i]));
        if (stored) static_cast<T*>(p.v_pool)[(((size_t)blk * p.n_kv + h) * p.block_size + (pos - bcol * p.block_size)) * p.dv + j] = v;
    }
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
    const int half = p.rot >> 1;
    const float* cs = turned ? p.cos_t + (size_t)pos * half : nullptr;
    const float* sn = turned ? p.sin_t + (size_t)pos * half : nullptr;
    for (int h = warp; h < p.n_q + p.n_kv; h += n_warps) {
        const bool is_q = h < p.n_q;
        const int first = h * p.d;                           // k's heads follow q's in the row
        const float r = is_q ? rq : rk;
        const float* w = p.q_w == nullptr ? nullptr : (is_q ? p.q_w + first : p.k_w + (first - nq));
        float* x = s_row + first;
        auto value = [&](int j) { return x[j] * r * (w != nullptr ? w[j] : 1.f); };
        auto rotated = [&](int j) -> float {
            if (!turned || j >= p.rot) return value(j);
            return j < half ? value(j) * cs[j] - value(j + half) * sn[j] : value(j) * cs[j - half] + value(j - half) * sn[j - half];
        };
        float inv = 1.f;
        if (p.head_norm) {
            float ss = 0.f;
            for (int j = lane; j < p.d; j += 32) { const float v = rotated(j); ss = fmaf(v, v, ss); }
            inv = 1.f / sqrtf(warp_sum(ss) / (float)p.head_count + p.eps);
        }
        T* dst = nullptr;
        if (is_q) dst = static_cast<T*>(p.q_out) + (size_t)t * nq + first;
        else if (stored)
            dst = static_cast<T*>(p.k_pool) + (((size_t)blk * p.n_kv + (h - p.n_q)) * p.block_size + (pos - bcol * p.block_size)) * p.d;
        if (dst == nullptr) continue;
        for (int j = lane; j < p.d; j += 32) dst[j] = from_float<T>(rotated(j) * inv);
    }
}

}  // namespace fd

using namespace fd;
typedef __nv_bfloat16 bf16;

// dtype (0 float32, 1 bfloat16): proj, q_out, v_first and the pools alike.  q_w [n_q d] and k_w [n_kv d]: both or neither.
// cos_t / sin_t [table_len, rot / 2] (unused when rot == 0).  lam: one float on the device (v_mode 2).
extern "C" int fd_rope_norm_append(const void* proj, int ld, int dtype, void* q_out, void* k_pool, void* v_pool, void* v_first,
                                   const float* q_w, const float* k_w, float eps, const float* cos_t, const float* sin_t,
                                   int table_len, int rot, int head_norm, int v_mode, const float* lam, const int* tok_row,
                                   const int* tok_pos, const int* row_slot, const int* block_table, int max_blocks, int num_blocks,
                                   int block_size, int T, int n_q, int n_kv, int d, int dv, int q_count, int k_count, int head_count,
                                   int write_kv, int* status, cudaStream_t stream) {
    if (T == 0) return 0;
    FD_REQUIRE(n_q > 0 && n_kv > 0 && d > 0 && dv > 0 && block_size > 0 && ld >= (n_q + n_kv) * d + n_kv * dv, -2,
               "rope_norm_append: %d + %d heads of %d and %d in rows of %d", n_q, n_kv, d, dv, ld);
    FD_REQUIRE(rot >= 0 && rot % 2 == 0 && rot <= d && (rot == 0 || (cos_t && sin_t)), -2, "rope_norm_append: %d rotated dimensions of %d", rot, d);
    FD_REQUIRE((q_w == nullptr) == (k_w == nullptr) && q_count > 0 && k_count > 0 && head_count > 0, -2, "rope_norm_append: bad norms");
    FD_REQUIRE(v_mode >= 0 && v_mode <= 2 && (v_mode == 0 || v_first) && (v_mode != 2 || lam), -2, "rope_norm_append: value mixing %d", v_mode);
    RopeNorm p = {proj, ld, q_out, k_pool, v_pool, v_first, q_w, k_w, eps, cos_t, sin_t, table_len, rot, head_norm, v_mode, lam, tok_row,
                  tok_pos, row_slot, block_table, max_blocks, num_blocks, block_size, n_q, n_kv, d, dv, q_count, k_count, head_count,
                  write_kv, status};
    const size_t smem = (size_t)(n_q + n_kv) * d * sizeof(float);
    FD_REQUIRE(smem <= 200 * 1024, -2, "rope_norm_append: q and k of %d values do not fit shared memory", (n_q + n_kv) * d);
    static size_t configured[2] = {48 * 1024, 48 * 1024};
    const int which = dtype == 0 ? 0 : 1;
    if (smem > configured[which]) {
        cudaError_t e = which == 0 ? cudaFuncSetAttribute(rope_norm_append_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)
                                   : cudaFuncSetAttribute(rope_norm_append_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return fail(-3, "rope_norm_append: cannot get %zu bytes of shared memory: %s", smem, cudaGetErrorString(e));
        configured[which] = smem;
    }
    const dim3 block((n_q + n_kv) * d >= 1024 ? 256 : 128);
    if (dtype == 0) return launch("rope_norm_append", rope_norm_append_kernel<float>, dim3(T), block, smem, stream, dim3(1, 1, 1), p);
    return launch("rope_norm_append", rope_norm_append_kernel<bf16>, dim3(T), block, smem, stream, dim3(1, 1, 1), p);
}
