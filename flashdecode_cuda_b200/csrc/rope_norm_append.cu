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
    void* q_out; void* k_pool; void* v_pool; void* v_first;     // v_first [T, n_kv v_true] or null: only the true dimensions of padded heads
    const float* q_w; const float* k_w;
    float eps;
    const float* cos_t; const float* sin_t; int table_len, rot;
    int head_norm;                       // 1: divide every head of q and k by its root mean square after the rotation
    int v_mode; const float* lam;        // 0: values as they are; 1: also to v_first; 2: mixed with v_first by *lam
    const int* tok_row; const int* tok_pos; const int* row_slot; const int* block_table;
    int max_blocks, num_blocks, block_size, n_q, n_kv, d, dv, q_count, k_count, head_count, write_kv, v_true;
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
        if (p.v_mode != 0 && j < p.v_true) {
            T* f = vf + ((size_t)t * p.n_kv + h) * p.v_true + j;
            if (p.v_mode == 1) *f = v;
            else v = from_float<T>((1.f - lam) * to_float(v) + lam * to_float(*f));
        }
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

// four neighbouring elements as floats, and back
__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 ld4(const __nv_bfloat16* p) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.y));
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void st4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void st4(__nv_bfloat16* p, float4 v) {
    uint2 o;
    *reinterpret_cast<__nv_bfloat162*>(&o.x) = __floats2bfloat162_rn(v.x, v.y);
    *reinterpret_cast<__nv_bfloat162*>(&o.y) = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = o;
}

// The same four elements at a time, for heads of up to 128 dimensions: head sizes and row lengths multiples of 4, the rotation's
// half too, everything aligned.  A head takes the power of two of lanes that covers d / 4, so a warp takes several small heads.
template <typename T>
__global__ void __launch_bounds__(256)
rope_norm_append_vec_kernel(const RopeNorm p) {
    extern __shared__ __align__(16) float s_row[];           // q and k of the token, before the norm
    __shared__ float red[33];
    const int t = blockIdx.x;
    const int slot = p.row_slot[p.tok_row[t]];
    if (slot < 0) return;
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
#pragma unroll 4
    for (int i = threadIdx.x * 4; i < nq + nk; i += blockDim.x * 4) {
        const float4 v = ld4(row + i);
        *reinterpret_cast<float4*>(s_row + i) = v;
        const float s = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, v.w * v.w)));
        if (i < nq) sq += s; else sk += s;
    }
    T* vf = static_cast<T*>(p.v_first);
    const float lam = p.v_mode == 2 ? *p.lam : 0.f;
    const int in_blk = pos - bcol * p.block_size;
    for (int i = threadIdx.x * 4; i < nv; i += blockDim.x * 4) {
        const int h = i / p.dv, j = i - h * p.dv;
        float4 v = ld4(row + nq + nk + i);
        T* at = vf + ((size_t)t * p.n_kv + h) * p.v_true + j;
        if (p.v_mode == 1 && j < p.v_true) st4(at, v);
        else if (p.v_mode == 2 && j < p.v_true) {
            const float4 f = ld4(at);
            v = make_float4((1.f - lam) * v.x + lam * f.x, (1.f - lam) * v.y + lam * f.y, (1.f - lam) * v.z + lam * f.z,
                            (1.f - lam) * v.w + lam * f.w);
        }
        if (stored) st4(static_cast<T*>(p.v_pool) + (((size_t)blk * p.n_kv + h) * p.block_size + in_blk) * p.dv + j, v);
    }
    float rq = 1.f, rk = 1.f;
    if (p.q_w != nullptr) {
        rq = 1.f / sqrtf(block_sum(sq, red) / (float)p.q_count + p.eps);
        rk = 1.f / sqrtf(block_sum(sk, red) / (float)p.k_count + p.eps);
    } else {
        __syncthreads();
    }
    int lanes = 1;                                           // lanes of a head
    while (lanes * 4 < p.d) lanes <<= 1;
    const int half = p.rot >> 1;
    const int j = (threadIdx.x & (lanes - 1)) * 4;
    for (int h0 = 0; h0 < p.n_q + p.n_kv; h0 += blockDim.x / lanes) {
        const int h = h0 + threadIdx.x / lanes;
        const bool mine = j < p.d && h < p.n_q + p.n_kv;
        const bool is_q = h < p.n_q;
        const int first = h * p.d;
        const float r = is_q ? rq : rk;
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        if (mine) {
            const float* w = p.q_w == nullptr ? nullptr : (is_q ? p.q_w + first : p.k_w + (first - nq));
            auto value = [&](int at) {
                const float4 x = *reinterpret_cast<const float4*>(s_row + first + at);
                if (w == nullptr) return x;
                const float4 g = *reinterpret_cast<const float4*>(w + at);
                return make_float4(x.x * r * g.x, x.y * r * g.y, x.z * r * g.z, x.w * r * g.w);
            };
            v = value(j);
            if (turned && j < p.rot) {
                const bool low = j < half;
                const float4 o = value(low ? j + half : j - half);
                const float4 c = *reinterpret_cast<const float4*>(p.cos_t + (size_t)pos * half + (low ? j : j - half));
                float4 s = *reinterpret_cast<const float4*>(p.sin_t + (size_t)pos * half + (low ? j : j - half));
                if (low) s = make_float4(-s.x, -s.y, -s.z, -s.w);
                v = make_float4(v.x * c.x + o.x * s.x, v.y * c.y + o.y * s.y, v.z * c.z + o.z * s.z, v.w * c.w + o.w * s.w);
            }
        }
        if (p.head_norm) {
            float ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, v.w * v.w)));
            for (int off = 1; off < lanes; off <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
            const float inv = 1.f / sqrtf(ss / (float)p.head_count + p.eps);
            v = make_float4(v.x * inv, v.y * inv, v.z * inv, v.w * inv);
        }
        if (!mine) continue;
        if (is_q) st4(static_cast<T*>(p.q_out) + (size_t)t * nq + first + j, v);
        else if (stored)
            st4(static_cast<T*>(p.k_pool) + (((size_t)blk * p.n_kv + (h - p.n_q)) * p.block_size + in_blk) * p.d + j, v);
    }
}

}  // namespace fd

using namespace fd;
typedef __nv_bfloat16 bf16;

// dtype (0 float32, 1 bfloat16): proj, q_out, v_first and the pools alike.  q_w [n_q d] and k_w [n_kv d]: both or neither.
// cos_t / sin_t [table_len, rot / 2] (unused when rot == 0).  v_true: true size of a (padded) value head.  lam: one float on the device (v_mode 2).
extern "C" int fd_rope_norm_append(const void* proj, int ld, int dtype, void* q_out, void* k_pool, void* v_pool, void* v_first,
                                   const float* q_w, const float* k_w, float eps, const float* cos_t, const float* sin_t,
                                   int table_len, int rot, int head_norm, int v_mode, const float* lam, const int* tok_row,
                                   const int* tok_pos, const int* row_slot, const int* block_table, int max_blocks, int num_blocks,
                                   int block_size, int T, int n_q, int n_kv, int d, int dv, int q_count, int k_count, int head_count,
                                   int v_true, int write_kv, int* status, cudaStream_t stream) {
    if (T == 0) return 0;
    FD_REQUIRE(n_q > 0 && n_kv > 0 && d > 0 && dv > 0 && block_size > 0 && ld >= (n_q + n_kv) * d + n_kv * dv, -2,
               "rope_norm_append: %d + %d heads of %d and %d in rows of %d", n_q, n_kv, d, dv, ld);
    FD_REQUIRE(rot >= 0 && rot % 2 == 0 && rot <= d && (rot == 0 || (cos_t && sin_t)), -2, "rope_norm_append: %d rotated dimensions of %d", rot, d);
    FD_REQUIRE((q_w == nullptr) == (k_w == nullptr) && q_count > 0 && k_count > 0 && head_count > 0, -2, "rope_norm_append: bad norms");
    FD_REQUIRE(v_mode >= 0 && v_mode <= 2 && (v_mode == 0 || v_first) && (v_mode != 2 || lam) && v_true >= 1 && v_true <= dv, -2,
               "rope_norm_append: value mixing %d, %d of %d value dimensions", v_mode, v_true, dv);
    RopeNorm p = {proj, ld, q_out, k_pool, v_pool, v_first, q_w, k_w, eps, cos_t, sin_t, table_len, rot, head_norm, v_mode, lam, tok_row,
                  tok_pos, row_slot, block_table, max_blocks, num_blocks, block_size, n_q, n_kv, d, dv, q_count, k_count, head_count,
                  write_kv, v_true, status};
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
    auto al = [](const void* x) { return (uintptr_t)x % 16 == 0; };
    if (d % 4 == 0 && d <= 128 && dv % 4 == 0 && ld % 4 == 0 && rot % 8 == 0 && v_true % 4 == 0 && smem <= 48 * 1024 && (uintptr_t)proj % 8 == 0 && al(q_out) &&
        al(k_pool) && al(v_pool) && al(v_first) && al(q_w) && al(k_w) && al(cos_t) && al(sin_t) && (dtype != 0 || al(proj))) {
        if (dtype == 0) return launch("rope_norm_append", rope_norm_append_vec_kernel<float>, dim3(T), block, smem, stream, dim3(1, 1, 1), p);
        return launch("rope_norm_append", rope_norm_append_vec_kernel<bf16>, dim3(T), block, smem, stream, dim3(1, 1, 1), p);
    }
    if (dtype == 0) return launch("rope_norm_append", rope_norm_append_kernel<float>, dim3(T), block, smem, stream, dim3(1, 1, 1), p);
    return launch("rope_norm_append", rope_norm_append_kernel<bf16>, dim3(T), block, smem, stream, dim3(1, 1, 1), p);
}
