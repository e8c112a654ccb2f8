// Attention of many query heads over ONE cached row per position (bfloat16): the row [dk] is the key of every head and
// its first r dimensions are the value of every head - a latent-attention mixer whose queries have been taken into the
// latent's basis.  Decode steps and later portions of prompts; a CTA takes 16 or 32 heads of one token and a range of its
// keys.
//
//   S[heads, 64 keys] = Q K^T      mma.m16n8k16, the heads as rows: warp w takes keys 8 w .. 8 w + 7 of the tile against the
//                                  whole row; with 16 heads the queries' fragments stay in registers for good
//   softmax                        running maximum and sum per head in float (base 2); the warps' maxima meet in shared
//                                  memory, P goes there as two bfloat16 numbers (the rounded weight and what the
//                                  rounding took away: 16 bits of mantissa)
//   O[heads, r] += P C             warp w takes the 16-column groups w, w + 8, ... of the same tile's rows (read transposed)
//
// A tile of 64 rows is fetched once by cp.async (rows found through the block table, 8 per warp) and serves both products;
// two to four tiles are in shared memory.  The keys of a token may be cut into splits at absolute multiples of split_len:
// a split leaves (maximum, sum, accumulators) in scratch memory and the merge kernel of attention_simt.cu adds them up.
// A keyless term exp(sink[h]) may join a head's denominator.
#include <math.h>

#include "attention.cuh"
#include "mma_utils.cuh"

namespace fd {

constexpr int AL_KEYS = 64;                  // keys of a tile
constexpr int AL_WARPS = 8;
constexpr int AL_THREADS = AL_WARPS * 32;
constexpr int AL_PST = 2 * AL_KEYS + 8;      // elements of a row of P: the weights, then their rests
constexpr int AL_GROUPS = 4;                 // 16-column groups of O per warp (r up to 512)
constexpr int AL_MAX_R = AL_WARPS * AL_GROUPS * 16;
constexpr int AL_MAX_DK = 640;
constexpr int AL_SMEM = 200 * 1024;          // what the tiles in flight may fill up to

__device__ __forceinline__ float al_ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ void al_ldmatrix_x2(uint32_t addr, uint32_t& r0, uint32_t& r1) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];\n" : "=r"(r0), "=r"(r1) : "r"(addr));
}

// elements of a row in shared memory: the row up to a multiple of 16, and 8 more so that eight rows' 16-byte pieces lie in
// different banks
__host__ __device__ __forceinline__ int al_stride(int dk) { return (dk + 15) / 16 * 16 + 8; }

// MT: groups of 16 heads of the CTA.  KS > 0 (MT 1): k-steps of 16 whose query fragments are held in registers (at least
// as many as the row has); KS 0: they are read from shared memory every time.
template <int MT, int KS>
__global__ void __launch_bounds__(AL_THREADS, 1)
attn_latent_kernel(const AttnParams p, const int* __restrict__ tok_row, const int stages) {
    const int t = blockIdx.z, split = blockIdx.x, h0 = blockIdx.y * MT * 16;
    const int b = tok_row[t];
    const int slot = p.row_slot[b];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int r = p.dv, dk = p.d;
    const int nh = min(MT * 16, p.n_q - h0);                 // heads of this CTA
    __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out) + ((size_t)t * p.n_q + h0) * r;
    if (slot < 0) {                                          // padding row: zeros (the merge kernel writes them otherwise)
        if (p.n_splits == 1)
            for (int e = tid; e < nh * r; e += AL_THREADS) out[e] = __float2bfloat16_rn(0.f);
        return;
    }
    const int pos = p.row_ctx_len[b] + (t - p.row_q_start[b]);
    int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
    int hi = pos + 1;
    if (p.n_splits > 1) {
        lo = max(lo, split * p.split_len);
        hi = min(hi, (split + 1) * p.split_len);
        if (lo >= hi) {                                      // no key of this token in the range
            for (int h = tid; h < nh; h += AL_THREADS) {
                const size_t pi = ((size_t)t * p.n_q + h0 + h) * p.n_splits + split;
                p.part_m[pi] = -INFINITY;
                p.part_l[pi] = 0.f;
            }
            return;
        }
    }
    const int st = al_stride(dk);
    const int nks = (dk + 15) >> 4;
    extern __shared__ __align__(16) unsigned char al_raw[];
    __nv_bfloat16* q_s = reinterpret_cast<__nv_bfloat16*>(al_raw);          // [MT * 16][st]
    __nv_bfloat16* p_s = q_s + MT * 16 * st;                                // [MT * 16][AL_PST]
    float* m_s = reinterpret_cast<float*>(p_s + MT * 16 * AL_PST);          // [warps][MT * 16]
    float* l_s = m_s + AL_WARPS * MT * 16;                                  // [warps][MT * 16]
    __nv_bfloat16* k_s = reinterpret_cast<__nv_bfloat16*>(l_s + AL_WARPS * MT * 16);     // [stages][AL_KEYS][st]
    const int stage_el = AL_KEYS * st;

    // ---- rows of a tile: warp w fetches keys 8 w .. 8 w + 7; their places are looked up a tile ahead of their use ----
    const __nv_bfloat16* pool = static_cast<const __nv_bfloat16*>(p.k_pool);
    const int t_begin = lo / AL_KEYS * AL_KEYS;
    const int n_tiles = (hi - t_begin + AL_KEYS - 1) / AL_KEYS;
    const int bs = p.block_size, cpr = dk >> 3;
    auto place = [&](int it) -> int {                        // lanes 0..7: the row in the pool of one of the warp's keys, or -1
        const int key = t_begin + it * AL_KEYS + warp * 8 + (lane & 7);
        if (lane >= 8 || it >= n_tiles || key < lo || key >= hi) return -1;
        const int col = key / bs;
        const int blk = col < p.max_blocks ? p.block_table[(size_t)slot * p.max_blocks + col] : -1;
        if (blk < 0 || blk >= p.num_blocks) { set_status(p.status, STATUS_BAD_BLOCK); return -1; }
        return blk * bs + (key - col * bs);
    };
    int row_next = place(0);
    auto issue = [&](int it) {
        const int row = row_next;
        row_next = place(it + 1);
        if (it < n_tiles) {
            __nv_bfloat16* dst = k_s + (it % stages) * stage_el + warp * 8 * st;
#pragma unroll
            for (int k = 0; k < 8; ++k) {
                const int rw = __shfl_sync(0xffffffffu, row, k);
                const __nv_bfloat16* src = pool + (size_t)max(rw, 0) * dk;
                for (int c = lane; c < cpr; c += 32) cp_async16(smem_u32(dst + k * st + c * 8), src + c * 8, rw >= 0 ? 16 : 0);
            }
        }
        cp_async_commit();
    };
    for (int s = 0; s < stages - 1; ++s) issue(s);

    // ---- queries, and zeros where a row is filled up to a multiple of 16 ----
    {
        const __nv_bfloat16* qg = static_cast<const __nv_bfloat16*>(p.q) + ((size_t)t * p.n_q + h0) * dk;
        const uint4 zero = make_uint4(0, 0, 0, 0);
        const int cps = st >> 3;
        for (int e = tid; e < MT * 16 * cps; e += AL_THREADS) {
            const int h = e / cps, c = e - h * cps;
            *reinterpret_cast<uint4*>(q_s + h * st + c * 8) =
                h < nh && c < cpr ? *reinterpret_cast<const uint4*>(qg + (size_t)h * dk + c * 8) : zero;
        }
        const int fill = cps - cpr;                          // 1 or 2 pieces behind every key row
        for (int e = tid; e < stages * AL_KEYS * fill; e += AL_THREADS) {
            const int k = e / fill;
            *reinterpret_cast<uint4*>(k_s + (size_t)k * st + (cpr + e - k * fill) * 8) = zero;
        }
    }
    __syncthreads();
    uint32_t qf[KS > 0 ? KS : 1][4];
    const uint32_t q_addr = smem_u32(q_s + (lane & 15) * st + (lane >> 4) * 8);
    if (KS > 0) {
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) {
            qf[ks][0] = qf[ks][1] = qf[ks][2] = qf[ks][3] = 0;
            if (ks < nks) ldmatrix_x4(q_addr + ks * 32, qf[ks][0], qf[ks][1], qf[ks][2], qf[ks][3]);
        }
    }

    const float scale_log2 = p.scale * 1.4426950408889634f;
    float m_run[MT][2], l_run[MT][2];
    float acc[MT][AL_GROUPS][2][4];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
        m_run[mt][0] = m_run[mt][1] = -INFINITY;
        l_run[mt][0] = l_run[mt][1] = 0.f;
#pragma unroll
        for (int g = 0; g < AL_GROUPS; ++g)
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int e = 0; e < 4; ++e) acc[mt][g][j][e] = 0.f;
    }
    const int gr = lane >> 2, tg = lane & 3;                 // this thread's rows gr, gr + 8 and columns 2 tg, 2 tg + 1

    for (int it = 0; it < n_tiles; ++it) {
        // the tiles after this one that may still be under way: stages - 2
        if (stages == 2) cp_async_wait<0>();
        else if (stages == 3) cp_async_wait<1>();
        else cp_async_wait<2>();
        __syncthreads();                                     // the tile is in; everyone is done with the one before
        issue(it + stages - 1);
        const __nv_bfloat16* ks_ = k_s + (it % stages) * stage_el;
        // scores of 8 keys
        float s[MT][4];
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) s[mt][0] = s[mt][1] = s[mt][2] = s[mt][3] = 0.f;
        const uint32_t k_addr = smem_u32(ks_ + (warp * 8 + (lane & 7)) * st + (lane >> 3) * 8);
        if (KS > 0) {
            float s2[4] = {0.f, 0.f, 0.f, 0.f};              // two chains of products
#pragma unroll
            for (int kp = 0; kp < KS / 2; ++kp) {
                if (2 * kp + 1 < nks) {
                    uint32_t b0, b1, b2, b3;
                    ldmatrix_x4(k_addr + kp * 64, b0, b1, b2, b3);
                    mma_bf16(s[0], qf[2 * kp][0], qf[2 * kp][1], qf[2 * kp][2], qf[2 * kp][3], b0, b1);
                    mma_bf16(s2, qf[2 * kp + 1][0], qf[2 * kp + 1][1], qf[2 * kp + 1][2], qf[2 * kp + 1][3], b2, b3);
                } else if (2 * kp < nks) {
                    uint32_t b0, b1;
                    al_ldmatrix_x2(smem_u32(ks_ + (warp * 8 + (lane & 7)) * st + ((lane >> 3) & 1) * 8) + kp * 64, b0, b1);
                    mma_bf16(s[0], qf[2 * kp][0], qf[2 * kp][1], qf[2 * kp][2], qf[2 * kp][3], b0, b1);
                }
            }
#pragma unroll
            for (int e = 0; e < 4; ++e) s[0][e] += s2[e];
        } else {
            const uint32_t k2 = smem_u32(ks_ + (warp * 8 + (lane & 7)) * st + ((lane >> 3) & 1) * 8);
#pragma unroll 4
            for (int ks = 0; ks < nks; ++ks) {
                uint32_t b0, b1;
                al_ldmatrix_x2(k2 + ks * 32, b0, b1);
#pragma unroll
                for (int mt = 0; mt < MT; ++mt) {
                    uint32_t a0, a1, a2, a3;
                    ldmatrix_x4(q_addr + (mt * 16 * st) * 2 + ks * 32, a0, a1, a2, a3);
                    mma_bf16(s[mt], a0, a1, a2, a3, b0, b1);
                }
            }
        }
        // mask, and this warp's maxima
        const int key = t_begin + it * AL_KEYS + warp * 8 + 2 * tg;
        const bool v0 = key >= lo && key < hi, v1 = key + 1 >= lo && key + 1 < hi;
#pragma unroll
        for (int mt = 0; mt < MT; ++mt)
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                float& a = s[mt][2 * half];
                float& c = s[mt][2 * half + 1];
                a = v0 ? a * scale_log2 : -INFINITY;
                c = v1 ? c * scale_log2 : -INFINITY;
                float m = fmaxf(a, c);
                m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, 1));
                m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, 2));
                if (tg == 0) m_s[warp * (MT * 16) + mt * 16 + half * 8 + gr] = m;
            }
        __syncthreads();
        float alpha[MT][2];
        bool moved = false;
#pragma unroll
        for (int mt = 0; mt < MT; ++mt)
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int row = mt * 16 + half * 8 + gr;
                float m = m_run[mt][half];
#pragma unroll
                for (int w = 0; w < AL_WARPS; ++w) m = fmaxf(m, m_s[w * (MT * 16) + row]);
                // (every tile has a visible key, so m is finite)
                const float al = al_ex2(m_run[mt][half] - m);
                alpha[mt][half] = al;
                moved |= al != 1.f;
                m_run[mt][half] = m;
                const float p0 = al_ex2(s[mt][2 * half] - m), p1 = al_ex2(s[mt][2 * half + 1] - m);
                l_run[mt][half] = l_run[mt][half] * al + (p0 + p1);
                *reinterpret_cast<uint32_t*>(p_s + row * AL_PST + warp * 8 + 2 * tg) = pack_bf16(p0, p1);
                *reinterpret_cast<uint32_t*>(p_s + row * AL_PST + AL_KEYS + warp * 8 + 2 * tg) = pack_bf16_rest(p0, p1);
            }
        __syncthreads();
        if (__any_sync(0xffffffffu, moved)) {
#pragma unroll
            for (int mt = 0; mt < MT; ++mt)
#pragma unroll
                for (int g = 0; g < AL_GROUPS; ++g)
#pragma unroll
                    for (int j = 0; j < 2; ++j) {
                        acc[mt][g][j][0] *= alpha[mt][0]; acc[mt][g][j][1] *= alpha[mt][0];
                        acc[mt][g][j][2] *= alpha[mt][1]; acc[mt][g][j][3] *= alpha[mt][1];
                    }
        }
#pragma unroll
        for (int kk = 0; kk < AL_KEYS / 16; ++kk) {
            uint32_t a[MT][4], rest[MT][4];
#pragma unroll
            for (int mt = 0; mt < MT; ++mt) {
                const uint32_t at = smem_u32(p_s + (mt * 16 + (lane & 15)) * AL_PST + kk * 16 + (lane >> 4) * 8);
                ldmatrix_x4(at, a[mt][0], a[mt][1], a[mt][2], a[mt][3]);
                ldmatrix_x4(at + AL_KEYS * 2, rest[mt][0], rest[mt][1], rest[mt][2], rest[mt][3]);
            }
#pragma unroll
            for (int g = 0; g < AL_GROUPS; ++g) {
                const int c0 = (warp + g * AL_WARPS) * 16;
                if (c0 >= r) continue;
                uint32_t b0, b1, b2, b3;
                ldmatrix_x4_trans(smem_u32(ks_ + (kk * 16 + (lane & 15)) * st + c0 + (lane >> 4) * 8), b0, b1, b2, b3);
#pragma unroll
                for (int mt = 0; mt < MT; ++mt) {
                    mma_bf16(acc[mt][g][0], a[mt][0], a[mt][1], a[mt][2], a[mt][3], b0, b1);
                    mma_bf16(acc[mt][g][1], a[mt][0], a[mt][1], a[mt][2], a[mt][3], b2, b3);
                    mma_bf16(acc[mt][g][0], rest[mt][0], rest[mt][1], rest[mt][2], rest[mt][3], b0, b1);
                    mma_bf16(acc[mt][g][1], rest[mt][0], rest[mt][1], rest[mt][2], rest[mt][3], b2, b3);
                }
            }
        }
    }
    cp_async_wait<0>();
    // the warps' sums
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            float l = l_run[mt][half];
            l += __shfl_xor_sync(0xffffffffu, l, 1);
            l += __shfl_xor_sync(0xffffffffu, l, 2);
            if (tg == 0) l_s[warp * (MT * 16) + mt * 16 + half * 8 + gr] = l;
        }
    __syncthreads();
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int row = mt * 16 + half * 8 + gr;
            if (row >= nh) continue;
            float l = 0.f;
#pragma unroll
            for (int w = 0; w < AL_WARPS; ++w) l += l_s[w * (MT * 16) + row];
            const float m = m_run[mt][half];
            if (p.n_splits > 1) {
                const size_t pi = ((size_t)t * p.n_q + h0 + row) * p.n_splits + split;
                if (warp == 0 && tg == 0) { p.part_m[pi] = m * 0.6931471805599453f; p.part_l[pi] = l; }
                float* pa = p.part_acc + pi * r;
#pragma unroll
                for (int g = 0; g < AL_GROUPS; ++g)
#pragma unroll
                    for (int j = 0; j < 2; ++j) {
                        const int c = (warp + g * AL_WARPS) * 16 + j * 8 + 2 * tg;
                        if (c < r) *reinterpret_cast<float2*>(pa + c) = make_float2(acc[mt][g][j][2 * half], acc[mt][g][j][2 * half + 1]);
                    }
            } else {
                float f = 1.f;
                if (p.sink != nullptr) {
                    const float sk = p.sink[h0 + row] * 1.4426950408889634f;
                    const float m2 = fmaxf(m, sk);
                    f = al_ex2(m - m2);
                    l = l * f + al_ex2(sk - m2);
                }
                const float inv = f / l;
#pragma unroll
                for (int g = 0; g < AL_GROUPS; ++g)
#pragma unroll
                    for (int j = 0; j < 2; ++j) {
                        const int c = (warp + g * AL_WARPS) * 16 + j * 8 + 2 * tg;
                        if (c < r)
                            *reinterpret_cast<uint32_t*>(out + (size_t)row * r + c) =
                                pack_bf16(acc[mt][g][j][2 * half] * inv, acc[mt][g][j][2 * half + 1] * inv);
                    }
            }
        }
}

template <int MT, int KS>
static int launch_al(const AttnParams& p, const int* tok_row, int T, cudaStream_t stream) {
    const int st = al_stride(p.d);
    const size_t fixed = (size_t)MT * 16 * (st + AL_PST) * 2 + 2 * AL_WARPS * MT * 16 * sizeof(float);
    const size_t stage = (size_t)AL_KEYS * st * 2;
    int stages = 4;
    while (stages > 2 && fixed + stages * stage > AL_SMEM) --stages;
    const size_t smem = fixed + stages * stage;
    auto k = attn_latent_kernel<MT, KS>;
    static size_t configured = 0;
    if (smem > configured) {
        cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return fail(-3, "attention: cannot get %zu bytes of shared memory: %s", smem, cudaGetErrorString(e));
        configured = smem;
    }
    const dim3 grid(p.n_splits, (p.n_q + MT * 16 - 1) / (MT * 16), T);
    return launch("attention_latent", k, grid, dim3(AL_THREADS), smem, stream, dim3(1, 1, 1), p, tok_row, stages);
}

// 1: the sizes are not taken
int launch_attn_latent_mma(const AttnParams& p, const int* tok_row, int T, cudaStream_t stream) {
    if (p.d % 8 || p.dv % 8 || p.d > AL_MAX_DK || p.dv > AL_MAX_R || p.dv > p.d || T > 65535) return 1;
    if (p.n_q > 16) return launch_al<2, 0>(p, tok_row, T, stream);
    if (p.d <= 128) return launch_al<1, 8>(p, tok_row, T, stream);
    if (p.d <= 320) return launch_al<1, 20>(p, tok_row, T, stream);
    return launch_al<1, 40>(p, tok_row, T, stream);
}

}  // namespace fd
