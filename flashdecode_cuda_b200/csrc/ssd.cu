// What stands around the state-space recurrence of a Mamba-2 mixer (linear_scan.cu, mode 3):
//
//  * ssd_prepare: x, B and C - neighbouring columns of the packed projection - pass a causal convolution over time per channel
//    with bias (short_conv.cuh) and silu, and are left as floats [T, C]; per token and head the step size dt =
//    softplus(raw + bias) and the decay exp(-exp(A_h) dt), floats [T, H, 2];
//  * ssd_gate_norm: (y + D_h x) * silu(z), RMS-normed in equal parts, times a weight, times a constant.
//
// Everything is float from the projection on, and rounded once on the way to the output product.
//
// Prompts in bfloat16 take the recurrence in chunks of 128 tokens on the tensor cores (mma.m16n8k16) instead of the scan: with
// L_t the sum of the chunk's log decays up to token t and S the state before the chunk,
//     y_i = exp(L_i) C_i S + sum_(j<=i) (C_i . B_j) exp(L_i - L_j) dt_j x_j,      U = sum_j exp(L_end - L_j) dt_j B_j x_j^T,
//  * ssd_chunk_state: every chunk's U (nothing in it depends on the state) and its whole decay;
//  * ssd_chunk_chain: S <- exp(L_end) S + U from chunk to chunk in float, a thread per state element; leaves every chunk the
//    state before it, and the cache slot the last one;
//  * ssd_chunk_out: the outputs.
// B, C and x enter the products as bfloat16 (they are outputs of a convolution and its activation); dt, decays, their logarithms
// and exponentials, sums and the state are float.  Where a float factor enters a product (dt_j exp(..) x_j, the weights of the
// inner sum, the state) it goes in as two bfloat16 numbers, the rounded one and what the rounding took away, 16 bits in all.
// All exponents are of sums of decays of later tokens, at most 0: nothing is divided by a product that could vanish.
#include <math.h>

#include "mma_utils.cuh"
#include "short_conv.cuh"

namespace fd {

constexpr int SSD_THREADS = 128;

template <typename T>
__global__ void __launch_bounds__(SSD_THREADS)
ssd_prepare_kernel(const T* __restrict__ proj, int ld, int col, int C, int dt_col, const float* __restrict__ conv_w,
                   const float* __restrict__ conv_b, float* ring, int taps, int keep, const float* __restrict__ dt_bias,
                   const float* __restrict__ A_log, float* __restrict__ xbc, __nv_bfloat16* __restrict__ xbc16, int float_cols,
                   float* __restrict__ step, const int* __restrict__ tok_row,
                   const int* __restrict__ tok_pos, const int* __restrict__ row_slot, const int* __restrict__ row_q_start,
                   const int* __restrict__ row_q_len, int n_tok, int H, int tpc) {
    __shared__ ConvMeta meta;
    const int t0 = blockIdx.x * tpc, nt = min(tpc, n_tok - t0);
    conv_meta(meta, t0, nt, tok_row, tok_pos, row_slot, row_q_start, row_q_len);
    const int c = blockIdx.y * SSD_THREADS + threadIdx.x;
    float u[SC_VALS];
    if (tpc > 1 && c < C) conv_load<T>(proj + col + c, ld, t0, nt, u);
    __syncthreads();
    if (blockIdx.y == gridDim.y - 1) {                       // step sizes and decays
        for (int e = threadIdx.x; e < nt * H; e += blockDim.x) {
            const int tt = e / H, h = e - tt * H;
            const float dt = sc_softplus(to_float(proj[(size_t)(t0 + tt) * ld + dt_col + h]) + dt_bias[h]);
            *reinterpret_cast<float2*>(step + ((size_t)(t0 + tt) * H + h) * 2) = make_float2(dt, expf(-expf(A_log[h]) * dt));
        }
        return;
    }
    if (c >= C) return;
    float y[SC_TOK];
    conv_channel<T>(proj + col + c, ld, conv_w + (size_t)c * taps, conv_b[c], taps, ring, c, C, meta, t0, nt, keep, u, y);
#pragma unroll
    for (int tt = 0; tt < SC_TOK; ++tt)
        if (tt < nt && meta.slot[tt] >= 0) {
            const float v = sc_silu<T>(y[tt]);
            if (c < float_cols) xbc[(size_t)(t0 + tt) * C + c] = v;
            if (xbc16 != nullptr) xbc16[(size_t)(t0 + tt) * C + c] = __float2bfloat16_rn(v);
        }
}

// grid (parts, tokens); the gated values of a part wait in shared memory for its root mean square
template <typename T>
__global__ void __launch_bounds__(256)
ssd_gate_norm_kernel(const float* __restrict__ y, const float* __restrict__ xbc, int ldx, const float* __restrict__ D,
                     const T* __restrict__ z, int ldz, const float* __restrict__ w, T* __restrict__ out, int ld_out, int inner, int dv,
                     int part, float eps, float scale) {
    extern __shared__ float g_s[];
    __shared__ float red[33];
    const size_t t = blockIdx.y;
    const int c0 = blockIdx.x * part;
    float ss = 0.f;
#pragma unroll 4
    for (int j = threadIdx.x; j < part; j += blockDim.x) {
        const int c = c0 + j;
        const float v = fmaf(D[c / dv], xbc[t * ldx + c], y[t * inner + c]) * sc_silu<T>(to_float(z[t * ldz + c]));
        g_s[j] = v;
        ss = fmaf(v, v, ss);
    }
    const float rs = scale / sqrtf(block_sum(ss, red) / (float)part + eps);
    for (int j = threadIdx.x; j < part; j += blockDim.x) out[t * ld_out + c0 + j] = from_float<T>(g_s[j] * rs * w[c0 + j]);
}

// ---- prompts in chunks on the tensor cores ----
constexpr int SC_L = 128;                      // tokens of a chunk
constexpr int SC_DV = 64;                      // value columns of a CTA
constexpr int SCH_THREADS = 256;

struct SsdChunks {
    const __nv_bfloat16* xbc; int ld;          // [T, ld]: x (H dv columns), B (G N), C (G N)
    const float* step;                         // [T, H, 2]: dt and the decay
    const float* A_log;                        // [H]
    float* u; float* total;                    // [chunk slots, H, N, dv] and [chunk slots, H]
    float* state;                              // [slots, H, N, dv]
    float* y;                                  // [T, H dv]
    const int* row_slot; const int* row_q_start; const int* row_q_len;
    int H, G, N, dv, max_chunks, write_state, aligned;
};
__device__ __forceinline__ int chunk_slot(int q_start, int r, int c) { return q_start / SC_L + r + c; }

// L_t of the chunk's tokens (n of them; later ones repeat the last) into cs, dt into dts; the caller synchronises
__device__ __forceinline__ void chunk_decays(const SsdChunks& p, int tok0, int n, int h, float* cs, float* dts) {
    if (threadIdx.x < 32) {
        const float rate = expf(p.A_log[h]);
        const int lane = threadIdx.x;
        float v[SC_L / 32], sum = 0.f;
#pragma unroll
        for (int e = 0; e < SC_L / 32; ++e) {
            const int t = lane * (SC_L / 32) + e;
            const float dt = t < n ? p.step[((size_t)(tok0 + t) * p.H + h) * 2] : 0.f;
            dts[t] = dt;
            sum -= rate * dt;
            v[e] = sum;
        }
        float before = sum;                                  // exclusive sum over the lanes
#pragma unroll
        for (int off = 1; off < 32; off <<= 1) {
            const float o = __shfl_up_sync(0xffffffffu, before, off);
            if (lane >= off) before += o;
        }
        before -= sum;
#pragma unroll
        for (int e = 0; e < SC_L / 32; ++e) cs[lane * (SC_L / 32) + e] = before + v[e];
    }
}

// rows x COLS of bfloat16 from a matrix with rows of ld elements to a swizzled tile; rows from n on and columns from n_cols on zero
template <int COLS>
__device__ __forceinline__ void load_tile(unsigned char* dst, const __nv_bfloat16* src, int ld, int n, int n_cols, int aligned) {
    constexpr int CPR = COLS / 8;
    for (int c = threadIdx.x; c < SC_L * CPR; c += SCH_THREADS) {
        const int r = c / CPR, cc = c - r * CPR;
        if (aligned) {
            const bool in = r < n && cc * 8 < n_cols;
            cp_async16(smem_u32(dst + swz<COLS>(r, cc)), in ? src + (size_t)r * ld + cc * 8 : src, in ? 16 : 0);
        } else {
            __nv_bfloat16* at = reinterpret_cast<__nv_bfloat16*>(dst + swz<COLS>(r, cc));
#pragma unroll
            for (int e = 0; e < 8; ++e)
                at[e] = r < n && cc * 8 + e < n_cols ? src[(size_t)r * ld + cc * 8 + e] : __float2bfloat16_rn(0.f);
        }
    }
}

template <int NP>
__global__ void __launch_bounds__(SCH_THREADS)
ssd_chunk_state_kernel(const SsdChunks p) {
    constexpr int BT = SC_L * NP * 2, XT = SC_L * SC_DV * 2;
    extern __shared__ __align__(128) unsigned char sm[];
    unsigned char* b_s = sm;                   // B [128][NP]
    unsigned char* x_s = sm + BT;              // the weighted x, rounded, then the rest
    unsigned char* x_r = x_s + XT;
    __shared__ float cs[SC_L], dts[SC_L];
    const int r = blockIdx.x / p.max_chunks, c = blockIdx.x - r * p.max_chunks, h = blockIdx.y, v0 = blockIdx.z * SC_DV;
    const int q_start = p.row_q_start[r], q_len = p.row_q_len[r];
    if (p.row_slot[r] < 0 || c * SC_L >= q_len) return;
    const int tok0 = q_start + c * SC_L, n = min(SC_L, q_len - c * SC_L);
    const int inner = p.H * p.dv, g = h / (p.H / p.G), vw = min(SC_DV, p.dv - v0);
    load_tile<NP>(b_s, p.xbc + (size_t)tok0 * p.ld + inner + g * p.N, p.ld, n, p.N, p.aligned);
    cp_async_commit();
    chunk_decays(p, tok0, n, h, cs, dts);
    __syncthreads();
    const float last = cs[SC_L - 1];
    constexpr int UNR = 8;                     // loads in flight per thread
#pragma unroll 1
    for (int e0 = threadIdx.x; e0 < SC_L * SC_DV / 2; e0 += SCH_THREADS * UNR) {
        float2 x[UNR];
#pragma unroll
        for (int k = 0; k < UNR; ++k) {
            const int e = e0 + k * SCH_THREADS, t = e / (SC_DV / 2), j = (e - t * (SC_DV / 2)) * 2;
            const __nv_bfloat16* src = p.xbc + (size_t)(tok0 + t) * p.ld + h * p.dv + v0 + j;
            x[k] = make_float2(0.f, 0.f);
            if (t < n && j < vw) {
                if (p.aligned) x[k] = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(src));
                else x[k] = make_float2(__bfloat162float(src[0]), j + 1 < vw ? __bfloat162float(src[1]) : 0.f);
            }
        }
#pragma unroll
        for (int k = 0; k < UNR; ++k) {
            const int e = e0 + k * SCH_THREADS, t = e / (SC_DV / 2), j = (e - t * (SC_DV / 2)) * 2;
            const float w = expf(last - cs[t]) * dts[t];
            const int at = swz<SC_DV>(t, j >> 3) + (j & 7) * 2;
            *reinterpret_cast<uint32_t*>(x_s + at) = pack_bf16(w * x[k].x, w * x[k].y);
            *reinterpret_cast<uint32_t*>(x_r + at) = pack_bf16_rest(w * x[k].x, w * x[k].y);
        }
    }
    cp_async_wait<0>();
    __syncthreads();
    // U [NP x 64] = B^T (w x): a warp takes 16 rows and, with fewer than eight row tiles, a share of the columns
    constexpr int WT = NP / 16, SHARE = 8 / WT, NT = SC_DV / 8 / SHARE;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, mi = lane >> 3;
    const int m0 = (warp % WT) * 16, nt0 = (warp / WT) * NT;
    float acc[NT][4];
#pragma unroll
    for (int i = 0; i < NT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < SC_L / 16; ++kk) {
        uint32_t a0, a1, a2, a3;
        ldmatrix_x4_trans(smem_u32(b_s + swz<NP>(kk * 16 + (mi >> 1) * 8 + (lane & 7), m0 / 8 + (mi & 1))), a0, a1, a2, a3);
#pragma unroll
        for (int np = 0; np < NT / 2; ++np) {
            const int at = swz<SC_DV>(kk * 16 + (mi & 1) * 8 + (lane & 7), nt0 + np * 2 + (mi >> 1));
            uint32_t b0, b1, b2, b3;
            ldmatrix_x4_trans(smem_u32(x_s + at), b0, b1, b2, b3);
            mma_bf16(acc[np * 2], a0, a1, a2, a3, b0, b1);
            mma_bf16(acc[np * 2 + 1], a0, a1, a2, a3, b2, b3);
            ldmatrix_x4_trans(smem_u32(x_r + at), b0, b1, b2, b3);
            mma_bf16(acc[np * 2], a0, a1, a2, a3, b0, b1);
            mma_bf16(acc[np * 2 + 1], a0, a1, a2, a3, b2, b3);
        }
    }
    const size_t slot = (size_t)chunk_slot(q_start, r, c) * p.H + h;
    float* u = p.u + slot * p.N * p.dv + v0;
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int m = m0 + (lane >> 2) + (e >> 1) * 8, j = (nt0 + i) * 8 + (lane & 3) * 2 + (e & 1);
            if (m < p.N && j < vw) u[(size_t)m * p.dv + j] = acc[i][e];
        }
    if (threadIdx.x == 0 && blockIdx.z == 0) p.total[slot] = expf(last);
}

__global__ void ssd_chunk_chain_kernel(const SsdChunks p) {
    const int r = blockIdx.z, h = blockIdx.y, slot = p.row_slot[r];
    const int e = blockIdx.x * blockDim.x + threadIdx.x, size = p.N * p.dv;
    if (slot < 0 || e >= size) return;
    const int n = (p.row_q_len[r] + SC_L - 1) / SC_L;
    const size_t s0 = chunk_slot(p.row_q_start[r], r, 0);
    float cur = p.state[((size_t)slot * p.H + h) * size + e];
    constexpr int AHEAD = 8;
    for (int c0 = 0; c0 < n; c0 += AHEAD) {
        float u[AHEAD], a[AHEAD];
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
            const size_t s = (s0 + c0 + i) * p.H + h;
            u[i] = c0 + i < n ? p.u[s * size + e] : 0.f;
            a[i] = c0 + i < n ? p.total[s] : 0.f;
        }
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
            if (c0 + i >= n) break;
            p.u[((s0 + c0 + i) * p.H + h) * size + e] = cur;       // the state before the chunk, in the place of its U
            cur = fmaf(a[i], cur, u[i]);
        }
    }
    if (p.write_state) p.state[((size_t)slot * p.H + h) * size + e] = cur;
}

template <int NP>
__global__ void __launch_bounds__(SCH_THREADS)
ssd_chunk_out_kernel(const SsdChunks p) {
    constexpr int BT = SC_L * NP * 2, XT = SC_L * SC_DV * 2, ST = NP * SC_DV * 2;
    extern __shared__ __align__(128) unsigned char sm[];
    unsigned char* b_s = sm;                   // B [128][NP]
    unsigned char* c_s = b_s + BT;             // C [128][NP]
    unsigned char* x_s = c_s + BT;             // x [128][64]
    unsigned char* s_s = x_s + XT;             // the state before the chunk [NP][64], rounded, then the rest
    unsigned char* s_r = s_s + ST;
    __shared__ float cs[SC_L], dts[SC_L];
    const int r = blockIdx.x / p.max_chunks, c = blockIdx.x - r * p.max_chunks, h = blockIdx.y, v0 = blockIdx.z * SC_DV;
    const int q_start = p.row_q_start[r], q_len = p.row_q_len[r];
    if (p.row_slot[r] < 0 || c * SC_L >= q_len) return;
    const int tok0 = q_start + c * SC_L, n = min(SC_L, q_len - c * SC_L);
    const int inner = p.H * p.dv, g = h / (p.H / p.G), vw = min(SC_DV, p.dv - v0);
    const __nv_bfloat16* row0 = p.xbc + (size_t)tok0 * p.ld;
    load_tile<NP>(b_s, row0 + inner + g * p.N, p.ld, n, p.N, p.aligned);
    load_tile<NP>(c_s, row0 + inner + (p.G + g) * p.N, p.ld, n, p.N, p.aligned);
    load_tile<SC_DV>(x_s, row0 + h * p.dv + v0, p.ld, n, vw, p.aligned);
    cp_async_commit();
    chunk_decays(p, tok0, n, h, cs, dts);
    const float* st = p.u + ((size_t)chunk_slot(q_start, r, c) * p.H + h) * p.N * p.dv + v0;
    constexpr int UNR = 8;                     // loads in flight per thread
#pragma unroll 1
    for (int e0 = threadIdx.x; e0 < NP * SC_DV / 2; e0 += SCH_THREADS * UNR) {
        float2 x[UNR];
#pragma unroll
        for (int k = 0; k < UNR; ++k) {
            const int e = e0 + k * SCH_THREADS, m = e / (SC_DV / 2), j = (e - m * (SC_DV / 2)) * 2;
            x[k] = make_float2(0.f, 0.f);
            if (m < p.N && j < vw) {
                if (p.aligned) x[k] = *reinterpret_cast<const float2*>(st + (size_t)m * p.dv + j);
                else x[k] = make_float2(st[(size_t)m * p.dv + j], j + 1 < vw ? st[(size_t)m * p.dv + j + 1] : 0.f);
            }
        }
#pragma unroll
        for (int k = 0; k < UNR; ++k) {
            const int e = e0 + k * SCH_THREADS, m = e / (SC_DV / 2), j = (e - m * (SC_DV / 2)) * 2;
            const int at = swz<SC_DV>(m, j >> 3) + (j & 7) * 2;
            *reinterpret_cast<uint32_t*>(s_s + at) = pack_bf16(x[k].x, x[k].y);
            *reinterpret_cast<uint32_t*>(s_r + at) = pack_bf16_rest(x[k].x, x[k].y);
        }
    }
    cp_async_wait<0>();
    __syncthreads();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, mi = lane >> 3;
    const int i0 = warp * 16;                  // the warp's 16 tokens
    if (i0 >= n) return;
    uint32_t cf[NP / 16][4];
#pragma unroll
    for (int ks = 0; ks < NP / 16; ++ks)
        ldmatrix_x4(smem_u32(c_s + swz<NP>(i0 + (mi & 1) * 8 + (lane & 7), ks * 2 + (mi >> 1))), cf[ks][0], cf[ks][1], cf[ks][2], cf[ks][3]);
    float acc[SC_DV / 8][4];
#pragma unroll
    for (int i = 0; i < SC_DV / 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    // what the state before the chunk contributes: C S, times exp(L_i)
#pragma unroll
    for (int kk = 0; kk < NP / 16; ++kk)
#pragma unroll
        for (int np = 0; np < SC_DV / 16; ++np) {
            const int at = swz<SC_DV>(kk * 16 + (mi & 1) * 8 + (lane & 7), np * 2 + (mi >> 1));
            uint32_t b0, b1, b2, b3;
            ldmatrix_x4_trans(smem_u32(s_s + at), b0, b1, b2, b3);
            mma_bf16(acc[np * 2], cf[kk][0], cf[kk][1], cf[kk][2], cf[kk][3], b0, b1);
            mma_bf16(acc[np * 2 + 1], cf[kk][0], cf[kk][1], cf[kk][2], cf[kk][3], b2, b3);
            ldmatrix_x4_trans(smem_u32(s_r + at), b0, b1, b2, b3);
            mma_bf16(acc[np * 2], cf[kk][0], cf[kk][1], cf[kk][2], cf[kk][3], b0, b1);
            mma_bf16(acc[np * 2 + 1], cf[kk][0], cf[kk][1], cf[kk][2], cf[kk][3], b2, b3);
        }
    const int ra = i0 + (lane >> 2);           // this thread's rows: ra and ra + 8
    const float la = cs[ra], lb = cs[ra + 8];
    {
        const float ea = expf(la), eb = expf(lb);
#pragma unroll
        for (int i = 0; i < SC_DV / 8; ++i) { acc[i][0] *= ea; acc[i][1] *= ea; acc[i][2] *= eb; acc[i][3] *= eb; }
    }
    // the chunk's own tokens, sixteen at a time
    for (int jb = 0; jb <= warp; ++jb) {
        float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
        for (int kk = 0; kk < NP / 16; ++kk) {
            uint32_t b0, b1, b2, b3;
            ldmatrix_x4(smem_u32(b_s + swz<NP>(jb * 16 + (mi >> 1) * 8 + (lane & 7), kk * 2 + (mi & 1))), b0, b1, b2, b3);
            mma_bf16(s[0], cf[kk][0], cf[kk][1], cf[kk][2], cf[kk][3], b0, b1);
            mma_bf16(s[1], cf[kk][0], cf[kk][1], cf[kk][2], cf[kk][3], b2, b3);
        }
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int j = jb * 16 + nt * 8 + (lane & 3) * 2 + (e & 1), i = ra + (e >> 1) * 8;
                s[nt][e] = j <= i ? s[nt][e] * expf(((e >> 1) ? lb : la) - cs[j]) * dts[j] : 0.f;
            }
        const uint32_t pa0 = pack_bf16(s[0][0], s[0][1]), pa1 = pack_bf16(s[0][2], s[0][3]);
        const uint32_t pa2 = pack_bf16(s[1][0], s[1][1]), pa3 = pack_bf16(s[1][2], s[1][3]);
        const uint32_t pb0 = pack_bf16_rest(s[0][0], s[0][1]), pb1 = pack_bf16_rest(s[0][2], s[0][3]);
        const uint32_t pb2 = pack_bf16_rest(s[1][0], s[1][1]), pb3 = pack_bf16_rest(s[1][2], s[1][3]);
#pragma unroll
        for (int np = 0; np < SC_DV / 16; ++np) {
            uint32_t b0, b1, b2, b3;
            ldmatrix_x4_trans(smem_u32(x_s + swz<SC_DV>(jb * 16 + (mi & 1) * 8 + (lane & 7), np * 2 + (mi >> 1))), b0, b1, b2, b3);
            mma_bf16(acc[np * 2], pa0, pa1, pa2, pa3, b0, b1);
            mma_bf16(acc[np * 2 + 1], pa0, pa1, pa2, pa3, b2, b3);
            mma_bf16(acc[np * 2], pb0, pb1, pb2, pb3, b0, b1);
            mma_bf16(acc[np * 2 + 1], pb0, pb1, pb2, pb3, b2, b3);
        }
    }
#pragma unroll
    for (int i = 0; i < SC_DV / 8; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int t = ra + (e >> 1) * 8, j = i * 8 + (lane & 3) * 2 + (e & 1);
            if (t < n && j < vw) p.y[(size_t)(tok0 + t) * inner + h * p.dv + v0 + j] = acc[i][e];
        }
}

template <int NP>
static int launch_chunks(const SsdChunks& p, int n_rows, cudaStream_t stream) {
    constexpr size_t smem_state = (size_t)SC_L * NP * 2 + 2 * SC_L * SC_DV * 2;
    constexpr size_t smem_out = 2 * (size_t)SC_L * NP * 2 + SC_L * SC_DV * 2 + 2 * NP * SC_DV * 2;
    static bool configured = false;
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(ssd_chunk_state_kernel<NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_state);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(ssd_chunk_out_kernel<NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_out);
        if (e != cudaSuccess) return fail(-3, "ssd_chunks: cannot get %zu bytes of shared memory: %s", smem_out, cudaGetErrorString(e));
        configured = true;
    }
    const dim3 one(1, 1, 1), block(SCH_THREADS), grid((unsigned)n_rows * p.max_chunks, p.H, (p.dv + SC_DV - 1) / SC_DV);
    int rc = launch("ssd_chunk_state", ssd_chunk_state_kernel<NP>, grid, block, smem_state, stream, one, p);
    if (rc) return rc;
    rc = launch("ssd_chunk_chain", ssd_chunk_chain_kernel, dim3((p.N * p.dv + 255) / 256, p.H, n_rows), dim3(256), 0, stream, one, p);
    if (rc) return rc;
    return launch("ssd_chunk_out", ssd_chunk_out_kernel<NP>, grid, block, smem_out, stream, one, p);
}

}  // namespace fd

using namespace fd;
typedef __nv_bfloat16 bf16;

// proj [T, ld] of `dtype` (0 float32, 1 bfloat16): x, B, C are the C columns from `col` on, the raw step sizes the H columns from
// dt_col on.  conv_w [C, taps], conv_b [C]; ring [slots, taps, C] (unused when taps == 1).  xbc [T, C], of which the first
// float_cols columns are written, and step [T, H, 2] float; xbc16 [T, C] bfloat16 or null.
// keep: rows of a single token leave their values in the ring here; longer rows need fd_conv_ring_update.
extern "C" int fd_ssd_prepare(const void* proj, int ld, int dtype, int col, int C, int dt_col, const float* conv_w, const float* conv_b,
                              float* ring, int taps, int keep, const float* dt_bias, const float* A_log, float* xbc, void* xbc16,
                              int float_cols, float* step,
                              const int* tok_row, const int* tok_pos, const int* row_slot, const int* row_q_start,
                              const int* row_q_len, int T, int H, cudaStream_t stream) {
    if (T == 0) return 0;
    FD_REQUIRE(C > 0 && H > 0 && ld >= col + C && ld >= dt_col + H, -2, "ssd_prepare: %d channels, %d heads in rows of %d", C, H, ld);
    FD_REQUIRE(taps >= 1 && (taps == 1 || ring != nullptr), -2, "ssd_prepare: %d taps need a ring", taps);
    const int tpc = T > 64 ? SC_TOK : 1;
    const dim3 grid((T + tpc - 1) / tpc, (C + SSD_THREADS - 1) / SSD_THREADS + 1);
    FD_REQUIRE(grid.y <= 65535, -2, "ssd_prepare: %d channels", C);
    if (dtype == 0)
        return launch("ssd_prepare", ssd_prepare_kernel<float>, grid, dim3(SSD_THREADS), 0, stream, dim3(1, 1, 1), (const float*)proj, ld,
                      col, C, dt_col, conv_w, conv_b, ring, taps, keep, dt_bias, A_log, xbc, (bf16*)xbc16, float_cols, step, tok_row, tok_pos, row_slot,
                      row_q_start, row_q_len, T, H, tpc);
    return launch("ssd_prepare", ssd_prepare_kernel<bf16>, grid, dim3(SSD_THREADS), 0, stream, dim3(1, 1, 1), (const bf16*)proj, ld, col,
                  C, dt_col, conv_w, conv_b, ring, taps, keep, dt_bias, A_log, xbc, (bf16*)xbc16, float_cols, step, tok_row, tok_pos, row_slot, row_q_start,
                  row_q_len, T, H, tpc);
}

// y [T, inner] float; xbc: the convolved x in the first `inner` columns of rows of ldx floats; D [inner / dv]; z: pointer to the first
// gate column (rows of ldz, dtype as out); w [inner]; out: pointer to the first output column, rows of ld_out.
extern "C" int fd_ssd_gate_norm(const float* y, const float* xbc, int ldx, const float* D, const void* z, int ldz, const float* w,
                                void* out, int ld_out, int dtype, int T, int inner, int dv, int parts, float eps, float scale,
                                cudaStream_t stream) {
    if (T == 0) return 0;
    FD_REQUIRE(dv > 0 && inner % dv == 0 && parts > 0 && inner % parts == 0 && parts <= 65535 && T <= 65535, -2,
               "ssd_gate_norm: %d channels in heads of %d and %d parts, %d tokens", inner, dv, parts, T);
    const int part = inner / parts;
    FD_REQUIRE(part <= 12000, -2, "ssd_gate_norm: parts of %d channels (at most 12000)", part);
    const dim3 grid(parts, T), block(part >= 256 ? 256 : (part + 31) / 32 * 32);
    const size_t smem = (size_t)part * sizeof(float);
    if (dtype == 0)
        return launch("ssd_gate_norm", ssd_gate_norm_kernel<float>, grid, block, smem, stream, dim3(1, 1, 1), y, xbc, ldx, D,
                      (const float*)z, ldz, w, (float*)out, ld_out, inner, dv, part, eps, scale);
    return launch("ssd_gate_norm", ssd_gate_norm_kernel<bf16>, grid, block, smem, stream, dim3(1, 1, 1), y, xbc, ldx, D, (const bf16*)z,
                  ldz, w, (bf16*)out, ld_out, inner, dv, part, eps, scale);
}

// Whether the chunk form takes the sizes, the tokens of a chunk, and the floats of scratch memory a step of T tokens in n_rows
// sequences needs.
extern "C" int fd_ssd_chunks_takes(int N, int dv) { return N >= 1 && N <= 128 && dv >= 1; }
extern "C" int fd_ssd_chunk() { return SC_L; }
extern "C" long long fd_ssd_chunks_scratch_floats(int T, int n_rows, int H, int N, int dv) {
    return (long long)(T / SC_L + n_rows + 1) * H * ((long long)N * dv + 1);
}

// xbc [T, ld] bfloat16: x (H dv columns), B (G N), C (G N); step [T, H, 2] float (step size, decay); A_log [H]; state
// [slots, H, N, dv] float; y [T, H dv] float; scratch: fd_ssd_chunks_scratch_floats floats.
extern "C" int fd_ssd_chunks(const void* xbc, int ld, const float* step, const float* A_log, float* state, float* y, const int* row_slot,
                             const int* row_q_start, const int* row_q_len, int n_rows, int T, int max_q_len, int H, int G, int N, int dv,
                             int write_state, float* scratch, long long scratch_floats, cudaStream_t stream) {
    if (n_rows == 0 || T == 0) return 0;
    FD_REQUIRE(fd_ssd_chunks_takes(N, dv) && H > 0 && G > 0 && H % G == 0 && ld >= H * dv + 2 * G * N, -2,
               "ssd_chunks: %d heads in %d groups, a state of %d x %d", H, G, N, dv);
    FD_REQUIRE(scratch != nullptr && scratch_floats >= fd_ssd_chunks_scratch_floats(T, n_rows, H, N, dv), -2,
               "ssd_chunks: %lld floats of scratch memory for %d tokens", scratch_floats, T);
    SsdChunks p;
    p.xbc = (const bf16*)xbc; p.ld = ld; p.step = step; p.A_log = A_log; p.state = state; p.y = y;
    p.u = scratch; p.total = scratch + (long long)(T / SC_L + n_rows + 1) * H * N * dv;
    p.row_slot = row_slot; p.row_q_start = row_q_start; p.row_q_len = row_q_len;
    p.H = H; p.G = G; p.N = N; p.dv = dv; p.max_chunks = (max_q_len + SC_L - 1) / SC_L; p.write_state = write_state;
    p.aligned = ld % 8 == 0 && dv % 8 == 0 && N % 8 == 0 && (H * dv) % 8 == 0 && (uintptr_t)xbc % 16 == 0;
    FD_REQUIRE(H <= 65535 && n_rows <= 65535 && (long long)n_rows * p.max_chunks < (1ll << 31), -2, "ssd_chunks: %d rows", n_rows);
    return N <= 64 ? launch_chunks<64>(p, n_rows, stream) : launch_chunks<128>(p, n_rows, stream);
}
