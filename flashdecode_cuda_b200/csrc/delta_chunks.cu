// The gated delta rule (delta_rule.cu) for prompts in bfloat16: sixteen tokens at a time on the tensor cores (mma.m16n8k16).
//
// With L_i the sum of a chunk's log decays up to token i (per key channel), S the state before the chunk, and
//     k~_i = exp(L_i) k_i,   q~_i = exp(L_i) q_i,   A_ij = sum_c k_i k_j exp(L_i - L_j) (j < i),   P_ij = the same with q_i (j <= i),
// the sixteen corrections solve (I + diag(beta) A) U = diag(beta) (V - K~ S); with T the inverse of that unit triangular matrix
//     U = (T diag(beta)) (V - K~ S),      O = Q~ S + P U,      S <- exp(L_end) S + sum_j (exp(L_end - L_j) k_j) u_j^T.
//  * delta_chunk_prepare: everything of a chunk that does not depend on the state - k~, q~, the tail-decayed keys, T diag(beta), P -
//    for all chunks side by side.  Exponents are sums of log decays of later tokens, at most 0: nothing is divided.
//  * delta_chunk_scan: the chunks in order.  A CTA takes 16 value columns, each of its warps 32 key channels: S^T [16, 32] as float
//    accumulators, which are at the same time, rounded, the first operand of the warp's products, so that no state goes
//    through memory between chunks.  The warps add up their shares of K~ S and Q~ S in shared memory, in a fixed order; that is
//    the one barrier of a chunk.
// State, decays, exponentials, sums and the inverse are float.  What enters a product goes in as two bfloat16 numbers, the rounded
// one and what the rounding took away (three products: 16 bits of mantissa on both sides).
#include <math.h>

#include "mma_utils.cuh"

namespace fd {

constexpr int DC_TOK = 16;
constexpr int DC_STAGES = 4;                   // chunks of the scan in flight or in use
constexpr int DC_VLD = 20;                     // floats of a token's 16 values in shared memory

struct DeltaChunks {
    const float* q; const float* k; const float* v; const float* lg; const float* beta;   // as delta_prepare leaves them
    float* state; float* out;                  // [slots, H, d, dv], [T, H dv]
    unsigned char* chunks;                     // [chunk slots, H, dc_bytes]
    const int* row_slot; const int* row_q_start; const int* row_q_len;
    int H, Hk, d, dv, dp, dvp, write_state, max_chunks, single;       // rows of up to `single` tokens are someone else's
};
// Bytes of a chunk: k~, q~, tail keys [16][DK] bfloat16, rounded and rest each; T diag(beta) and P [16][16] likewise; the whole decay [DK] float
template <int DK> __host__ __device__ constexpr int dc_bytes() { return 6 * DC_TOK * DK * 2 + 4 * DC_TOK * DC_TOK * 2 + DK * 4; }
// ... and of its place in the scan's shared memory: with the values of the CTA's 16 columns
template <int DK> __host__ __device__ constexpr int dc_stage() { return dc_bytes<DK>() + DC_TOK * DC_VLD * 4; }
__device__ __forceinline__ int dc_slot(int q_start, int r, int c) { return q_start / DC_TOK + r + c; }

template <int DK>
__global__ void __launch_bounds__(256)
delta_chunk_prepare_kernel(const DeltaChunks p) {
    constexpr int LD = DK + 1;
    __shared__ float L[DC_TOK * LD], k_s[DC_TOK * LD], q_s[DC_TOK * LD];
    __shared__ float a_s[DC_TOK][DC_TOK + 1], p_s[DC_TOK][DC_TOK + 1], t_s[DC_TOK][DC_TOK + 1], beta_s[DC_TOK];
    const int r = blockIdx.x / p.max_chunks, c = blockIdx.x - r * p.max_chunks, h = blockIdx.y;
    const int q_start = p.row_q_start[r], q_len = p.row_q_len[r];
    if (p.row_slot[r] < 0 || q_len <= p.single || c * DC_TOK >= q_len) return;
    const int n = min(DC_TOK, q_len - c * DC_TOK), hk = h / (p.H / p.Hk), tid = threadIdx.x;
    const size_t t0 = q_start + c * DC_TOK;
    if (tid < DC_TOK) beta_s[tid] = tid < n ? p.beta[(t0 + tid) * p.H + h] : 0.f;
    if (tid < DK) {                            // the log decays of a channel summed up over the chunk, in base 2
        float x[DC_TOK];
#pragma unroll
        for (int i = 0; i < DC_TOK; ++i) x[i] = i < n && tid < p.d ? p.lg[((t0 + i) * p.H + h) * p.dp + tid] : 0.f;
        float sum = 0.f;
#pragma unroll
        for (int i = 0; i < DC_TOK; ++i) { sum = fmaf(x[i], 1.4426950408889634f, sum); L[i * LD + tid] = sum; }
    }
#pragma unroll
    for (int e = 0; e < DC_TOK * DK / 256; ++e) {
        const int idx = tid + e * 256, i = idx / DK, ch = idx - i * DK;
        const bool in = i < n && ch < p.d;
        k_s[i * LD + ch] = in ? p.k[((t0 + i) * p.Hk + hk) * p.dp + ch] : 0.f;
        q_s[i * LD + ch] = in ? p.q[((t0 + i) * p.Hk + hk) * p.dp + ch] : 0.f;
    }
    __syncthreads();
    unsigned char* out = p.chunks + ((size_t)dc_slot(q_start, r, c) * p.H + h) * dc_bytes<DK>();
    uint32_t* vec = reinterpret_cast<uint32_t*>(out);
    constexpr int HALF = DC_TOK * DK / 2;      // pairs of one array
#pragma unroll
    for (int e = 0; e < HALF / 256; ++e) {
        const int idx = tid + e * 256, i = idx / (DK / 2), ch = (idx - i * (DK / 2)) * 2;
        const float l0 = L[i * LD + ch], l1 = L[i * LD + ch + 1];
        const float e0 = exp2f(l0), e1 = exp2f(l1);
        const float x0 = exp2f(L[(DC_TOK - 1) * LD + ch] - l0), x1 = exp2f(L[(DC_TOK - 1) * LD + ch + 1] - l1);
        const float k0 = k_s[i * LD + ch], k1 = k_s[i * LD + ch + 1], q0 = q_s[i * LD + ch], q1 = q_s[i * LD + ch + 1];
        vec[idx] = pack_bf16(e0 * k0, e1 * k1);
        vec[HALF + idx] = pack_bf16_rest(e0 * k0, e1 * k1);
        vec[2 * HALF + idx] = pack_bf16(e0 * q0, e1 * q1);
        vec[3 * HALF + idx] = pack_bf16_rest(e0 * q0, e1 * q1);
        vec[4 * HALF + idx] = pack_bf16(x0 * k0, x1 * k1);
        vec[5 * HALF + idx] = pack_bf16_rest(x0 * k0, x1 * k1);
    }
    float* whole = reinterpret_cast<float*>(out + 6 * DC_TOK * DK * 2 + 4 * DC_TOK * DC_TOK * 2);
    if (tid < DK) whole[tid] = exp2f(L[(DC_TOK - 1) * LD + tid]);
    // A and P: threads (i, j) and (j, i) share the pair, half of the channels each; a diagonal thread has P_ii, which decays by nothing
    {
        const int ti = tid / DC_TOK, tj = tid % DC_TOK, i = max(ti, tj), j = min(ti, tj);
        float a = 0.f, b = 0.f;
        if (i == j) {
            for (int ch = 0; ch < DK; ++ch) b = fmaf(q_s[i * LD + ch], k_s[i * LD + ch], b);
            p_s[i][i] = b;
        } else {
            const int c0 = ti > tj ? 0 : DK / 2;
#pragma unroll 8
            for (int ch = c0; ch < c0 + DK / 2; ++ch) {
                const float w = k_s[j * LD + ch] * exp2f(L[i * LD + ch] - L[j * LD + ch]);
                a = fmaf(k_s[i * LD + ch], w, a);
                b = fmaf(q_s[i * LD + ch], w, b);
            }
            a_s[ti][tj] = a;                   // the first half below the diagonal, the second above
            p_s[ti][tj] = b;
        }
    }
    __syncthreads();
    if (tid < 32) {
        const int j = tid & (DC_TOK - 1);      // column j of T: forward substitution
        float t[DC_TOK];
#pragma unroll
        for (int i = 0; i < DC_TOK; ++i) {
            float s = i == j ? 1.f : 0.f;
#pragma unroll
            for (int m = 0; m < DC_TOK; ++m) if (m < i) s = fmaf(-beta_s[i] * (a_s[i][m] + a_s[m][i]), t[m], s);
            t[i] = i < j ? 0.f : s;
        }
        if (tid < DC_TOK) {
#pragma unroll
            for (int i = 0; i < DC_TOK; ++i) t_s[i][j] = t[i] * beta_s[j];
        }
    }
    __syncthreads();
    uint32_t* mats = reinterpret_cast<uint32_t*>(out + 6 * DC_TOK * DK * 2);
    if (tid < 2 * DC_TOK * DC_TOK / 2) {
        const int which = tid >> 7, idx = tid & 127, i = idx >> 3, j = (idx & 7) * 2;
        float x0, x1;
        if (which == 0) { x0 = t_s[i][j]; x1 = t_s[i][j + 1]; }
        else {
            x0 = j < i ? p_s[i][j] + p_s[j][i] : (j == i ? p_s[i][i] : 0.f);
            x1 = j + 1 < i ? p_s[i][j + 1] + p_s[j + 1][i] : (j + 1 == i ? p_s[i][i] : 0.f);
        }
        mats[which * 256 + idx] = pack_bf16(x0, x1);
        mats[which * 256 + 128 + idx] = pack_bf16_rest(x0, x1);
    }
}

// a1 b1 + a1 b2 + a2 b1 into accumulators of their own: x ~ x1 + x2 on both sides
__device__ __forceinline__ void mma3(float hh[4], float hl[4], float lh[4], const uint32_t a1[4], const uint32_t a2[4], uint32_t b0, uint32_t b1,
                                     uint32_t r0, uint32_t r1) {
    mma_bf16(hh, a1[0], a1[1], a1[2], a1[3], b0, b1);
    mma_bf16(hl, a1[0], a1[1], a1[2], a1[3], r0, r1);
    mma_bf16(lh, a2[0], a2[1], a2[2], a2[3], b0, b1);
}
// two accumulator tiles of eight columns as the first operand of a product over those sixteen columns
__device__ __forceinline__ void as_operand(const float x[4], const float y[4], uint32_t hi[4], uint32_t lo[4]) {
    hi[0] = pack_bf16(x[0], x[1]); hi[1] = pack_bf16(x[2], x[3]); hi[2] = pack_bf16(y[0], y[1]); hi[3] = pack_bf16(y[2], y[3]);
    lo[0] = pack_bf16_rest(x[0], x[1]); lo[1] = pack_bf16_rest(x[2], x[3]); lo[2] = pack_bf16_rest(y[0], y[1]); lo[3] = pack_bf16_rest(y[2], y[3]);
}

template <int DK>
__global__ void __launch_bounds__(DK)
delta_chunk_scan_kernel(const DeltaChunks p) {
    constexpr int WARPS = DK / 32, THREADS = DK;
    constexpr int CPR = DK / 8, ARR = DC_TOK * DK * 2, MATS = 6 * ARR, TAIL = 4 * DC_TOK * DC_TOK * 2 + DK * 4, BYTES = dc_bytes<DK>();
    constexpr int STAGE = dc_stage<DK>();
    extern __shared__ __align__(128) unsigned char sm[];
    float4* red = reinterpret_cast<float4*>(sm + DC_STAGES * STAGE);       // [2][warp][X or Y][token tile][lane]
    const int tiles = (p.dv + 15) / 16;
    const int r = blockIdx.x / tiles, tile = blockIdx.x - r * tiles, h = blockIdx.y;
    const int slot = p.row_slot[r], q_start = p.row_q_start[r], q_len = p.row_q_len[r];
    if (slot < 0 || q_len <= p.single) return;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, mi = lane >> 3;
    const int v_a = tile * 16 + (lane >> 2), v_b = v_a + 8;                // the thread's two value columns
    const int c2 = (lane & 3) * 2;
    const bool in_a = v_a < p.dv, in_b = v_b < p.dv;
    float* st = p.state + ((size_t)slot * p.H + h) * p.d * p.dv;
    float S[4][4];                             // S^T: value columns v_a, v_b by key channels 32 warp + 8 t + c2, + 1
#pragma unroll
    for (int t = 0; t < 4; ++t)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int ch = warp * 32 + t * 8 + c2 + (e & 1);
            S[t][e] = ch < p.d && ((e >> 1) ? in_b : in_a) ? st[(size_t)ch * p.dv + ((e >> 1) ? v_b : v_a)] : 0.f;
        }
    const int n_chunks = (q_len + DC_TOK - 1) / DC_TOK;
    const size_t slot0 = (size_t)dc_slot(q_start, r, 0);
    auto issue = [&](int c) {
        if (c < n_chunks) {
            const unsigned char* src = p.chunks + ((slot0 + c) * p.H + h) * BYTES;
            unsigned char* dst = sm + (c % DC_STAGES) * STAGE;
#pragma unroll
            for (int e = 0; e < 6 * DC_TOK * CPR / THREADS; ++e) {
                const int idx = tid + e * THREADS, row = idx / CPR, cc = idx % CPR;     // row: array * 16 + token
                cp_async16(smem_u32(dst + (row >> 4) * ARR + swz<DK>(row & 15, cc)), src + idx * 16, 16);
            }
#pragma unroll
            for (int e = 0; e < (TAIL / 16 + THREADS - 1) / THREADS; ++e) {
                const int idx = tid + e * THREADS;
                if (idx < TAIL / 16) cp_async16(smem_u32(dst + MATS + idx * 16), src + MATS + idx * 16, 16);
            }
            if (tid < 64) {                    // the chunk's values of these columns, rows of DC_VLD floats
                const int t = tid >> 2, i = (tid & 3) * 4;
                const bool in = c * DC_TOK + t < q_len && tile * 16 + i < p.dvp;
                cp_async16(smem_u32(dst + BYTES + (t * DC_VLD + i) * 4),
                           in ? p.v + ((size_t)(q_start + c * DC_TOK + t) * p.H + h) * p.dvp + tile * 16 + i : p.v, in ? 16 : 0);
            }
        }
        cp_async_commit();
    };
#pragma unroll
    for (int c = 0; c < DC_STAGES - 1; ++c) issue(c);
    cp_async_wait<DC_STAGES - 2>();
    __syncthreads();
    for (int c = 0; c < n_chunks; ++c) {
        const unsigned char* buf = sm + (c % DC_STAGES) * STAGE;
        const uint32_t base = smem_u32(buf);
        float4* mine = red + (c & 1) * WARPS * 128;
        {
            float X[3][2][4], Y[3][2][4];
#pragma unroll
            for (int a = 0; a < 3; ++a)
#pragma unroll
                for (int t = 0; t < 2; ++t)
#pragma unroll
                    for (int e = 0; e < 4; ++e) X[a][t][e] = Y[a][t][e] = 0.f;
            // the warp's share of X^T = S^T K~^T and Y^T = S^T Q~^T: its 32 key channels
#pragma unroll
            for (int kk = 0; kk < 2; ++kk) {
                uint32_t hi[4], lo[4], b[4], s[4];
                as_operand(S[2 * kk], S[2 * kk + 1], hi, lo);
                const uint32_t at = base + swz<DK>((mi >> 1) * 8 + (lane & 7), (warp * 2 + kk) * 2 + (mi & 1));
                ldmatrix_x4(at, b[0], b[1], b[2], b[3]);
                ldmatrix_x4(at + ARR, s[0], s[1], s[2], s[3]);
                mma3(X[0][0], X[1][0], X[2][0], hi, lo, b[0], b[1], s[0], s[1]);
                mma3(X[0][1], X[1][1], X[2][1], hi, lo, b[2], b[3], s[2], s[3]);
                ldmatrix_x4(at + 2 * ARR, b[0], b[1], b[2], b[3]);
                ldmatrix_x4(at + 3 * ARR, s[0], s[1], s[2], s[3]);
                mma3(Y[0][0], Y[1][0], Y[2][0], hi, lo, b[0], b[1], s[0], s[1]);
                mma3(Y[0][1], Y[1][1], Y[2][1], hi, lo, b[2], b[3], s[2], s[3]);
            }
#pragma unroll
            for (int t = 0; t < 2; ++t) {
                float x[4], y[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    x[e] = X[0][t][e] + (X[1][t][e] + X[2][t][e]);
                    y[e] = Y[0][t][e] + (Y[1][t][e] + Y[2][t][e]);
                }
                mine[(warp * 4 + t) * 32 + lane] = make_float4(x[0], x[1], x[2], x[3]);
                mine[(warp * 4 + 2 + t) * 32 + lane] = make_float4(y[0], y[1], y[2], y[3]);
            }
        }
        // the one meeting of a chunk: the shares are there, the next chunk's data too, and everyone is through with the last one's
        cp_async_wait<DC_STAGES - 3>();
        __syncthreads();
        issue(c + DC_STAGES - 1);
        float D[2][4];
        const float* v_s = reinterpret_cast<const float*>(buf + BYTES);
#pragma unroll
        for (int t = 0; t < 2; ++t) {
            float x[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int w = 0; w < WARPS; ++w) {
                const float4 o = mine[(w * 4 + t) * 32 + lane];
                x[0] += o.x; x[1] += o.y; x[2] += o.z; x[3] += o.w;
            }
#pragma unroll
            for (int e = 0; e < 4; ++e) D[t][e] = v_s[(t * 8 + c2 + (e & 1)) * DC_VLD + (lane >> 2) + (e >> 1) * 8] - x[e];
        }
        // U^T = D^T (T diag(beta))^T
        uint32_t hi[4], lo[4], b[4], s[4];
        const uint32_t mat = base + MATS + ((mi >> 1) * 8 + (lane & 7)) * 32 + (mi & 1) * 16;
        float U[3][2][4];
#pragma unroll
        for (int a = 0; a < 3; ++a)
#pragma unroll
            for (int t = 0; t < 2; ++t)
#pragma unroll
                for (int e = 0; e < 4; ++e) U[a][t][e] = 0.f;
        as_operand(D[0], D[1], hi, lo);
        ldmatrix_x4(mat, b[0], b[1], b[2], b[3]);
        ldmatrix_x4(mat + 512, s[0], s[1], s[2], s[3]);
        mma3(U[0][0], U[1][0], U[2][0], hi, lo, b[0], b[1], s[0], s[1]);
        mma3(U[0][1], U[1][1], U[2][1], hi, lo, b[2], b[3], s[2], s[3]);
        // the tail-decayed keys and the decay while that is under way
        uint32_t kb[2][4], ks[2][4];
#pragma unroll
        for (int np = 0; np < 2; ++np) {
            const uint32_t at = base + 4 * ARR + swz<DK>((mi & 1) * 8 + (lane & 7), (warp * 2 + np) * 2 + (mi >> 1));
            ldmatrix_x4_trans(at, kb[np][0], kb[np][1], kb[np][2], kb[np][3]);
            ldmatrix_x4_trans(at + ARR, ks[np][0], ks[np][1], ks[np][2], ks[np][3]);
        }
        const unsigned char* whole = buf + MATS + 4 * DC_TOK * DC_TOK * 2;
#pragma unroll
        for (int t = 0; t < 4; ++t) {
            const float2 w = *reinterpret_cast<const float2*>(whole + (warp * 32 + t * 8 + c2) * 4);
            S[t][0] *= w.x; S[t][1] *= w.y; S[t][2] *= w.x; S[t][3] *= w.y;
        }
#pragma unroll
        for (int t = 0; t < 2; ++t)
#pragma unroll
            for (int e = 0; e < 4; ++e) U[0][t][e] += U[1][t][e] + U[2][t][e];
        as_operand(U[0][0], U[0][1], hi, lo);
        // S^T <- S^T exp(L_end) + U^T K_tail
#pragma unroll
        for (int np = 0; np < 2; ++np) {
            mma_bf16(S[2 * np], hi[0], hi[1], hi[2], hi[3], kb[np][0], kb[np][1]);
            mma_bf16(S[2 * np + 1], hi[0], hi[1], hi[2], hi[3], kb[np][2], kb[np][3]);
        }
#pragma unroll
        for (int np = 0; np < 2; ++np) {
            mma_bf16(S[2 * np], hi[0], hi[1], hi[2], hi[3], ks[np][0], ks[np][1]);
            mma_bf16(S[2 * np + 1], hi[0], hi[1], hi[2], hi[3], ks[np][2], ks[np][3]);
        }
#pragma unroll
        for (int np = 0; np < 2; ++np) {
            mma_bf16(S[2 * np], lo[0], lo[1], lo[2], lo[3], kb[np][0], kb[np][1]);
            mma_bf16(S[2 * np + 1], lo[0], lo[1], lo[2], lo[3], kb[np][2], kb[np][3]);
        }
        // O^T = Y^T + U^T P^T: the first two warps, eight tokens each
        if (warp < 2) {
            float o[3][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
            for (int w = 0; w < WARPS; ++w) {
                const float4 y = mine[(w * 4 + 2 + warp) * 32 + lane];
                o[0][0] += y.x; o[0][1] += y.y; o[0][2] += y.z; o[0][3] += y.w;
            }
            ldmatrix_x4(mat + 1024, b[0], b[1], b[2], b[3]);
            ldmatrix_x4(mat + 1536, s[0], s[1], s[2], s[3]);
            if (warp == 0) mma3(o[0], o[1], o[2], hi, lo, b[0], b[1], s[0], s[1]);
            else mma3(o[0], o[1], o[2], hi, lo, b[2], b[3], s[2], s[3]);
            const int t = c * DC_TOK + warp * 8 + c2;
            float* out = p.out + ((size_t)(q_start + t) * p.H + h) * p.dv;
            const size_t next = (size_t)p.H * p.dv;
#pragma unroll
            for (int e = 0; e < 4; ++e)
                if (t + (e & 1) < q_len && ((e >> 1) ? in_b : in_a)) out[(e & 1) * next + ((e >> 1) ? v_b : v_a)] = o[0][e] + (o[1][e] + o[2][e]);
        }
    }
    cp_async_wait<0>();
    if (p.write_state) {
#pragma unroll
        for (int t = 0; t < 4; ++t)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int ch = warp * 32 + t * 8 + c2 + (e & 1);
                if (ch < p.d && ((e >> 1) ? in_b : in_a)) st[(size_t)ch * p.dv + ((e >> 1) ? v_b : v_a)] = S[t][e];
            }
    }
}

template <int DK>
static int launch_delta_chunks(const DeltaChunks& p, int n_rows, cudaStream_t stream) {
    constexpr int smem = DC_STAGES * dc_stage<DK>() + 2 * (DK / 32) * 128 * 16;
    auto k = delta_chunk_scan_kernel<DK>;
    static bool configured = false;
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
        if (e != cudaSuccess) return fail(-3, "delta_chunks: cannot get %d bytes of shared memory: %s", smem, cudaGetErrorString(e));
        configured = true;
    }
    const dim3 one(1, 1, 1);
    int rc = launch("delta_chunk_prepare", delta_chunk_prepare_kernel<DK>, dim3((unsigned)n_rows * p.max_chunks, p.H), dim3(256), 0, stream, one, p);
    if (rc) return rc;
    return launch("delta_chunk_scan", k, dim3((unsigned)((p.dv + 15) / 16) * n_rows, p.H), dim3(DK), smem, stream, one, p);
}

}  // namespace fd

using namespace fd;

extern "C" int fd_delta_chunks_takes(int d) { return d >= 1 && d <= 128; }
extern "C" long long fd_delta_chunks_scratch_bytes(int T, int n_rows, int H, int d) {
    return (long long)(T / DC_TOK + n_rows + 1) * H * (d <= 64 ? dc_bytes<64>() : dc_bytes<128>());
}

// q, k [T, Hk, dp], lg [T, H, dp] (log decays), v [T, H, dvp], beta [T, H] as fd_delta_prepare leaves them; state [slots, H, d, dv] and out
// [T, H dv] float; scratch: fd_delta_chunks_scratch_bytes bytes, 16-byte aligned.  Rows of up to `single` tokens are left out.
extern "C" int fd_delta_chunks(const float* q, const float* k, const float* v, const float* lg, const float* beta, float* state, float* out,
                               const int* row_slot, const int* row_q_start, const int* row_q_len, int n_rows, int T, int max_q_len,
                               int H, int Hk, int d, int dv, int write_state, int single, void* scratch, long long scratch_bytes,
                               cudaStream_t stream) {
    if (n_rows == 0 || T == 0) return 0;
    FD_REQUIRE(fd_delta_chunks_takes(d) && H > 0 && Hk > 0 && H % Hk == 0 && dv > 0 && H <= 65535, -2,
               "delta_chunks: %d heads on %d of %d x %d (keys up to 128)", H, Hk, d, dv);
    FD_REQUIRE(scratch != nullptr && (uintptr_t)scratch % 16 == 0 && scratch_bytes >= fd_delta_chunks_scratch_bytes(T, n_rows, H, d), -2,
               "delta_chunks: %lld bytes of scratch memory for %d tokens", scratch_bytes, T);
    DeltaChunks p = {q, k, v, lg, beta, state, out, (unsigned char*)scratch, row_slot, row_q_start, row_q_len, H, Hk, d, dv,
                     (d + 3) / 4 * 4, (dv + 3) / 4 * 4, write_state, (max_q_len + DC_TOK - 1) / DC_TOK, single};
    FD_REQUIRE((long long)n_rows * p.max_chunks < (1ll << 31), -2, "delta_chunks: %d rows of %d tokens", n_rows, max_q_len);
    return d <= 64 ? launch_delta_chunks<64>(p, n_rows, stream) : launch_delta_chunks<128>(p, n_rows, stream);
}
