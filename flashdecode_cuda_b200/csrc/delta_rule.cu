// The gated delta rule with a decay per head and key channel, for prompts and decode steps:
//
//   F_t = diag(g_t) S_(t-1);  S_t = F_t + k_t u_t^T, u_t = beta_t (v_t - F_t^T k_t);  o_t = S_t^T q_t    S [d, dv] per sequence and head
//
//  * delta_prepare: everything that enters the recurrence, as floats.  q, k and v pass a short causal convolution over time
//    per channel (short_conv.cuh) and silu; every head of q and k becomes a unit vector, x / sqrt(sum x^2 + 1e-6), and q is
//    multiplied by a constant; the log decay log g = -exp(A_h) softplus(z + bias) per key channel with z a narrow vector times
//    a matrix (or handed over); beta = sigmoid of a column per head; by option the output gate's pre-activation from its own
//    narrow vector.
//  * delta_scan: the recurrence.  A CTA of 128 threads takes one sequence of the step, one head and 16 value columns; 8
//    adjacent lanes share a column and each holds NR adjacent rows of it in registers.  Tokens come to shared memory a chunk
//    ahead with cp.async.  Per token the lanes add up S^T k and S^T q of the decayed state with shuffles that run side
//    by side; the read-out after the write is o = S^T q + (k . q) u, with k . q added up beside them.
//    Rows of up to DR_SINGLE tokens only; longer ones:
//  * delta_blocks and delta_block_scan: four tokens at a time.  With c_i the product of the block's decays up to token i, the
//    corrections of a block follow from S^T (c_i k_i) alone and from products of the block's own keys,
//        u_i = beta_i (v_i - S^T (c_i k_i) - sum_(j<i) A_ij u_j),      o_i = S^T (c_i q_i) + sum_(j<=i) P_ij u_j,
//        S <- c_4 S + sum_j (g_(j+1) .. g_4 k_j) u_j^T,     A_ij = sum_c k_i k_j g_(j+1) .. g_i,  P_ij the same with q_i,
//    in which decays are only multiplied, never divided.  The first kernel leaves the 13 vectors and 16 products of
//    every block (nothing in it depends on the state); the second walks the blocks, one reduction over the lanes per block
//    instead of one per token, blocks three ahead on their way with cp.async.
//  * conv_ring_update: after a step with longer portions, the last values of every row go to its ring.
//
// State, decays, step sizes, unit vectors, sums: float.  A sequence's tokens are walked in order, so the sums of every
// state element are the same however a prompt was cut into steps.
#include <math.h>

#include "mma_utils.cuh"
#include "short_conv.cuh"

namespace fd {

constexpr float DELTA_UNIT_EPS = 1e-6f;
constexpr int DR_THREADS = 128;
constexpr int DR_DS = 8;                       // lanes that share a column
constexpr int DR_VT = DR_THREADS / DR_DS;      // value columns of a CTA
constexpr int DR_TC = 16;                      // tokens of a chunk
constexpr int DR_SINGLE = 16;                  // the most tokens of a row that is walked token by token
constexpr int DB_VT = 8;                       // block form: value columns of a CTA
constexpr int DB_TOK = 4, DB_VECS = 13, DB_SCAL = 20, DB_STAGES = 4;

struct DeltaParams {
    const void* proj; int ld;                  // [T, ld]
    int q_col, k_col, v_col, b_col, a_col, g_col;      // first columns of q, k, v, beta, and of the decay's and the gate's narrow vectors
    const float* conv_w;                       // [C, taps], C = 2 Hk d + H dv: the channels of q, k, v
    float* ring;                               // [slots, taps, C]
    int taps, keep;
    const void* a2; const void* g2;            // [H d, R] and [H dv, R2], type of proj; null: z_a / z_g hold the products already
    int R, R2;
    const float* z_a;                          // [T, H d] or null
    const float* A_log; const float* dt_bias;  // [H], [H d]
    float q_scale;
    float* q; float* k; float* v; float* g; float* beta; float* gate_z;    // [T, Hk, dp], [T, Hk, dp], [T, H, dvp], [T, H, dp], [T, H], [T, H dv]
    const int* tok_row; const int* tok_pos; const int* row_slot; const int* row_q_start; const int* row_q_len;
    int T, H, Hk, d, dv, dp, dvp, tpc;
};

// out[tt] = sum_r w[row, r] x[tt][r]: a narrow vector per token (in shared memory, [SC_TOK][R]) times one row of a matrix
template <typename T>
__device__ __forceinline__ void expand_row(const T* __restrict__ w, const float* x_s, int R, float out[SC_TOK]) {
#pragma unroll
    for (int tt = 0; tt < SC_TOK; ++tt) out[tt] = 0.f;
    constexpr int VEC = 16 / sizeof(T);
    if (R % VEC == 0) {
#pragma unroll 4
        for (int r0 = 0; r0 < R; r0 += VEC) {
            const uint4 raw = *reinterpret_cast<const uint4*>(w + r0);
            const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
            for (int j4 = 0; j4 < VEC; j4 += 4) {
                float wv[4];
#pragma unroll
                for (int j = 0; j < 4; ++j) wv[j] = to_float(e[j4 + j]);
#pragma unroll
                for (int tt = 0; tt < SC_TOK; ++tt) {
                    const float4 xv = *reinterpret_cast<const float4*>(x_s + tt * R + r0 + j4);
                    out[tt] = fmaf(wv[0], xv.x, out[tt]); out[tt] = fmaf(wv[1], xv.y, out[tt]);
                    out[tt] = fmaf(wv[2], xv.z, out[tt]); out[tt] = fmaf(wv[3], xv.w, out[tt]);
                }
            }
        }
    } else {
        for (int r = 0; r < R; ++r) {
            const float wv = to_float(w[r]);
#pragma unroll
            for (int tt = 0; tt < SC_TOK; ++tt) out[tt] = fmaf(wv, x_s[tt * R + r], out[tt]);
        }
    }
}

// grid (token tiles, units): q heads, k heads, v heads, decay heads, gate heads
// NARROW: decay heads (and gate heads, if any) expand their narrow vectors here
template <typename T, bool NARROW>
__global__ void __launch_bounds__(256)
delta_prepare_kernel(const DeltaParams p) {
    __shared__ ConvMeta meta;
    __shared__ float red[SC_TOK][8];
    extern __shared__ __align__(16) float x_s[];            // [SC_TOK][R] of the units that expand a narrow vector
    const int t0 = blockIdx.x * p.tpc, nt = min(p.tpc, p.T - t0);
    const int tid = threadIdx.x;
    const T* proj = static_cast<const T*>(p.proj);
    int u = blockIdx.y;
    const int nqk = p.Hk * p.d, C = 2 * nqk + p.H * p.dv;
    conv_meta(meta, t0, nt, p.tok_row, p.tok_pos, p.row_slot, p.row_q_start, p.row_q_len);
    if (u < 2 * p.Hk) {                                     // a head of q or k
        const bool is_q = u < p.Hk;
        const int h = is_q ? u : u - p.Hk;
        const bool active = tid < p.d;
        const int c = (is_q ? 0 : nqk) + h * p.d + (active ? tid : 0);
        const T* col = proj + (is_q ? p.q_col : p.k_col) + h * p.d + (active ? tid : 0);
        float x[SC_VALS], y[SC_TOK];
        if (p.tpc > 1) conv_load<T>(col, p.ld, t0, nt, x);
        __syncthreads();
        conv_channel<T>(col, p.ld, p.conv_w + (size_t)c * p.taps, 0.f, p.taps, p.ring, c, C, meta, t0, nt, p.keep && active, x, y);
#pragma unroll
        for (int tt = 0; tt < SC_TOK; ++tt) {
            if (tt >= nt) continue;
            y[tt] = active ? sc_silu<T>(y[tt]) : 0.f;
            const float s = warp_sum(y[tt] * y[tt]);
            if ((tid & 31) == 0) red[tt][tid >> 5] = s;
        }
        __syncthreads();
        if (tid >= p.dp) return;
        float* out = is_q ? p.q : p.k;
        const int nw = blockDim.x >> 5;
        const float scale = is_q ? p.q_scale : 1.f;
        out += ((size_t)t0 * p.Hk + h) * p.dp + tid;
#pragma unroll
        for (int tt = 0; tt < SC_TOK; ++tt) {
            if (tt >= nt || meta.slot[tt] < 0) continue;
            float total = 0.f;
            for (int w = 0; w < nw; ++w) total += red[tt][w];
            out[(size_t)tt * p.Hk * p.dp] = y[tt] * (scale * rsqrtf(total + DELTA_UNIT_EPS));
        }
        return;
    }
    u -= 2 * p.Hk;
    if (u < p.H) {                                          // a head of v
        __syncthreads();
        for (int j = tid; j < p.dvp; j += blockDim.x) {
            const bool active = j < p.dv;
            const int c = 2 * nqk + u * p.dv + (active ? j : 0);
            const T* col = proj + p.v_col + u * p.dv + (active ? j : 0);
            float x[SC_VALS], y[SC_TOK];
            if (p.tpc > 1) conv_load<T>(col, p.ld, t0, nt, x);
            conv_channel<T>(col, p.ld, p.conv_w + (size_t)c * p.taps, 0.f, p.taps, p.ring, c, C, meta, t0, nt, p.keep && active, x, y);
#pragma unroll
            for (int tt = 0; tt < SC_TOK; ++tt)
                if (tt < nt && meta.slot[tt] >= 0)
                    p.v[((size_t)(t0 + tt) * p.H + u) * p.dvp + j] = active ? sc_silu<T>(y[tt]) : 0.f;
        }
        return;
    }
    u -= p.H;
    const bool is_gate = u >= p.H;
    const int h = is_gate ? u - p.H : u;
    const int R = is_gate ? p.R2 : p.R, col = is_gate ? p.g_col : p.a_col;
    const T* w = static_cast<const T*>(is_gate ? p.g2 : p.a2);
    if (NARROW && w != nullptr)
        for (int e = tid; e < SC_TOK * R; e += blockDim.x) {
            const int tt = e / R, r = e - tt * R;
            x_s[e] = tt < nt ? to_float(proj[(size_t)(t0 + tt) * p.ld + col + r]) : 0.f;
        }
    __syncthreads();
    if (NARROW && is_gate) {
        for (int j = tid; j < p.dv; j += blockDim.x) {
            float z[SC_TOK];
            expand_row<T>(w + (size_t)(h * p.dv + j) * R, x_s, R, z);
#pragma unroll
            for (int tt = 0; tt < SC_TOK; ++tt)
                if (tt < nt) p.gate_z[((size_t)(t0 + tt) * p.H + h) * p.dv + j] = z[tt];
        }
        return;
    }
    if (tid < nt) p.beta[(size_t)(t0 + tid) * p.H + h] = sc_sigmoid(to_float(proj[(size_t)(t0 + tid) * p.ld + p.b_col + h]));
    const float rate = expf(p.A_log[h]);
    for (int j = tid; j < p.dp; j += blockDim.x) {
        float z[SC_TOK];
        const bool active = j < p.d;
        if (NARROW && active && w != nullptr) {
            expand_row<T>(w + (size_t)(h * p.d + j) * R, x_s, R, z);
        } else {
#pragma unroll
            for (int tt = 0; tt < SC_TOK; ++tt)
                z[tt] = active && tt < nt ? p.z_a[((size_t)(t0 + tt) * p.H + h) * p.d + j] : 0.f;
        }
        const float b = active ? p.dt_bias[h * p.d + j] : 0.f;
#pragma unroll
        for (int tt = 0; tt < SC_TOK; ++tt)
            if (tt < nt) p.g[((size_t)(t0 + tt) * p.H + h) * p.dp + j] = active ? -rate * sc_softplus(z[tt] + b) : 0.f;
    }
}

struct DeltaScan {
    const float* q; const float* k; const float* v; const float* g; const float* beta;      // g: log decays
    float* state; float* out;                  // [slots, H, d, dv], [T, H dv]
    const int* row_slot; const int* row_q_start; const int* row_q_len;
    int H, Hk, d, dv, dp, dvp, write_state;
    float* blocks; float* scal;                // block form: [block slots, H, DB_VECS, dp], [block slots, H, DB_SCAL]; or null
    int max_blocks;                            // blocks of the longest row
    int short_only;                            // rows of more than DR_SINGLE tokens are not walked token by token
};

// Block b of step row r has the slot q_start / 4 + r + b: slots of different rows never meet.
__device__ __forceinline__ int block_slot(int q_start, int r, int b) { return q_start / DB_TOK + r + b; }

// floats of NR rows in shared memory: 4 apart from a multiple of 32 banks, so that the DS lanes of a column read different banks
template <int NR> __host__ __device__ constexpr int dr_stride() { return NR == 4 ? 4 : NR + 4; }

template <int NR>
__global__ void __launch_bounds__(DR_THREADS)
delta_scan_kernel(const DeltaScan p) {
    constexpr int CS = DR_DS * dr_stride<NR>();              // floats of a token's k, q or g
    constexpr int TS = 3 * CS + DR_VT + 4;                   // and of the token: k, q, g, v, beta
    extern __shared__ __align__(16) float sm[];              // two chunks, filled in turn
    const int tiles = (p.dv + DR_VT - 1) / DR_VT;
    const int r = blockIdx.x / tiles, tile = blockIdx.x - r * tiles, h = blockIdx.y;
    const int slot = p.row_slot[r];
    if (slot < 0) return;
    const int q_start = p.row_q_start[r], q_len = p.row_q_len[r];
    if (p.short_only && q_len > DR_SINGLE) return;           // a row of another form
    const int hk = h / (p.H / p.Hk);
    const int tid = threadIdx.x;
    const int vl = tid / DR_DS, ds = tid % DR_DS;
    const int col = tile * DR_VT + vl;
    const bool live = col < p.dv;
    float* st = p.state + ((size_t)slot * p.H + h) * p.d * p.dv;

    float S[NR];
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        const int row = ds * NR + i;
        S[i] = live && row < p.d ? st[(size_t)row * p.dv + col] : 0.f;
    }
    if (p.dp < DR_DS * NR) {                                 // places of channels at or beyond dp are never filled: zero once
        for (int e = tid; e < 2 * DR_TC * TS; e += DR_THREADS) sm[e] = 0.f;
        __syncthreads();
    }

    auto issue = [&](int c0, int buf) {
        const int n = min(DR_TC, q_len - c0);
        float* dst = sm + buf * DR_TC * TS;
        const int per = p.dp >> 2;                           // 16-byte pieces of a token's k, q or g
        const size_t t = q_start + c0;
        for (int piece = tid; piece < 3 * per; piece += DR_THREADS) {      // a thread's piece of every token of the chunk
            const int which = piece >= 2 * per ? 2 : (piece >= per ? 1 : 0);
            const int i = (piece - which * per) * 4;
            const float* src = which == 2 ? p.g + (t * p.H + h) * p.dp + i : (which == 1 ? p.q : p.k) + (t * p.Hk + hk) * p.dp + i;
            const size_t step = (size_t)(which == 2 ? p.H : p.Hk) * p.dp;
            uint32_t at = smem_u32(dst + which * CS + (i / NR) * dr_stride<NR>() + i % NR);
#pragma unroll 4
            for (int tt = 0; tt < n; ++tt, src += step, at += TS * 4) cp_async16(at, src, 16);
        }
        if (tid < n * (DR_VT / 4)) {
            const int tt = tid / (DR_VT / 4), i = (tid % (DR_VT / 4)) * 4;
            const bool in = tile * DR_VT + i < p.dvp;
            cp_async16(smem_u32(dst + tt * TS + 3 * CS + i), in ? p.v + ((t + tt) * p.H + h) * p.dvp + tile * DR_VT + i : p.v, in ? 16 : 0);
        } else if (tid >= DR_THREADS - DR_TC && tid - (DR_THREADS - DR_TC) < n) {
            const int tt = tid - (DR_THREADS - DR_TC);
            asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(dst + tt * TS + 3 * CS + DR_VT)),
                         "l"(p.beta + (t + tt) * p.H + h) : "memory");
        }
        cp_async_commit();
    };
    issue(0, 0);
    int it = 0;
    for (int c0 = 0; c0 < q_len; c0 += DR_TC, ++it) {
        const int n = min(DR_TC, q_len - c0);
        float* buf = sm + (it & 1) * DR_TC * TS;
        if (c0 + DR_TC < q_len) { issue(c0 + DR_TC, (it + 1) & 1); cp_async_wait<1>(); }
        else cp_async_wait<0>();
        __syncthreads();
        for (int i = tid; i < n * p.dp; i += DR_THREADS) {   // the decays from their logarithms
            const int tt = i / p.dp, ch = i - tt * p.dp;
            float* at = buf + tt * TS + 2 * CS + (ch / NR) * dr_stride<NR>() + ch % NR;
            *at = expf(*at);
        }
        __syncthreads();
        const float* mine = buf + ds * dr_stride<NR>();
#pragma unroll 1
        for (int tt = 0; tt < n; ++tt) {
            const float* tk = mine + tt * TS;
            const float beta = buf[tt * TS + 3 * CS + DR_VT];
            const float v = buf[tt * TS + 3 * CS + vl];
            float kk[NR];
            float sk[4] = {0.f, 0.f, 0.f, 0.f}, sq[4] = {0.f, 0.f, 0.f, 0.f}, kq[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int i = 0; i < NR; i += 4) {
                const float4 k4 = *reinterpret_cast<const float4*>(tk + i);
                const float4 q4 = *reinterpret_cast<const float4*>(tk + CS + i);
                const float4 g4 = *reinterpret_cast<const float4*>(tk + 2 * CS + i);
                kk[i] = k4.x; kk[i + 1] = k4.y; kk[i + 2] = k4.z; kk[i + 3] = k4.w;
                S[i] *= g4.x; S[i + 1] *= g4.y; S[i + 2] *= g4.z; S[i + 3] *= g4.w;
                sk[0] = fmaf(S[i], k4.x, sk[0]); sk[1] = fmaf(S[i + 1], k4.y, sk[1]);
                sk[2] = fmaf(S[i + 2], k4.z, sk[2]); sk[3] = fmaf(S[i + 3], k4.w, sk[3]);
                sq[0] = fmaf(S[i], q4.x, sq[0]); sq[1] = fmaf(S[i + 1], q4.y, sq[1]);
                sq[2] = fmaf(S[i + 2], q4.z, sq[2]); sq[3] = fmaf(S[i + 3], q4.w, sq[3]);
                kq[0] = fmaf(k4.x, q4.x, kq[0]); kq[1] = fmaf(k4.y, q4.y, kq[1]);
                kq[2] = fmaf(k4.z, q4.z, kq[2]); kq[3] = fmaf(k4.w, q4.w, kq[3]);
            }
            float ak = (sk[0] + sk[1]) + (sk[2] + sk[3]), aq = (sq[0] + sq[1]) + (sq[2] + sq[3]);
            float akq = (kq[0] + kq[1]) + (kq[2] + kq[3]);
#pragma unroll
            for (int off = 1; off < DR_DS; off <<= 1) {
                ak += __shfl_xor_sync(0xffffffffu, ak, off);
                aq += __shfl_xor_sync(0xffffffffu, aq, off);
                akq += __shfl_xor_sync(0xffffffffu, akq, off);
            }
            const float un = beta * (v - ak);
#pragma unroll
            for (int i = 0; i < NR; ++i) S[i] = fmaf(kk[i], un, S[i]);
            if (ds == 0 && live) p.out[((size_t)(q_start + c0 + tt) * p.H + h) * p.dv + col] = fmaf(akq, un, aq);
        }
        __syncthreads();                                     // the chunk is through before its place is filled again
    }
    if (p.write_state && live) {
#pragma unroll
        for (int i = 0; i < NR; ++i) {
            const int row = ds * NR + i;
            if (row < p.d) st[(size_t)row * p.dv + col] = S[i];
        }
    }
}

// grid (rows x blocks, heads), a thread per key channel.  Vectors of a block: c_i k_i (4), c_i q_i (4), g_(j+1) .. g_4 k_j (4), c_4.
// Scalars: A_10, A_20, A_21, A_30, A_31, A_32, P_00, P_10, P_11, P_20, .. P_33, then beta_0 .. beta_3.
__global__ void __launch_bounds__(256)
delta_blocks_kernel(const DeltaScan p) {
    __shared__ float red[16][8];
    const int r = blockIdx.x / p.max_blocks, b = blockIdx.x - r * p.max_blocks, h = blockIdx.y;
    const int q_start = p.row_q_start[r], q_len = p.row_q_len[r];
    if (p.row_slot[r] < 0 || q_len <= DR_SINGLE || b * DB_TOK >= q_len) return;
    const int n = min(DB_TOK, q_len - b * DB_TOK);
    const int hk = h / (p.H / p.Hk), tid = threadIdx.x;
    const bool active = tid < p.dp;
    float k[4], q[4], g[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        k[i] = q[i] = 0.f; g[i] = 1.f;                       // tokens the row does not have change nothing
        if (active && i < n) {
            const size_t t = q_start + b * DB_TOK + i;
            k[i] = p.k[(t * p.Hk + hk) * p.dp + tid];
            q[i] = p.q[(t * p.Hk + hk) * p.dp + tid];
            g[i] = expf(p.g[(t * p.H + h) * p.dp + tid]);
        }
    }
    const size_t slot = (size_t)block_slot(q_start, r, b) * p.H + h;
    if (active) {
        float* out = p.blocks + slot * DB_VECS * p.dp + tid;
        float c = 1.f;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            c *= g[i];
            out[i * p.dp] = c * k[i];
            out[(4 + i) * p.dp] = c * q[i];
        }
        out[12 * p.dp] = c;
        float tail = 1.f;
#pragma unroll
        for (int j = 3; j >= 0; --j) {
            out[(8 + j) * p.dp] = tail * k[j];
            tail *= g[j];
        }
    }
    // products of the block's own keys and queries, the decays between the two tokens on them
    float x[16];
    int at_a = 0, at_p = 6;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        float w[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            w[j] = 1.f;
#pragma unroll
            for (int e = 0; e < 4; ++e) if (e > j && e <= i) w[j] *= g[e];
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            if (j < i) x[at_a++] = k[i] * k[j] * w[j];
            if (j <= i) x[at_p++] = q[i] * k[j] * w[j];
        }
    }
    const int lane = tid & 31, warp = tid >> 5, n_warps = blockDim.x >> 5;
#pragma unroll
    for (int e = 0; e < 16; ++e) {
        const float s = warp_sum(x[e]);
        if (lane == 0) red[e][warp] = s;
    }
    __syncthreads();
    if (tid < 16) {
        float s = 0.f;
        for (int w = 0; w < n_warps; ++w) s += red[tid][w];
        p.scal[slot * DB_SCAL + tid] = s;
    } else if (tid < DB_SCAL) {
        const int i = tid - 16;
        p.scal[slot * DB_SCAL + tid] = i < n ? p.beta[(size_t)(q_start + b * DB_TOK + i) * p.H + h] : 0.f;
    }
}

// two floats in one register pair: sm_100 multiplies and adds both in one instruction
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
    f32x2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
    f32x2 d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ f32x2 pair2(float lo, float hi) {
    f32x2 d;
    asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
    return d;
}
__device__ __forceinline__ float2 split2(f32x2 a) {
    float2 d;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(d.x), "=f"(d.y) : "l"(a));
    return d;
}

// DS lanes share a column and hold NR rows of it each.  What bounds the time is the chain of a block's own steps (loads, sums, the
// reduction, the four corrections, the update), one block after the other: so the sums run in eight chains side by side.
template <int NR, int DS>
__global__ void __launch_bounds__(DS * DB_VT)
delta_block_scan_kernel(const DeltaScan p) {
    constexpr int DB_THREADS = DS * DB_VT, WARPS = DB_THREADS / 32;
    constexpr int CS = DS * dr_stride<NR>();
    constexpr int VT = DB_VT;
    constexpr int BS = DB_VECS * CS + DB_TOK * VT + DB_SCAL; // floats of a block in shared memory
    extern __shared__ __align__(16) float sm[];
    const int tiles = (p.dv + VT - 1) / VT;
    const int r = blockIdx.x / tiles, tile = blockIdx.x - r * tiles, h = blockIdx.y;
    const int slot = p.row_slot[r];
    const int q_start = p.row_q_start[r], q_len = p.row_q_len[r];
    if (slot < 0 || q_len <= DR_SINGLE) return;
    const int tid = threadIdx.x, lane = tid & 31, vl = tid / DS, ds = tid % DS;
    const int col = tile * VT + vl;
    const bool live = col < p.dv;
    float* st = p.state + ((size_t)slot * p.H + h) * p.d * p.dv;
    f32x2 S[NR / 2];                                         // rows ds * NR + 2 i and the next of the thread's column
#pragma unroll
    for (int i = 0; i < NR / 2; ++i) {
        const int row = ds * NR + 2 * i;
        S[i] = pair2(live && row < p.d ? st[(size_t)row * p.dv + col] : 0.f, live && row + 1 < p.d ? st[(size_t)(row + 1) * p.dv + col] : 0.f);
    }
    if (p.dp < DS * NR) {                                 // places of channels at or beyond dp are never filled: zero once
        for (int e = tid; e < DB_STAGES * BS; e += DB_THREADS) sm[e] = 0.f;
        __syncthreads();
    }
    const int n_blocks = (q_len + DB_TOK - 1) / DB_TOK;
    const int per = p.dp >> 2;
    const size_t slot0 = (size_t)block_slot(q_start, r, 0);
    auto issue = [&](int b) {
        if (b < n_blocks) {
            float* dst = sm + (b % DB_STAGES) * BS;
            const size_t bs = (slot0 + b) * p.H + h;
            const float* src = p.blocks + bs * DB_VECS * p.dp;
            for (int piece = lane; piece < per; piece += 32) {      // the warps take the vectors in turn
                const int i = piece * 4;
                const uint32_t at = smem_u32(dst + (i / NR) * dr_stride<NR>() + i % NR);
                const float* from = src + i;
#pragma unroll
                for (int e = 0; e < (DB_VECS + WARPS - 1) / WARPS; ++e) {
                    const int v = (tid >> 5) + e * WARPS;
                    if (v < DB_VECS) cp_async16(at + v * CS * 4, from + v * p.dp, 16);
                }
            }
            if (tid >= 32 && tid < 32 + DB_TOK * VT / 4) {
                const int e = tid - 32, tt = e / (VT / 4), i = (e % (VT / 4)) * 4, t = b * DB_TOK + tt;
                const bool in = tile * VT + i < p.dvp && t < q_len;
                cp_async16(smem_u32(dst + DB_VECS * CS + tt * VT + i),
                           in ? p.v + ((size_t)(q_start + t) * p.H + h) * p.dvp + tile * VT + i : p.v, in ? 16 : 0);
            } else if (tid >= 48 && tid < 48 + DB_SCAL / 4) {
                const int e = tid - 48;
                cp_async16(smem_u32(dst + DB_VECS * CS + DB_TOK * VT + e * 4), p.scal + bs * DB_SCAL + e * 4, 16);
            }
        }
        cp_async_commit();
    };
#pragma unroll
    for (int b = 0; b < DB_STAGES - 1; ++b) issue(b);
    for (int b = 0; b < n_blocks; ++b) {
        cp_async_wait<DB_STAGES - 2>();
        __syncthreads();                                     // block b is there, and everyone is through with block b - 1
        issue(b + DB_STAGES - 1);
        const float* buf = sm + (b % DB_STAGES) * BS;
        const float* mine = buf + ds * dr_stride<NR>();
        f32x2 ak[4], aq[4];
#pragma unroll
        for (int t = 0; t < 4; ++t) ak[t] = aq[t] = 0ull;    // two zeros
#pragma unroll
        for (int i = 0; i < NR; i += 4) {
            ulonglong2 k4[4], q4[4];
#pragma unroll
            for (int t = 0; t < 4; ++t) {
                k4[t] = *reinterpret_cast<const ulonglong2*>(mine + t * CS + i);
                q4[t] = *reinterpret_cast<const ulonglong2*>(mine + (4 + t) * CS + i);
            }
#pragma unroll
            for (int t = 0; t < 4; ++t) { ak[t] = fma2(S[i / 2], k4[t].x, ak[t]); aq[t] = fma2(S[i / 2], q4[t].x, aq[t]); }
#pragma unroll
            for (int t = 0; t < 4; ++t) { ak[t] = fma2(S[i / 2 + 1], k4[t].y, ak[t]); aq[t] = fma2(S[i / 2 + 1], q4[t].y, aq[t]); }
        }
        // what the update needs from memory, and the decay, while the reduction runs
        ulonglong2 w4[4][NR / 4];
#pragma unroll
        for (int t = 0; t < 4; ++t)
#pragma unroll
            for (int i = 0; i < NR / 4; ++i) w4[t][i] = *reinterpret_cast<const ulonglong2*>(mine + (8 + t) * CS + i * 4);
#pragma unroll
        for (int i = 0; i < NR / 4; ++i) {
            const ulonglong2 c4 = *reinterpret_cast<const ulonglong2*>(mine + 12 * CS + i * 4);
            S[2 * i] = mul2(S[2 * i], c4.x);
            S[2 * i + 1] = mul2(S[2 * i + 1], c4.y);
        }
        float dk[4], dq[4];
#pragma unroll
        for (int t = 0; t < 4; ++t) {
            const float2 a = split2(ak[t]), c = split2(aq[t]);
            dk[t] = a.x + a.y;
            dq[t] = c.x + c.y;
        }
#pragma unroll
        for (int off = 1; off < DS; off <<= 1)
#pragma unroll
            for (int t = 0; t < 4; ++t) {
                dk[t] += __shfl_xor_sync(0xffffffffu, dk[t], off);
                dq[t] += __shfl_xor_sync(0xffffffffu, dq[t], off);
            }
        const float* v_s = buf + DB_VECS * CS + vl;
        const float4* sc = reinterpret_cast<const float4*>(buf + DB_VECS * CS + DB_TOK * VT);
        const float4 s0 = sc[0], s1 = sc[1], s2 = sc[2], s3 = sc[3], be = sc[4];
        const float A[6] = {s0.x, s0.y, s0.z, s0.w, s1.x, s1.y};
        const float P[10] = {s1.z, s1.w, s2.x, s2.y, s2.z, s2.w, s3.x, s3.y, s3.z, s3.w};
        const float beta[4] = {be.x, be.y, be.z, be.w};
        float u[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            float s = v_s[i * VT] - dk[i];
#pragma unroll
            for (int j = 0; j < 4; ++j) if (j < i) s = fmaf(-A[i * (i - 1) / 2 + j], u[j], s);
            u[i] = beta[i] * s;
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) {
#pragma unroll
            for (int j = 0; j < 4; ++j) if (j <= i) dq[i] = fmaf(P[i * (i + 1) / 2 + j], u[j], dq[i]);
        }
        f32x2 uu[4];
#pragma unroll
        for (int t = 0; t < 4; ++t) uu[t] = pair2(u[t], u[t]);
#pragma unroll
        for (int t = 0; t < 4; ++t)
#pragma unroll
            for (int i = 0; i < NR / 4; ++i) {
                S[2 * i] = fma2(w4[t][i].x, uu[t], S[2 * i]);
                S[2 * i + 1] = fma2(w4[t][i].y, uu[t], S[2 * i + 1]);
            }
        if (ds < 4 && b * DB_TOK + ds < q_len && live) {     // lane t of the first four writes token t
            const float o = ds == 0 ? dq[0] : ds == 1 ? dq[1] : ds == 2 ? dq[2] : dq[3];
            p.out[((size_t)(q_start + b * DB_TOK + ds) * p.H + h) * p.dv + col] = o;
        }
    }
    cp_async_wait<0>();
    if (p.write_state && live) {
#pragma unroll
        for (int i = 0; i < NR / 2; ++i) {
            const int row = ds * NR + 2 * i;
            const float2 x = split2(S[i]);
            if (row < p.d) st[(size_t)row * p.dv + col] = x.x;
            if (row + 1 < p.d) st[(size_t)(row + 1) * p.dv + col] = x.y;
        }
    }
}

// ring[slot][p % taps] <- the value of position p for the last taps - 1 positions that a row of several tokens brought
template <typename T>
__global__ void conv_ring_update_kernel(const T* __restrict__ proj, int ld, float* __restrict__ ring, const int* __restrict__ row_slot,
                                        const int* __restrict__ row_q_start, const int* __restrict__ row_q_len,
                                        const int* __restrict__ row_ctx_len, int C, int taps) {
    const int r = blockIdx.y, slot = row_slot[r], n = row_q_len[r];
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    if (slot < 0 || n <= 1 || c >= C) return;
    float* rg = ring + (size_t)slot * taps * C + c;
    for (int i = max(0, n - (taps - 1)); i < n; ++i)
        rg[(size_t)((row_ctx_len[r] + i) % taps) * C] = to_float(proj[(size_t)(row_q_start[r] + i) * ld + c]);
}

template <int NR>
static int launch_delta_scan(const DeltaScan& p, int n_rows, cudaStream_t stream) {
    constexpr size_t smem = 2 * (size_t)DR_TC * (3 * DR_DS * dr_stride<NR>() + DR_VT + 4) * sizeof(float);
    auto k = delta_scan_kernel<NR>;
    static bool configured = false;
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return fail(-3, "delta_scan: cannot get %zu bytes of shared memory: %s", smem, cudaGetErrorString(e));
        configured = true;
    }
    const int tiles = (p.dv + DR_VT - 1) / DR_VT;
    const dim3 one(1, 1, 1);
    int rc = launch("delta_scan", k, dim3((unsigned)tiles * n_rows, p.H), dim3(DR_THREADS), smem, stream, one, p);
    if (rc || p.blocks == nullptr) return rc;
    constexpr int BNR = NR > 8 ? NR / 2 : NR, BDS = NR > 8 ? 2 * DR_DS : DR_DS;      // block form: fewer rows in more lanes
    constexpr size_t bsmem = DB_STAGES * (size_t)(DB_VECS * BDS * dr_stride<BNR>() + DB_TOK * DB_VT + DB_SCAL) * sizeof(float);
    auto kb = delta_block_scan_kernel<BNR, BDS>;
    static bool block_configured = false;
    if (!block_configured) {
        cudaError_t e = cudaFuncSetAttribute(kb, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bsmem);
        if (e != cudaSuccess) return fail(-3, "delta_scan: cannot get %zu bytes of shared memory: %s", bsmem, cudaGetErrorString(e));
        block_configured = true;
    }
    rc = launch("delta_blocks", delta_blocks_kernel, dim3((unsigned)n_rows * p.max_blocks, p.H), dim3((p.dp + 31) / 32 * 32), 0, stream, one, p);
    if (rc) return rc;
    return launch("delta_block_scan", kb, dim3((unsigned)((p.dv + DB_VT - 1) / DB_VT) * n_rows, p.H), dim3(BDS * DB_VT), bsmem, stream, one, p);
}

}  // namespace fd

using namespace fd;
typedef __nv_bfloat16 bf16;

// dtype (0 float32, 1 bfloat16): type of proj, a2 and g2.  Columns count from the pointer.  conv_w [2 Hk d + H dv, taps]; ring
// [slots, taps, 2 Hk d + H dv] (unused when taps == 1).  a2 [H d, R] or null with z_a [T, H d]; g2 [H dv, R2] or null (the gate's
// pre-activation is then not made here).  Outputs: q, k [T, Hk, dp], g [T, H, dp] with dp = d rounded up to 4 (zeros after d; g: log decays), v
// [T, H, dvp], dvp = dv rounded up to 4, beta [T, H], gate_z [T, H dv]; all float.  keep: rows of a single token leave their
// values in the ring here; longer rows need fd_conv_ring_update.
extern "C" int fd_delta_prepare(const void* proj, int ld, int dtype, int q_col, int k_col, int v_col, int b_col, int a_col, int g_col,
                                const float* conv_w, float* ring, int taps, int keep, const void* a2, int R, const float* z_a,
                                const void* g2, int R2, const float* A_log, const float* dt_bias, float q_scale, float* q, float* k,
                                float* v, float* g, float* beta, float* gate_z, const int* tok_row, const int* tok_pos,
                                const int* row_slot, const int* row_q_start, const int* row_q_len, int T, int H, int Hk, int d,
                                int dv, cudaStream_t stream) {
    if (T == 0) return 0;
    FD_REQUIRE(H > 0 && Hk > 0 && H % Hk == 0 && d > 0 && d <= 256 && dv > 0, -2, "delta_prepare: %d heads on %d of %d x %d (keys up to 256)", H, Hk, d, dv);
    FD_REQUIRE(taps >= 1 && (taps == 1 || ring != nullptr), -2, "delta_prepare: %d taps need a ring", taps);
    FD_REQUIRE((a2 != nullptr && R >= 1) || z_a != nullptr, -2, "delta_prepare: no decay");
    FD_REQUIRE(g2 == nullptr || (R2 >= 1 && gate_z != nullptr), -2, "delta_prepare: the gate needs its output");
    const int r_max = (a2 ? R : 0) > (g2 ? R2 : 0) ? R : (g2 ? R2 : 0);
    FD_REQUIRE(r_max <= 1024, -2, "delta_prepare: narrow vectors of %d (at most 1024)", r_max);
    FD_REQUIRE((uintptr_t)a2 % 16 == 0 && (uintptr_t)g2 % 16 == 0, -2, "delta_prepare: 16-byte alignment");
    DeltaParams p;
    p.proj = proj; p.ld = ld; p.q_col = q_col; p.k_col = k_col; p.v_col = v_col; p.b_col = b_col; p.a_col = a_col; p.g_col = g_col;
    p.conv_w = conv_w; p.ring = ring; p.taps = taps; p.keep = keep; p.a2 = a2; p.g2 = g2; p.R = R; p.R2 = R2; p.z_a = z_a;
    p.A_log = A_log; p.dt_bias = dt_bias; p.q_scale = q_scale;
    p.q = q; p.k = k; p.v = v; p.g = g; p.beta = beta; p.gate_z = gate_z;
    p.tok_row = tok_row; p.tok_pos = tok_pos; p.row_slot = row_slot; p.row_q_start = row_q_start; p.row_q_len = row_q_len;
    p.T = T; p.H = H; p.Hk = Hk; p.d = d; p.dv = dv; p.dp = (d + 3) / 4 * 4; p.dvp = (dv + 3) / 4 * 4;
    p.tpc = T > 64 ? SC_TOK : 1;
    const int threads = p.dp > 128 ? 256 : (p.dp > 64 || dv > 64 ? 128 : 64);
    const size_t smem = (size_t)SC_TOK * r_max * sizeof(float);
    const dim3 grid((T + p.tpc - 1) / p.tpc, 2 * Hk + 2 * H + (g2 ? H : 0));
    FD_REQUIRE(grid.y <= 65535, -2, "delta_prepare: %d heads", H);
    const bool narrow = a2 != nullptr || g2 != nullptr;
    if (dtype == 0) {
        if (narrow) return launch("delta_prepare", delta_prepare_kernel<float, true>, grid, dim3(threads), smem, stream, dim3(1, 1, 1), p);
        return launch("delta_prepare", delta_prepare_kernel<float, false>, grid, dim3(threads), smem, stream, dim3(1, 1, 1), p);
    }
    if (narrow) return launch("delta_prepare", delta_prepare_kernel<bf16, true>, grid, dim3(threads), smem, stream, dim3(1, 1, 1), p);
    return launch("delta_prepare", delta_prepare_kernel<bf16, false>, grid, dim3(threads), smem, stream, dim3(1, 1, 1), p);
}

// q, k [T, Hk, dp], g [T, H, dp], v [T, H, dvp], beta [T, H] as fd_delta_prepare leaves them; state [slots, H, d, dv] and
// out [T, H dv] float.  max_q_len: the longest row of the step; rows of more than 16 tokens take the block form and need scratch
// memory, fd_delta_scan_scratch_floats floats (without it every row is walked token by token).  short_only: rows of more
// than 16 tokens are left out (fd_delta_chunks takes them).
extern "C" int fd_delta_scan_single() { return DR_SINGLE; }
extern "C" long long fd_delta_scan_scratch_floats(int T, int n_rows, int H, int d) {
    return (long long)(T / DB_TOK + n_rows + 1) * H * (DB_VECS * ((d + 3) / 4 * 4) + DB_SCAL);
}
extern "C" int fd_delta_scan(const float* q, const float* k, const float* v, const float* g, const float* beta, float* state,
                             float* out, const int* row_slot, const int* row_q_start, const int* row_q_len, int n_rows, int H,
                             int Hk, int d, int dv, int write_state, int T, int max_q_len, float* scratch, long long scratch_floats,
                             int short_only,
                             cudaStream_t stream) {
    if (n_rows == 0) return 0;
    FD_REQUIRE(H > 0 && Hk > 0 && H % Hk == 0 && d > 0 && d <= 256 && dv > 0, -2, "delta_scan: %d heads on %d of %d x %d (keys up to 256)", H, Hk, d, dv);
    FD_REQUIRE(H <= 65535 && (long long)n_rows * ((dv + DR_VT - 1) / DR_VT) < (1ll << 31), -2, "delta_scan: %d rows", n_rows);
    auto al = [](const void* x) { return (uintptr_t)x % 16 == 0; };
    FD_REQUIRE(al(q) && al(k) && al(v) && al(g), -2, "delta_scan: 16-byte alignment");
    DeltaScan p = {q, k, v, g, beta, state, out, row_slot, row_q_start, row_q_len, H, Hk, d, dv, (d + 3) / 4 * 4, (dv + 3) / 4 * 4, write_state,
                   nullptr, nullptr, 0, short_only || scratch != nullptr};
    if (scratch != nullptr && !short_only && max_q_len > DR_SINGLE) {
        FD_REQUIRE(scratch_floats >= fd_delta_scan_scratch_floats(T, n_rows, H, d) && (uintptr_t)scratch % 16 == 0, -2,
                   "delta_scan: %lld floats of scratch memory for %d tokens", scratch_floats, T);
        p.blocks = scratch;
        p.scal = scratch + (long long)(T / DB_TOK + n_rows + 1) * H * DB_VECS * p.dp;
        p.max_blocks = (max_q_len + DB_TOK - 1) / DB_TOK;
        FD_REQUIRE((long long)n_rows * p.max_blocks < (1ll << 31), -2, "delta_scan: %d rows of %d tokens", n_rows, max_q_len);
    }
    if (d <= 32) return launch_delta_scan<4>(p, n_rows, stream);
    if (d <= 64) return launch_delta_scan<8>(p, n_rows, stream);
    if (d <= 128) return launch_delta_scan<16>(p, n_rows, stream);
    return launch_delta_scan<32>(p, n_rows, stream);
}

// proj: pointer to the first of the C columns; ring [slots, taps, C].  Rows that bring a single token are left out.
extern "C" int fd_conv_ring_update(const void* proj, int ld, int dtype, float* ring, const int* row_slot, const int* row_q_start,
                                   const int* row_q_len, const int* row_ctx_len, int n_rows, int C, int taps, cudaStream_t stream) {
    if (n_rows == 0 || taps <= 1) return 0;
    FD_REQUIRE(ring != nullptr && C > 0 && ld >= C && n_rows <= 65535, -2, "conv_ring_update: bad arguments");
    const dim3 grid((C + 127) / 128, n_rows);
    if (dtype == 0)
        return launch("conv_ring_update", conv_ring_update_kernel<float>, grid, dim3(128), 0, stream, dim3(1, 1, 1), (const float*)proj,
                      ld, ring, row_slot, row_q_start, row_q_len, row_ctx_len, C, taps);
    return launch("conv_ring_update", conv_ring_update_kernel<bf16>, grid, dim3(128), 0, stream, dim3(1, 1, 1), (const bf16*)proj, ld,
                  ring, row_slot, row_q_start, row_q_len, row_ctx_len, C, taps);
}
