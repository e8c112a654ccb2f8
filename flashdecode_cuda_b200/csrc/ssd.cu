// What stands around the state-space recurrence of a Mamba-2 mixer (linear_scan.cu, mode 3):
//
//  * ssd_prepare: x, B and C - neighbouring columns of the packed projection - pass a causal convolution over time per channel
//    with bias (short_conv.cuh) and silu, and are left as floats [T, C]; per token and head the step size dt =
//    softplus(raw + bias) and the decay exp(-exp(A_h) dt), floats [T, H, 2];
//  * ssd_gate_norm: (y + D_h x) * silu(z), RMS-normed in equal parts, times a weight, times a constant.
//
// Everything is float from the projection on, and rounded once on the way to the output product.
#include <math.h>

#include "short_conv.cuh"

namespace fd {

constexpr int SSD_THREADS = 128;

template <typename T>
__global__ void __launch_bounds__(SSD_THREADS)
ssd_prepare_kernel(const T* __restrict__ proj, int ld, int col, int C, int dt_col, const float* __restrict__ conv_w,
                   const float* __restrict__ conv_b, float* ring, int taps, int keep, const float* __restrict__ dt_bias,
                   const float* __restrict__ A_log, float* __restrict__ xbc, float* __restrict__ step, const int* __restrict__ tok_row,
                   const int* __restrict__ tok_pos, const int* __restrict__ row_slot, const int* __restrict__ row_q_start,
                   const int* __restrict__ row_q_len, int n_tok, int H, int tpc) {
    __shared__ ConvMeta meta;
    const int t0 = blockIdx.x * tpc, nt = min(tpc, n_tok - t0);
    conv_meta(meta, t0, nt, tok_row, tok_pos, row_slot, row_q_start, row_q_len);
    __syncthreads();
    if (blockIdx.y == gridDim.y - 1) {                       // step sizes and decays
        for (int e = threadIdx.x; e < nt * H; e += blockDim.x) {
            const int tt = e / H, h = e - tt * H;
            const float dt = sc_softplus(to_float(proj[(size_t)(t0 + tt) * ld + dt_col + h]) + dt_bias[h]);
            *reinterpret_cast<float2*>(step + ((size_t)(t0 + tt) * H + h) * 2) = make_float2(dt, expf(-expf(A_log[h]) * dt));
        }
        return;
    }
    const int c = blockIdx.y * SSD_THREADS + threadIdx.x;
    if (c >= C) return;
    float y[SC_TOK];
    conv_channel<T>(proj + col + c, ld, conv_w + (size_t)c * taps, conv_b[c], taps, ring, c, C, meta, t0, nt, keep, y);
#pragma unroll
    for (int tt = 0; tt < SC_TOK; ++tt)
        if (tt < nt && meta.slot[tt] >= 0) xbc[(size_t)(t0 + tt) * C + c] = sc_silu(y[tt]);
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
    for (int j = threadIdx.x; j < part; j += blockDim.x) {
        const int c = c0 + j;
        const float gate = to_float(z[t * ldz + c]);
        const float v = fmaf(D[c / dv], xbc[t * ldx + c], y[t * inner + c]) * (gate / (1.f + expf(-gate)));
        g_s[j] = v;
        ss = fmaf(v, v, ss);
    }
    const float rs = scale / sqrtf(block_sum(ss, red) / (float)part + eps);
    for (int j = threadIdx.x; j < part; j += blockDim.x) out[t * ld_out + c0 + j] = from_float<T>(g_s[j] * rs * w[c0 + j]);
}

}  // namespace fd

using namespace fd;
typedef __nv_bfloat16 bf16;

// proj [T, ld] of `dtype` (0 float32, 1 bfloat16): x, B, C are the C columns from `col` on, the raw step sizes the H columns from
// dt_col on.  conv_w [C, taps], conv_b [C]; ring [slots, taps, C] (unused when taps == 1).  xbc [T, C], step [T, H, 2] float.
// keep: rows of a single token leave their values in the ring here; longer rows need fd_conv_ring_update.
extern "C" int fd_ssd_prepare(const void* proj, int ld, int dtype, int col, int C, int dt_col, const float* conv_w, const float* conv_b,
                              float* ring, int taps, int keep, const float* dt_bias, const float* A_log, float* xbc, float* step,
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
                      col, C, dt_col, conv_w, conv_b, ring, taps, keep, dt_bias, A_log, xbc, step, tok_row, tok_pos, row_slot,
                      row_q_start, row_q_len, T, H, tpc);
    return launch("ssd_prepare", ssd_prepare_kernel<bf16>, grid, dim3(SSD_THREADS), 0, stream, dim3(1, 1, 1), (const bf16*)proj, ld, col,
                  C, dt_col, conv_w, conv_b, ring, taps, keep, dt_bias, A_log, xbc, step, tok_row, tok_pos, row_slot, row_q_start,
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
