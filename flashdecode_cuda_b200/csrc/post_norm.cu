// What stands between two sub-layers of a layer whose norms sit on the sub-layers' outputs, on the float residual
// stream; a CTA per row, all of it float, one rounding on store:
//
//   x = resid[r] + norm(y[r])            y: rows in the model's dtype, or the chosen experts' rows of a routed
//                                        feed-forward, summed here with their weights (in the order of the choices)
//   norm(y): y in G equal groups of neighbouring channels, each over its own sqrt(mean + eps), the whole times w
//   keep[r] = x                          (optional: this layer's own result, for the averages of later layers)
//   x = sum_j a[j] * history[j][r] + a[n] * x        (optional: a learned average over the layers' results so far)
//   resid[r] = x                         (optional)
//   out[j] = x  |  norm'(x)  |  x + conv(x)          (j = the row's place among the wanted rows, or r)
//
// conv is a causal convolution over time on every channel, conv(x)_t = sum_k c[k] x_(t - taps + 1 + k); a step of
// single tokens finds the earlier inputs in the sequence's state and moves it on here.  Steps with longer portions
// take a kernel of their own (stream_conv), because a row then needs its neighbours' completed streams.
//
// A group is summed by a set of whole warps (several groups one after another where there are more groups than warps):
// lane order, then warp order - no sum depends on the step's other rows.
#include "common.cuh"

namespace fd {

constexpr int PN_MAX_GROUP_SUMS = 1024;
constexpr int PN_MAX_TOP = 128;

struct PostNormParams {
    const void* y;                        // [T, H], or [pairs, H] with wts; null: nothing pending
    const float* wts; const int* pair_pos; int top;
    const float* w; int groups; float eps;
    float* resid; int write_resid;
    float* history; size_t hist_stride; int n_hist, put; const float* depth_w;
    void* out; const float* out_w; int out_groups; float out_eps;
    const float* conv_w; float* conv_state; int taps;
    const int* tok_row; const int* row_slot;
    const int* rows; int H;
};

template <int V> __device__ __forceinline__ void pn_load(const float* p, float f[V]) {
    if (V == 4) {
        const float4 v = *reinterpret_cast<const float4*>(p);
        f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
    } else {
        f[0] = *p;
    }
}
template <int V> __device__ __forceinline__ void pn_load(const __nv_bfloat16* p, float f[V]) {
    if (V == 4) {
        const uint2 v = *reinterpret_cast<const uint2*>(p);
        const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&v.x), b = *reinterpret_cast<const __nv_bfloat162*>(&v.y);
        f[0] = __low2float(a); f[1] = __high2float(a); f[2] = __low2float(b); f[3] = __high2float(b);
    } else {
        f[0] = __bfloat162float(*p);
    }
}
template <int V> __device__ __forceinline__ void pn_store(float* p, const float f[V]) {
    if (V == 4) *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
    else *p = f[0];
}
template <int V> __device__ __forceinline__ void pn_store(__nv_bfloat16* p, const float f[V]) {
    if (V == 4) {
        uint2 v;
        __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&v);
        h[0] = __floats2bfloat162_rn(f[0], f[1]);
        h[1] = __floats2bfloat162_rn(f[2], f[3]);
        *reinterpret_cast<uint2*>(p) = v;
    } else {
        *p = __float2bfloat16_rn(f[0]);
    }
}

// How the CTA's warps share `groups` groups of `gsize` channels: sets of wpg warps, set s takes groups s, s + sets, ...
struct Sets {
    int wpg, sets, set, lane;             // lane: this thread's place in its set
    __device__ Sets(int groups) {
        const int nw = blockDim.x >> 5, warp = threadIdx.x >> 5;
        wpg = groups < nw ? nw / groups : 1;
        sets = nw / wpg;
        set = warp / wpg;
        lane = (warp - set * wpg) * 32 + (threadIdx.x & 31);
    }
};

// rstd[g] for every group of the row in `row` (shared memory, written by the threads that read it here).
template <int V>
__device__ __forceinline__ void group_rstd(const float* row, int H, int groups, float eps, const Sets& s, float* part, float* rstd) {
    const int gsize = H / groups;
    const int warp = threadIdx.x >> 5;
    for (int g = s.set; g < groups && s.set < s.sets; g += s.sets) {
        float ss = 0.f;
        for (int i = s.lane * V; i < gsize; i += s.wpg * 32 * V) {
#pragma unroll
            for (int e = 0; e < V; ++e) { const float v = row[g * gsize + i + e]; ss = fmaf(v, v, ss); }
        }
        ss = warp_sum(ss);
        // one warp per set: its group is finished; several: their sums meet below (groups <= warps then: one round)
        if ((threadIdx.x & 31) == 0) {
            if (s.wpg == 1) rstd[g] = rsqrtf(ss / (float)gsize + eps);
            else part[warp] = ss;
        }
    }
    __syncthreads();
    if (s.wpg > 1) {
        for (int g = threadIdx.x; g < groups; g += blockDim.x) {
            float ss = 0.f;
            for (int k = 0; k < s.wpg; ++k) ss += part[g * s.wpg + k];
            rstd[g] = rsqrtf(ss / (float)gsize + eps);
        }
        __syncthreads();
    }
}

template <typename TY, typename TO, int V>
__global__ void __launch_bounds__(256)
post_norm_kernel(const PostNormParams p) {
    extern __shared__ __align__(16) float pn_row[];            // [H]
    __shared__ float part[8];
    __shared__ float rstd[PN_MAX_GROUP_SUMS];
    __shared__ int pos_s[PN_MAX_TOP];
    __shared__ float wts_s[PN_MAX_TOP];
    const int j = blockIdx.x;
    const int r = p.rows != nullptr ? p.rows[j] : j;
    const int H = p.H;
    float* xr = p.resid + (size_t)r * H;
    // The elementwise passes walk the row by the sets of the norm that made it (a thread always returns to its own channels)
    const int groups = p.y != nullptr ? p.groups : (p.out_w != nullptr ? p.out_groups : 1);
    const int gsize = H / groups;
    const Sets s(groups);
    const bool active = s.set < s.sets;
    if (p.y != nullptr) {
        const TY* y = static_cast<const TY*>(p.y);
        if (p.wts != nullptr) {
            for (int c = threadIdx.x; c < p.top; c += blockDim.x) {
                pos_s[c] = p.pair_pos[(size_t)r * p.top + c];
                wts_s[c] = p.wts[(size_t)r * p.top + c];
            }
            __syncthreads();
        }
        for (int g = s.set; g < groups && active; g += s.sets)
            for (int i = s.lane * V; i < gsize; i += s.wpg * 32 * V) {
                const int c = g * gsize + i;
                float v[V];
                if (p.wts != nullptr) {
#pragma unroll
                    for (int e = 0; e < V; ++e) v[e] = 0.f;
#pragma unroll 4
                    for (int k = 0; k < p.top; ++k) {
                        const int pos = pos_s[k];
                        if (pos < 0) continue;
                        float f[V];
                        pn_load<V>(y + (size_t)pos * H + c, f);
#pragma unroll
                        for (int e = 0; e < V; ++e) v[e] = fmaf(wts_s[k], f[e], v[e]);
                    }
                } else {
                    pn_load<V>(y + (size_t)r * H + c, v);
                }
                pn_store<V>(pn_row + c, v);
            }
        group_rstd<V>(pn_row, H, groups, p.eps, s, part, rstd);
    }
    int slot = -1;
    if (p.conv_w != nullptr) slot = p.row_slot[p.tok_row[r]];
    TO* out = static_cast<TO*>(p.out);
    for (int g = s.set; g < groups && active; g += s.sets) {
        const float rs = p.y != nullptr ? rstd[g] : 0.f;
        for (int i = s.lane * V; i < gsize; i += s.wpg * 32 * V) {
            const int c = g * gsize + i;
            float x[V];
            pn_load<V>(xr + c, x);
            if (p.y != nullptr) {
                float v[V], w[V];
                pn_load<V>(pn_row + c, v);
                pn_load<V>(p.w + c, w);
#pragma unroll
                for (int e = 0; e < V; ++e) x[e] = fmaf(v[e] * rs, w[e], x[e]);
            }
            if (p.put >= 0) pn_store<V>(p.history + p.put * p.hist_stride + (size_t)r * H + c, x);
            if (p.depth_w != nullptr) {
                float a[V];
#pragma unroll
                for (int e = 0; e < V; ++e) a[e] = 0.f;
#pragma unroll 4
                for (int k = 0; k < p.n_hist; ++k) {
                    float f[V];
                    pn_load<V>(p.history + k * p.hist_stride + (size_t)r * H + c, f);
                    const float dw = p.depth_w[k];
#pragma unroll
                    for (int e = 0; e < V; ++e) a[e] = fmaf(dw, f[e], a[e]);
                }
                const float dw = p.depth_w[p.n_hist];
#pragma unroll
                for (int e = 0; e < V; ++e) x[e] = fmaf(dw, x[e], a[e]);
            }
            if (p.write_resid) pn_store<V>(xr + c, x);
            if (p.out_w != nullptr) {
                pn_store<V>(pn_row + c, x);
                continue;
            }
            if (p.conv_w != nullptr) {
                // the taps in the order k = 0, 1, ... (oldest input first), then the input itself
                const int hist = p.taps - 1;
                float acc[V];
#pragma unroll
                for (int e = 0; e < V; ++e) acc[e] = 0.f;
                if (slot >= 0 && p.conv_state != nullptr) {
                    float* st = p.conv_state + (size_t)slot * hist * H + c;
                    for (int k = 0; k < hist; ++k) {
                        float f[V], w[V];
                        pn_load<V>(st + (size_t)k * H, f);
                        pn_load<V>(p.conv_w + (size_t)k * H + c, w);
#pragma unroll
                        for (int e = 0; e < V; ++e) acc[e] = fmaf(w[e], f[e], acc[e]);
                        if (k > 0) pn_store<V>(st + (size_t)(k - 1) * H, f);
                    }
                    if (hist > 0) pn_store<V>(st + (size_t)(hist - 1) * H, x);
                }
                float w[V];
                pn_load<V>(p.conv_w + (size_t)hist * H + c, w);
#pragma unroll
                for (int e = 0; e < V; ++e) x[e] += fmaf(w[e], x[e], acc[e]);
            }
            if (out != nullptr) pn_store<V>(out + (size_t)j * H + c, x);
        }
    }
    if (p.out_w == nullptr) return;
    const Sets so(p.out_groups);
    __syncthreads();                      // the sets of the two norms may differ: the whole row is in shared memory now
    group_rstd<V>(pn_row, H, p.out_groups, p.out_eps, so, part, rstd);
    const int osize = H / p.out_groups;
    for (int g = so.set; g < p.out_groups && so.set < so.sets; g += so.sets)
        for (int i = so.lane * V; i < osize; i += so.wpg * 32 * V) {
            const int c = g * osize + i;
            float x[V], w[V];
            pn_load<V>(pn_row + c, x);
            pn_load<V>(p.out_w + c, w);
#pragma unroll
            for (int e = 0; e < V; ++e) x[e] = x[e] * rstd[g] * w[e];
            pn_store<V>(out + (size_t)j * H + c, x);
        }
}

// out[t] = x[t] + conv(x)[t] for steps with longer portions: a thread takes V adjacent channels of SC_TPC consecutive
// tokens; inputs before the row's first token of the step come from the sequence's state (zeros for a padding row).
constexpr int SC_TPC = 8, SC_THREADS = 128;

template <typename TO, int V>
__global__ void __launch_bounds__(SC_THREADS)
stream_conv_kernel(const float* __restrict__ x, const float* __restrict__ w, const float* __restrict__ state, TO* __restrict__ out,
                   const int* __restrict__ tok_row, const int* __restrict__ row_slot, const int* __restrict__ row_q_start, int T,
                   int H, int taps) {
    const int c = (blockIdx.x * SC_THREADS + threadIdx.x) * V;
    if (c >= H) return;
    const int hist = taps - 1;
    const int t1 = min(T, (int)(blockIdx.y + 1) * SC_TPC);
#pragma unroll 2
    for (int t = blockIdx.y * SC_TPC; t < t1; ++t) {
        const int row = tok_row[t];
        const int i = t - row_q_start[row];
        const int slot = row_slot[row];
        float acc[V];
#pragma unroll
        for (int e = 0; e < V; ++e) acc[e] = 0.f;
#pragma unroll 4
        for (int k = 0; k < hist; ++k) {
            const int back = hist - k;                          // the k-th tap reads the input `back` steps ago
            float f[V], wk[V];
#pragma unroll
            for (int e = 0; e < V; ++e) f[e] = 0.f;
            if (i >= back) pn_load<V>(x + (size_t)(t - back) * H + c, f);
            else if (slot >= 0 && state != nullptr) pn_load<V>(state + ((size_t)slot * hist + (hist + i - back)) * H + c, f);
            pn_load<V>(w + (size_t)k * H + c, wk);
#pragma unroll
            for (int e = 0; e < V; ++e) acc[e] = fmaf(wk[e], f[e], acc[e]);
        }
        float f[V], wk[V];
        pn_load<V>(x + (size_t)t * H + c, f);
        pn_load<V>(w + (size_t)hist * H + c, wk);
#pragma unroll
        for (int e = 0; e < V; ++e) f[e] += fmaf(wk[e], f[e], acc[e]);
        pn_store<V>(out + (size_t)t * H + c, f);
    }
}

}  // namespace fd

using namespace fd;
typedef __nv_bfloat16 bf16;

static bool pn_al(const void* p) { return (uintptr_t)p % 16 == 0; }

template <typename TY, typename TO>
static int launch_post_norm(const PostNormParams& p, int n_out, bool vec, int threads, cudaStream_t stream) {
    const size_t smem = (size_t)p.H * sizeof(float);
    if (vec) return launch("post_norm", post_norm_kernel<TY, TO, 4>, dim3(n_out), dim3(threads), smem, stream, dim3(1, 1, 1), p);
    return launch("post_norm", post_norm_kernel<TY, TO, 1>, dim3(n_out), dim3(threads), smem, stream, dim3(1, 1, 1), p);
}

// y_dtype / out_dtype: 0 float32, 1 bfloat16.  y null: nothing pending.  wts [T, top] and pair_pos [T * top] with a routed
// feed-forward's rows in y.  history [slots][hist_stride]: n_hist of them averaged with depth_w [n_hist + 1] when that is
// given; put >= 0: the completed stream's slot.  out_w: out is the stream normed in out_groups groups.  conv_w [taps, H]:
// out is the stream plus its convolution, conv_state [slots, taps - 1, H] moved on.  rows: the rows that out lists.
extern "C" int fd_post_norm(const void* y, int y_dtype, const float* wts, const int* pair_pos, int top, const float* w,
                            int groups, float eps, float* resid, int write_resid, float* history, long long hist_stride,
                            int n_hist, int put, const float* depth_w, void* out, int out_dtype, const float* out_w,
                            int out_groups, float out_eps, const float* conv_w, float* conv_state, int taps,
                            const int* tok_row, const int* row_slot, const int* rows, int n_out, int H, cudaStream_t stream) {
    if (n_out == 0) return 0;
    FD_REQUIRE(H > 0 && H <= 11000, -2, "post_norm: rows of %d (at most 11000)", H);
    FD_REQUIRE(groups > 0 && H % groups == 0 && groups <= PN_MAX_GROUP_SUMS && out_groups > 0 && H % out_groups == 0 &&
               out_groups <= PN_MAX_GROUP_SUMS, -2, "post_norm: %d and %d groups of %d channels", groups, out_groups, H);
    FD_REQUIRE(y == nullptr || w != nullptr, -2, "post_norm: a pending output needs its norm weight");
    FD_REQUIRE(wts == nullptr || (top > 0 && top <= PN_MAX_TOP && pair_pos != nullptr), -2, "post_norm: %d choices", top);
    FD_REQUIRE((put < 0 && depth_w == nullptr) || history != nullptr, -2, "post_norm: no history memory");
    FD_REQUIRE(conv_w == nullptr || (taps >= 1 && tok_row && row_slot && rows == nullptr && out_w == nullptr && (taps == 1 || conv_state)), -2,
               "post_norm: bad convolution arguments");
    FD_REQUIRE(out_w == nullptr || out != nullptr, -2, "post_norm: nowhere to put the normed rows");
    PostNormParams p;
    p.y = y; p.wts = wts; p.pair_pos = pair_pos; p.top = top; p.w = w; p.groups = groups; p.eps = eps;
    p.resid = resid; p.write_resid = write_resid;
    p.history = history; p.hist_stride = (size_t)hist_stride; p.n_hist = n_hist; p.put = put; p.depth_w = depth_w;
    p.out = out; p.out_w = out_w; p.out_groups = out_groups; p.out_eps = out_eps;
    p.conv_w = conv_w; p.conv_state = conv_state; p.taps = taps; p.tok_row = tok_row; p.row_slot = row_slot;
    p.rows = rows; p.H = H;
    const int g = y != nullptr ? groups : (out_w != nullptr ? out_groups : 1);
    const bool vec = (H / g) % 4 == 0 && (H / out_groups) % 4 == 0 && pn_al(y) && pn_al(w) && pn_al(resid) && pn_al(history) &&
                     hist_stride % 4 == 0 && pn_al(out) && pn_al(out_w) && pn_al(conv_w) && pn_al(conv_state);
    int warps = H >= 1024 ? 8 : 4;
    if (g <= warps) warps = warps / g * g;
    const int threads = warps * 32;
    if (y_dtype == 0) {
        if (out_dtype == 0) return launch_post_norm<float, float>(p, n_out, vec, threads, stream);
        return launch_post_norm<float, bf16>(p, n_out, vec, threads, stream);
    }
    if (out_dtype == 0) return launch_post_norm<bf16, float>(p, n_out, vec, threads, stream);
    return launch_post_norm<bf16, bf16>(p, n_out, vec, threads, stream);
}

// x [T, H] float, w [taps, H] float, state [slots, taps - 1, H] float (null with one tap), out [T, H] of out_dtype.
extern "C" int fd_stream_conv(const float* x, const float* w, const float* state, void* out, int out_dtype, const int* tok_row,
                              const int* row_slot, const int* row_q_start, int T, int H, int taps, cudaStream_t stream) {
    if (T == 0) return 0;
    FD_REQUIRE(H > 0 && taps >= 1 && (taps == 1 || state != nullptr), -2, "stream_conv: %d taps on %d channels", taps, H);
    const bool vec = H % 4 == 0 && pn_al(x) && pn_al(w) && pn_al(state) && pn_al(out);
    const int V = vec ? 4 : 1;
    const dim3 grid((H + SC_THREADS * V - 1) / (SC_THREADS * V), (T + SC_TPC - 1) / SC_TPC);
    FD_REQUIRE(grid.y <= 65535, -2, "stream_conv: %d tokens are too many", T);
    const dim3 block(SC_THREADS), one(1, 1, 1);
#define FD_STREAM_CONV(TO, VV)                                                                                             \
    launch("stream_conv", stream_conv_kernel<TO, VV>, grid, block, 0, stream, one, x, w, state, (TO*)out, tok_row, row_slot, \
           row_q_start, T, H, taps)
    if (out_dtype == 0) return vec ? FD_STREAM_CONV(float, 4) : FD_STREAM_CONV(float, 1);
    return vec ? FD_STREAM_CONV(bf16, 4) : FD_STREAM_CONV(bf16, 1);
#undef FD_STREAM_CONV
}
