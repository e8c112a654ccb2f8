// Short causal convolution over time of one channel, for the kernels that prepare a recurrence's inputs.
//
// y[t] = bias + sum_k w[k] u[t - (taps - 1) + k], zeros before the sequence's start.  The values of earlier steps come from
// the sequence's ring, float [slots, taps, C]: the value of position p lies at place p % taps.  A ring of `taps` places
// (one more than a token needs) lets a step of single tokens write its own value, at the place of the value that no
// one reads any more, while other CTAs still read the earlier ones.  A place whose position would lie before the start is
// never read, so a slot's old contents do not matter.  The taps are added in the order k = 0, 1, ... after the bias,
// from the same values wherever they come from: how a prompt is cut changes no bit.
#pragma once

#include "common.cuh"

namespace fd {

constexpr int SC_TOK = 8;             // tokens of a tile at most
constexpr int SC_TAPS = 4;            // more taps than this take the plain loop

struct ConvMeta {                     // what the tokens of a tile need to know, in shared memory
    int slot[SC_TOK], i[SC_TOK], pos[SC_TOK], single[SC_TOK];     // slot -1: padding row; i: place in its row's new tokens
    int one_row;                      // the tile has several tokens, all of one row (and none is padding)
};

// threads 0 .. nt - 1 fill the tile's entries; the caller synchronises
__device__ __forceinline__ void conv_meta(ConvMeta& m, int t0, int nt, const int* tok_row, const int* tok_pos,
                                          const int* row_slot, const int* row_q_start, const int* row_q_len) {
    if (threadIdx.x < nt) {
        const int t = t0 + threadIdx.x, r = tok_row[t];
        m.slot[threadIdx.x] = row_slot[r];
        m.i[threadIdx.x] = t - row_q_start[r];
        m.pos[threadIdx.x] = tok_pos[t];
        m.single[threadIdx.x] = row_q_len[r] == 1;
        if (threadIdx.x == 0) m.one_row = nt > 1 && m.slot[0] >= 0 && tok_row[t0 + nt - 1] == r;
    }
}

constexpr int SC_VALS = SC_TOK + SC_TAPS - 1;      // values the taps of a tile's tokens see; place SC_TAPS - 1 + j is token t0 + j

// The values of a tile as they lie in the step's rows, before anything is known of its tokens: so the loads pass beside those of the
// tile's ConvMeta.  Those before the row's first token are wrong yet; conv_channel puts the ring's in their place.
template <typename T>
__device__ __forceinline__ void conv_load(const T* __restrict__ col, int ld, int t0, int nt, float u[SC_VALS]) {
#pragma unroll
    for (int e = 0; e < SC_VALS; ++e) {
        const int j = e - (SC_TAPS - 1);
        u[e] = j < nt && t0 + j >= 0 ? to_float(col[(size_t)(t0 + j) * ld]) : 0.f;
    }
}

// The nt <= SC_TOK tokens from t0 on of channel c of C (column `col` points at it in token 0's row, rows of ld elements; u: what
// conv_load made of it, looked at only in tiles of one row);
// rows that bring a single token leave their value in the ring when `keep` is set.
template <typename T>
__device__ __forceinline__ void conv_channel(const T* __restrict__ col, int ld, const float* __restrict__ w, float bias, int taps,
                                             float* ring, int c, int C, const ConvMeta& m, int t0, int nt, bool keep,
                                             float u[SC_VALS], float y[SC_TOK]) {
    float wk[SC_TAPS];
#pragma unroll
    for (int k = 0; k < SC_TAPS; ++k) wk[k] = k < taps ? w[k] : 0.f;
    if (m.one_row && !m.single[0] && taps <= SC_TAPS) {
        // consecutive tokens of one row
        const int i0 = m.i[0], pos0 = m.pos[0];
        const float* rg = ring + (size_t)m.slot[0] * taps * C + c;
        if (i0 < taps - 1) {
#pragma unroll
            for (int e = 0; e < SC_TAPS - 1; ++e) {
                const int j = e - (SC_TAPS - 1);
                if (i0 + j < 0) u[e] = -j < taps && pos0 + j >= 0 ? rg[(size_t)((pos0 + j) % taps) * C] : 0.f;
            }
        }
        // the weights moved to the end, so that tap k of `taps` meets the place it would meet below
        float we[SC_TAPS];
#pragma unroll
        for (int e = 0; e < SC_TAPS; ++e) {
            we[e] = 0.f;
#pragma unroll
            for (int k = 0; k < SC_TAPS; ++k) if (k < taps && SC_TAPS - taps + k == e) we[e] = wk[k];
        }
#pragma unroll
        for (int tt = 0; tt < SC_TOK; ++tt) {
            float a = bias;
#pragma unroll
            for (int e = 0; e < SC_TAPS; ++e) if (e >= SC_TAPS - taps) a = fmaf(we[e], u[tt + e], a);
            y[tt] = tt < nt ? a : 0.f;
        }
        return;
    }
#pragma unroll
    for (int tt = 0; tt < SC_TOK; ++tt) {
        y[tt] = 0.f;
        if (tt >= nt || m.slot[tt] < 0) continue;
        const int t = t0 + tt, i = m.i[tt], pos = m.pos[tt];
        float* rg = ring + (size_t)m.slot[tt] * taps * C + c;
        auto value = [&](int back) -> float {
            if (back <= i) return to_float(col[(size_t)(t - back) * ld]);
            return back <= pos ? rg[(size_t)((pos - back) % taps) * C] : 0.f;
        };
        float a = bias;
        const float cur = value(0);
        if (taps <= SC_TAPS) {
            float x[SC_TAPS];
#pragma unroll
            for (int k = 0; k < SC_TAPS; ++k) x[k] = k < taps - 1 ? value(taps - 1 - k) : (k == taps - 1 ? cur : 0.f);
#pragma unroll
            for (int k = 0; k < SC_TAPS; ++k) if (k < taps) a = fmaf(wk[k], x[k], a);
        } else {
            for (int k = 0; k < taps; ++k) a = fmaf(w[k], value(taps - 1 - k), a);
        }
        if (keep && taps > 1 && m.single[tt]) rg[(size_t)(pos % taps) * C] = cur;
        y[tt] = a;
    }
}

// z sigmoid(z); behind bfloat16 projections with the special function unit's exponential and reciprocal (a few units in the
// last place of a float)
template <typename T> __device__ __forceinline__ float sc_silu(float z) { return z / (1.f + expf(-z)); }
template <> __device__ __forceinline__ float sc_silu<__nv_bfloat16>(float z) { return z * __frcp_rn(1.f + __expf(-z)); }
__device__ __forceinline__ float sc_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float sc_softplus(float z) { return z > 0.f ? z + log1pf(expf(-z)) : log1pf(expf(z)); }

}  // namespace fd
