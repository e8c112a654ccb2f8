// One small matrix product per head:
//
//     out[t, h, n] = sum_k a[t, h, k] * w[h, n, k]        a [T, heads, K], w [heads, N, K], out [T, heads, N]
//
// The heads of a and of out may lie in longer places (strides a_hs, o_hs); out may be multiplied by sigmoid(gate[t, h, n]).
// rope_heads turns a part of every head at the token's position (dimension 2i paired with 2i + 1), in place or into
// another array: the rotated part of a latent attention's queries, which passes its per-head product by.
//
// (a per-head change of basis: a latent-attention mixer folds every head's key
// expansion into its queries this way, and expands every head's attended latent
// into values).  CUDA cores, float accumulation, k ascending in one fmaf chain
// per output, so no bit of a row depends on what else is in the step; float or
// bfloat16 storage.  A CTA takes 32 rows x 64 columns of one head.
#include "common.cuh"

namespace fd {

constexpr int HG_MT = 32, HG_NT = 64, HG_KT = 32, HG_THREADS = 256;

// Where the heads lie: row and head strides of a, of out and of the gate (null: none), in elements.
struct HeadStrides {
    int a_ld, a_hs, o_ld, o_hs, g_ld, g_hs;
};

__device__ __forceinline__ float hg_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }

template <typename T>
__global__ void __launch_bounds__(HG_THREADS)
head_gemm_kernel(const T* __restrict__ a, const T* __restrict__ w, T* __restrict__ out, const T* __restrict__ gate,
                 const HeadStrides st, int T_rows, int heads, int N, int K) {
    __shared__ float a_s[HG_MT][HG_KT + 1];
    __shared__ float b_s[HG_NT][HG_KT + 1];
    const int h = blockIdx.z;
    const int m0 = blockIdx.y * HG_MT, n0 = blockIdx.x * HG_NT;
    const int tid = threadIdx.x;
    const T* ah = a + (size_t)h * st.a_hs;
    const T* wh = w + (size_t)h * N * K;
    const size_t lda = st.a_ld, ldo = st.o_ld;
    const int ty = tid / 16, tx = tid % 16;          // rows 2 ty, 2 ty + 1; columns tx + 16 j
    float acc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
    for (int k0 = 0; k0 < K; k0 += HG_KT) {
        for (int i = tid; i < HG_MT * HG_KT; i += HG_THREADS) {
            const int r = i / HG_KT, kk = i - r * HG_KT;
            a_s[r][kk] = (m0 + r < T_rows && k0 + kk < K) ? to_float(ah[(size_t)(m0 + r) * lda + k0 + kk]) : 0.f;
        }
        for (int i = tid; i < HG_NT * HG_KT; i += HG_THREADS) {
            const int c = i / HG_KT, kk = i - c * HG_KT;
            b_s[c][kk] = (n0 + c < N && k0 + kk < K) ? to_float(wh[(size_t)(n0 + c) * K + k0 + kk]) : 0.f;
        }
        __syncthreads();
#pragma unroll 8
        for (int kk = 0; kk < HG_KT; ++kk) {
            const float a0 = a_s[2 * ty][kk], a1 = a_s[2 * ty + 1][kk];
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const float b = b_s[tx + 16 * j][kk];
                acc[0][j] = fmaf(a0, b, acc[0][j]);
                acc[1][j] = fmaf(a1, b, acc[1][j]);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const int r = m0 + 2 * ty + i;
        if (r >= T_rows) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int c = n0 + tx + 16 * j;
            if (c >= N) continue;
            float v = acc[i][j];
            if (gate != nullptr) v *= hg_sigmoid(to_float(gate[(size_t)r * st.g_ld + (size_t)h * st.g_hs + c]));
            out[(size_t)r * ldo + (size_t)h * st.o_hs + c] = from_float<T>(v);
        }
    }
}

// A rotated part of every head: dst[t, h, 0 .. places) = rot(src[t, h, 0 .. nr)), zeros after it; src and dst may be the
// same memory (places == nr then).  Pointers at the first rotated dimension of the first head.
template <typename T>
struct RopePart {
    const T* src; int s_ld, s_hs;
    T* dst; int d_ld, d_hs;
    const float* cos_t; const float* sin_t; int table_len;
    const int* tok_pos;
    int heads, nr, places;
    int* status;
};

template <typename T>
__device__ __forceinline__ void rope_token(const RopePart<T>& r, int t) {
    const int pos = r.tok_pos[t];
    if (pos < 0 || pos >= r.table_len) {
        if (threadIdx.x == 0) set_status(r.status, STATUS_BAD_POSITION);
        return;
    }
    const int half = r.nr >> 1, pp = r.places >> 1;
    const float* c = r.cos_t + (size_t)pos * half;
    const float* s = r.sin_t + (size_t)pos * half;
    for (int e = threadIdx.x; e < r.heads * pp; e += blockDim.x) {
        const int h = e / pp, i = e - h * pp;
        T a = from_float<T>(0.f), b = a;
        if (i < half) {
            const T* x = r.src + (size_t)t * r.s_ld + (size_t)h * r.s_hs + 2 * i;
            const float u = to_float(x[0]), v = to_float(x[1]);
            a = from_float<T>(u * c[i] - v * s[i]);
            b = from_float<T>(v * c[i] + u * s[i]);
        }
        T* o = r.dst + (size_t)t * r.d_ld + (size_t)h * r.d_hs + 2 * i;
        o[0] = a;
        o[1] = b;
    }
}

template <typename T>
__global__ void rope_heads_kernel(const RopePart<T> r) { rope_token<T>(r, blockIdx.x); }

// Steps of few rows in bfloat16 (K a multiple of 8): a warp per output column (head, n) reads that row of w once in
// 16-byte pieces and takes it against every row of a; eight warps per CTA.  The CTAs behind those (rope.heads > 0: one per row)
// turn the heads' rotated parts.
template <int MAXT>
__global__ void __launch_bounds__(256)
head_gemv_kernel(const __nv_bfloat16* __restrict__ a, const __nv_bfloat16* __restrict__ w, __nv_bfloat16* __restrict__ out,
                 const __nv_bfloat16* __restrict__ gate, const HeadStrides st, const RopePart<__nv_bfloat16> rope, int n_product_ctas,
                 int T_rows, int heads, int N, int K) {
    if ((int)blockIdx.x >= n_product_ctas) {
        rope_token<__nv_bfloat16>(rope, blockIdx.x - n_product_ctas);
        return;
    }
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int col = blockIdx.x * 8 + warp;
    if (col >= heads * N) return;
    const int h = col / N;
    const __nv_bfloat16* wr = w + (size_t)col * K;
    const __nv_bfloat16* ah = a + (size_t)h * st.a_hs;
    const size_t lda = st.a_ld;
    const int n = col - h * N;
    float acc[MAXT];
#pragma unroll
    for (int t = 0; t < MAXT; ++t) acc[t] = 0.f;
    for (int c = lane * 8; c < K; c += 256) {
        const uint4 wv = *reinterpret_cast<const uint4*>(wr + c);
        const __nv_bfloat162* w2 = reinterpret_cast<const __nv_bfloat162*>(&wv);
#pragma unroll
        for (int t = 0; t < MAXT; ++t) {
            if (t < T_rows) {
                const uint4 av = *reinterpret_cast<const uint4*>(ah + t * lda + c);
                const __nv_bfloat162* a2 = reinterpret_cast<const __nv_bfloat162*>(&av);
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    acc[t] = fmaf(__low2float(w2[e]), __low2float(a2[e]), acc[t]);
                    acc[t] = fmaf(__high2float(w2[e]), __high2float(a2[e]), acc[t]);
                }
            }
        }
    }
#pragma unroll
    for (int t = 0; t < MAXT; ++t) {
        if (t < T_rows) {
            float v = warp_sum(acc[t]);
            if (lane == 0) {
                if (gate != nullptr) v *= hg_sigmoid(__bfloat162float(gate[(size_t)t * st.g_ld + (size_t)h * st.g_hs + n]));
                out[(size_t)t * st.o_ld + (size_t)h * st.o_hs + n] = __float2bfloat16_rn(v);
            }
        }
    }
}

}  // namespace fd

using namespace fd;

template <typename T>
static int launch_rope(const RopePart<T>& r, int n_tok, cudaStream_t stream) {
    const int work = r.heads * r.places / 2;
    const dim3 block(work >= 256 ? 256 : (work + 31) / 32 * 32);
    return launch("rope_heads", rope_heads_kernel<T>, dim3(n_tok), block, 0, stream, dim3(1, 1, 1), r);
}

template <typename T>
static RopePart<T> rope_part(const void* src, int s_ld, int s_hs, void* dst, int d_ld, int d_hs, const float* cos_t,
                             const float* sin_t, int table_len, const int* tok_pos, int heads, int nr, int places, int* status) {
    RopePart<T> r;
    r.src = static_cast<const T*>(src); r.s_ld = s_ld; r.s_hs = s_hs;
    r.dst = static_cast<T*>(dst); r.d_ld = d_ld; r.d_hs = d_hs;
    r.cos_t = cos_t; r.sin_t = sin_t; r.table_len = table_len; r.tok_pos = tok_pos;
    r.heads = heads; r.nr = nr; r.places = places; r.status = status;
    return r;
}

// a: [T, heads, K] with row stride a_ld and head stride a_hs (elements); out likewise; gate (or null): sigmoid(gate) times out.
// nr > 0: the nr dimensions at a + r_src of every head are turned (cos_t / sin_t [table_len, nr / 2]) into the r_places at
// out + r_dst, in the same launch where the product is the one for few rows.
extern "C" int fd_head_gemm(const void* a, int a_ld, int a_hs, const void* w, void* out, int o_ld, int o_hs, const void* gate,
                            int g_ld, int g_hs, int dtype, int T, int heads, int N, int K, int r_src, int r_dst, int nr,
                            int r_places, const float* cos_t, const float* sin_t, int table_len, const int* tok_pos, int* status,
                            cudaStream_t stream) {
    if (T == 0) return 0;
    FD_REQUIRE(heads > 0 && heads <= 65535 && N > 0 && K > 0, -2, "head_gemm: %d heads, N %d, K %d", heads, N, K);
    FD_REQUIRE(nr >= 0 && nr % 2 == 0 && (nr == 0 || (r_places >= nr && r_places % 2 == 0 && cos_t && sin_t && tok_pos)), -2,
               "head_gemm: a rotated part of %d dimensions in %d places", nr, r_places);
    typedef __nv_bfloat16 bf16;
    const HeadStrides st = {a_ld, a_hs, o_ld, o_hs, g_ld, g_hs};
    const dim3 one(1, 1, 1);
    if (dtype == 1 && T <= 16 && K % 8 == 0 && a_ld % 8 == 0 && a_hs % 8 == 0 && (uintptr_t)a % 16 == 0 && (uintptr_t)w % 16 == 0) {
        const int ctas = (int)((heads * (long long)N + 7) / 8);
        const RopePart<bf16> rp = rope_part<bf16>((const bf16*)a + r_src, a_ld, a_hs, (bf16*)out + r_dst, o_ld, o_hs, cos_t, sin_t,
                                                  table_len, tok_pos, heads, nr, r_places, status);
        const dim3 g((unsigned)(ctas + (nr > 0 ? T : 0)));
        if (T <= 8)
            return launch("head_gemm", head_gemv_kernel<8>, g, dim3(256), 0, stream, one, (const bf16*)a, (const bf16*)w, (bf16*)out,
                          (const bf16*)gate, st, rp, ctas, T, heads, N, K);
        return launch("head_gemm", head_gemv_kernel<16>, g, dim3(256), 0, stream, one, (const bf16*)a, (const bf16*)w, (bf16*)out,
                      (const bf16*)gate, st, rp, ctas, T, heads, N, K);
    }
    dim3 grid((N + HG_NT - 1) / HG_NT, (T + HG_MT - 1) / HG_MT, heads);
    FD_REQUIRE(grid.y <= 65535, -2, "head_gemm: %d rows are too many", T);
    int rc;
    if (dtype == 0)
        rc = launch("head_gemm", head_gemm_kernel<float>, grid, dim3(HG_THREADS), 0, stream, one, (const float*)a, (const float*)w,
                    (float*)out, (const float*)gate, st, T, heads, N, K);
    else
        rc = launch("head_gemm", head_gemm_kernel<bf16>, grid, dim3(HG_THREADS), 0, stream, one, (const bf16*)a, (const bf16*)w,
                    (bf16*)out, (const bf16*)gate, st, T, heads, N, K);
    if (rc || nr == 0) return rc;
    if (dtype == 0)
        return launch_rope(rope_part<float>((const float*)a + r_src, a_ld, a_hs, (float*)out + r_dst, o_ld, o_hs, cos_t, sin_t,
                                            table_len, tok_pos, heads, nr, r_places, status), T, stream);
    return launch_rope(rope_part<bf16>((const bf16*)a + r_src, a_ld, a_hs, (bf16*)out + r_dst, o_ld, o_hs, cos_t, sin_t, table_len,
                                       tok_pos, heads, nr, r_places, status), T, stream);
}

// src / dst: pointers to the first rotated dimension of the first head; cos_t / sin_t [table_len, nr / 2].
extern "C" int fd_rope_heads(const void* src, int s_ld, int s_hs, void* dst, int d_ld, int d_hs, int dtype, const float* cos_t,
                             const float* sin_t, int table_len, const int* tok_pos, int T, int heads, int nr, int places,
                             int* status, cudaStream_t stream) {
    if (T == 0 || nr == 0) return 0;
    FD_REQUIRE(heads > 0 && nr > 0 && nr % 2 == 0 && places >= nr && places % 2 == 0, -2, "rope_heads: %d of %d dimensions", nr, places);
    FD_REQUIRE(src != dst || places == nr, -2, "rope_heads: in place there is nothing to fill up");
    if (dtype == 0)
        return launch_rope(rope_part<float>(src, s_ld, s_hs, dst, d_ld, d_hs, cos_t, sin_t, table_len, tok_pos, heads, nr, places,
                                            status), T, stream);
    return launch_rope(rope_part<__nv_bfloat16>(src, s_ld, s_hs, dst, d_ld, d_hs, cos_t, sin_t, table_len, tok_pos, heads, nr,
                                                places, status), T, stream);
}
