// prima.cpp_b200/csrc/wkv.cu — the decay of the WKV mixer: a low-rank map of the token's mix,  decay = exp(-exp(w0 + W2 tanh(W1 m)))  per channel
// (declarations and semantics: layers.h).  It enters the recurrence's exponent, so inputs, weights, products, tanh and both exponentials are
// fp32 in either compute type.  Two products through one tile kernel; few tokens take the weight-streaming kernel for the first one.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>

#include "layers.h"
#include "mixers.cuh"

namespace pb {
namespace {

// C[t][n] = f(bias[n] + sum_k g(A[t][k]) B[n][k]):  a CTA of 256 threads owns TT tokens x 64 columns, K in steps of 64; thread (ty, tx) = (tid / 16,
// tid % 16) keeps tokens ty, ty + 16, .. and columns tx + 16 j.  Rows of both tiles are 68 floats apart: 16-byte loads along k without bank
// conflicts.  UP: g = tanh and f(z) = exp(-exp(z)), otherwise both are the identity.
constexpr int LR_COLS = 64, LR_K = 64, LR_S = LR_K + 4;
template <int TT, bool UP>
__global__ void __launch_bounds__(256) k_lowrank(const float * __restrict__ A, int64_t lda, const float * __restrict__ B, int64_t ldb, const float * __restrict__ bias,
                                                 float * __restrict__ C, int64_t ldc, int T, int N, int K) {
    __shared__ __align__(16) float As[TT][LR_S];
    __shared__ __align__(16) float Bs[LR_COLS][LR_S];
    constexpr int TR = TT / 16;
    const int t0 = blockIdx.y * TT, n0 = blockIdx.x * LR_COLS;
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    float acc[TR][4];
#pragma unroll
    for (int i = 0; i < TR; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) acc[i][j] = 0.f;
    constexpr int NA = TT * LR_K / 256, NB = LR_COLS * LR_K / 256;
    float ra[NA], rb[NB];
    auto fetch = [&](int k0) {   // the next step's values travel while the current one is multiplied
#pragma unroll
        for (int u = 0; u < NA; u++) {
            const int i = tid + 256 * u, t = t0 + i / LR_K, k = k0 + i % LR_K;
            ra[u] = t < T && k < K ? A[(int64_t) t * lda + k] : 0.f;
        }
#pragma unroll
        for (int u = 0; u < NB; u++) {
            const int i = tid + 256 * u, n = n0 + i / LR_K, k = k0 + i % LR_K;
            rb[u] = n < N && k < K ? B[(int64_t) n * ldb + k] : 0.f;
        }
    };
    fetch(0);
    for (int k0 = 0; k0 < K; k0 += LR_K) {
        __syncthreads();
#pragma unroll
        for (int u = 0; u < NA; u++) {
            const int i = tid + 256 * u;
            As[i / LR_K][i % LR_K] = UP ? tanhf(ra[u]) : ra[u];
        }
#pragma unroll
        for (int u = 0; u < NB; u++) {
            const int i = tid + 256 * u;
            Bs[i / LR_K][i % LR_K] = rb[u];
        }
        __syncthreads();
        if (k0 + LR_K < K) fetch(k0 + LR_K);
#pragma unroll 4
        for (int k = 0; k < LR_K; k += 4) {
            float4 a[TR], b[4];
#pragma unroll
            for (int i = 0; i < TR; i++) a[i] = *reinterpret_cast<const float4 *>(&As[ty + 16 * i][k]);
#pragma unroll
            for (int j = 0; j < 4; j++) b[j] = *reinterpret_cast<const float4 *>(&Bs[tx + 16 * j][k]);
#pragma unroll
            for (int i = 0; i < TR; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) {
                    acc[i][j] = fmaf(a[i].x, b[j].x, acc[i][j]); acc[i][j] = fmaf(a[i].y, b[j].y, acc[i][j]);
                    acc[i][j] = fmaf(a[i].z, b[j].z, acc[i][j]); acc[i][j] = fmaf(a[i].w, b[j].w, acc[i][j]);
                }
        }
    }
#pragma unroll
    for (int i = 0; i < TR; i++) {
        const int t = t0 + ty + 16 * i;
        if (t >= T) continue;
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int n = n0 + tx + 16 * j;
            if (n >= N) continue;
            float v = acc[i][j];
            if (UP) v = expf(-expf(v + bias[n]));
            C[(int64_t) t * ldc + n] = v;
        }
    }
}

}  // namespace

int launch_lowrank_decay(const float * m, const float * w1, const float * w2, const float * w0, int n_tokens, int width, int rank, int channels, float * tmp,
                         float * decay, cudaStream_t st) {
    if (n_tokens <= 0 || channels <= 0) return 0;
    if (!m || !w1 || !w2 || !w0 || !tmp || !decay || width <= 0 || rank <= 0) return (int) cudaErrorInvalidValue;
    int rc;
    if (n_tokens <= 8) {
        rc = launch_dense(0 /* T_F32 */, m, width, w1, width, tmp, rank, n_tokens, rank, width, nullptr, nullptr, 0, 1.f, st);
    } else {
        const dim3 g1((unsigned) ((rank + LR_COLS - 1) / LR_COLS), (unsigned) ((n_tokens + 15) / 16));
        rc = ck_launch([&] { k_lowrank<16, false><<<g1, 256, 0, st>>>(m, width, w1, width, nullptr, tmp, rank, n_tokens, rank, width); });
    }
    if (rc) return rc;
    if (n_tokens <= 64) {
        const dim3 g2((unsigned) ((channels + LR_COLS - 1) / LR_COLS), (unsigned) ((n_tokens + 15) / 16));
        return ck_launch([&] { k_lowrank<16, true><<<g2, 256, 0, st>>>(tmp, rank, w2, rank, w0, decay, channels, n_tokens, channels, rank); });
    }
    const dim3 g2((unsigned) ((channels + LR_COLS - 1) / LR_COLS), (unsigned) ((n_tokens + 63) / 64));
    return ck_launch([&] { k_lowrank<64, true><<<g2, 256, 0, st>>>(tmp, rank, w2, rank, w0, decay, channels, n_tokens, channels, rank); });
}

}  // namespace pb
