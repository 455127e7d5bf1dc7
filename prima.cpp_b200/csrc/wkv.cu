// prima.cpp_b200/csrc/wkv.cu — low-rank maps of the token that end in decays or gates, and the WKV mixer's own kernels (declarations and
// semantics: layers.h): the WKV decay, a low-rank map of the token's mix,
// decay = exp(-exp(w0 + W2 tanh(W1 m)))  per channel, and the recurrence for the usual head sizes (any other size runs through the kernels of
// gated.cu).  Everything that reaches the recurrence's state is fp32 in either compute type: the map's inputs, weights, products, tanh and both
// exponentials, keys, values and the state.
#include <cooperative_groups.h>
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>

#include "layers.h"
#include "mixers.cuh"

namespace cg = cooperative_groups;

namespace pb {
namespace {

// ---- the decay's map ----
// One tile step: a CTA of 256 threads owns TT tokens x 64 columns; thread (ty, tx) = (tid / 16, tid % 16) keeps tokens ty, ty + 16, .. and columns
// tx + 16 j.  Rows of both tiles are 68 floats apart: 16-byte loads along k without bank conflicts.
constexpr int LR_COLS = 64, LR_K = 64, LR_S = LR_K + 4;
template <int TT>
__device__ __forceinline__ void lowrank_tile(const float (&As)[TT][LR_S], const float (&Bs)[LR_COLS][LR_S], int ty, int tx, float (&acc)[TT / 16][4]) {
    constexpr int TR = TT / 16;
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
// rows [r0, r0 + ROWS) x k [k0, k0 + 64) of a row-major matrix through registers into a tile (zeros beyond the edges)
template <int ROWS>
struct LowrankFetch {
    static constexpr int NV = ROWS * LR_K / 256;
    float v[NV];
    __device__ __forceinline__ void load(const float * __restrict__ M, int64_t ld, int r0, int rows, int k0, int K) {
#pragma unroll
        for (int u = 0; u < NV; u++) {
            const int i = threadIdx.x + 256 * u, r = r0 + i / LR_K, k = k0 + i % LR_K;
            v[u] = r < rows && k < K ? M[(int64_t) r * ld + k] : 0.f;
        }
    }
    __device__ __forceinline__ void store(float (&S)[ROWS][LR_S]) const {
#pragma unroll
        for (int u = 0; u < NV; u++) { const int i = threadIdx.x + 256 * u; S[i / LR_K][i % LR_K] = v[u]; }
    }
};

// tmp[t][j] = tanh(sum_k m[t][k] w1[j][k]): a cluster of 8 CTAs shares a tile, each walks its eighth of the width; the partial sums meet through
// distributed shared memory, summed in the order of the CTAs (a token's result depends on the width alone, not on the batch)
constexpr int LR_SPLIT = 8;
template <int TT>
__global__ void __cluster_dims__(1, 1, LR_SPLIT) __launch_bounds__(256) k_lowrank_down(const float * __restrict__ m, const float * __restrict__ w1,
                                                                                    float * __restrict__ tmp, int T, int rank, int width) {
    __shared__ __align__(16) float As[TT][LR_S];
    __shared__ __align__(16) float Bs[LR_COLS][LR_S];
    cg::cluster_group cl = cg::this_cluster();
    const int me = (int) cl.block_rank();
    const int t0 = blockIdx.y * TT, n0 = blockIdx.x * LR_COLS;
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const int steps = (width + LR_K - 1) / LR_K, per = (steps + LR_SPLIT - 1) / LR_SPLIT;
    const int s_lo = me * per, s_hi = min(steps, s_lo + per);
    float acc[TT / 16][4];
#pragma unroll
    for (int i = 0; i < TT / 16; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) acc[i][j] = 0.f;
    LowrankFetch<TT> fa;
    LowrankFetch<LR_COLS> fb;
    if (s_lo < s_hi) { fa.load(m, width, t0, T, s_lo * LR_K, width); fb.load(w1, width, n0, rank, s_lo * LR_K, width); }
    for (int s = s_lo; s < s_hi; s++) {
        __syncthreads();
        fa.store(As);
        fb.store(Bs);
        __syncthreads();
        if (s + 1 < s_hi) { fa.load(m, width, t0, T, (s + 1) * LR_K, width); fb.load(w1, width, n0, rank, (s + 1) * LR_K, width); }   // travels meanwhile
        lowrank_tile<TT>(As, Bs, ty, tx, acc);
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < TT / 16; i++)   // the operand tile's memory takes the partial sums
#pragma unroll
        for (int j = 0; j < 4; j++) As[ty + 16 * i][tx + 16 * j] = acc[i][j];
    cl.sync();
    for (int i = me * 256 + tid; i < TT * LR_COLS; i += LR_SPLIT * 256) {
        const int t = t0 + i / LR_COLS, n = n0 + i % LR_COLS;
        float v = 0.f;
#pragma unroll
        for (int r = 0; r < LR_SPLIT; r++) v += cl.map_shared_rank(&As[0][0], r)[(i / LR_COLS) * LR_S + i % LR_COLS];
        if (t < T && n < rank) tmp[(int64_t) t * rank + n] = tanhf(v);
    }
    cl.sync();   // nobody leaves while its partial sums may still be read
}
// decay[t][n] = exp(-exp(w0[n] + sum_j tmp[t][j] w2[n][j]));  RAW: tmp holds the sums before their tanh
template <int TT, bool RAW>
__global__ void __launch_bounds__(256) k_lowrank_up(const float * __restrict__ tmp, const float * __restrict__ w2, const float * __restrict__ w0,
                                                    float * __restrict__ decay, int T, int N, int rank) {
    __shared__ __align__(16) float As[TT][LR_S];
    __shared__ __align__(16) float Bs[LR_COLS][LR_S];
    const int t0 = blockIdx.y * TT, n0 = blockIdx.x * LR_COLS;
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    float acc[TT / 16][4];
#pragma unroll
    for (int i = 0; i < TT / 16; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) acc[i][j] = 0.f;
    LowrankFetch<TT> fa;
    LowrankFetch<LR_COLS> fb;
    for (int k0 = 0; k0 < rank; k0 += LR_K) {
        fa.load(tmp, rank, t0, T, k0, rank);
        if constexpr (RAW) {
#pragma unroll
            for (int u = 0; u < LowrankFetch<TT>::NV; u++) fa.v[u] = tanhf(fa.v[u]);
        }
        fb.load(w2, rank, n0, N, k0, rank);
        __syncthreads();
        fa.store(As);
        fb.store(Bs);
        __syncthreads();
        lowrank_tile<TT>(As, Bs, ty, tx, acc);
    }
#pragma unroll
    for (int i = 0; i < TT / 16; i++) {
        const int t = t0 + ty + 16 * i;
        if (t >= T) continue;
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int n = n0 + tx + 16 * j;
            if (n < N) decay[(int64_t) t * N + n] = expf(-expf(acc[i][j] + w0[n]));
        }
    }
}

// two maps side by side (LowrankMaps): column tiles of the decay first, then those of the gate
template <int TT>
__global__ void __launch_bounds__(256) k_lowrank_maps(LowrankMaps mp, int T, int a_tiles) {
    __shared__ __align__(16) float As[TT][LR_S];
    __shared__ __align__(16) float Bs[LR_COLS][LR_S];
    const bool is_a = (int) blockIdx.x < a_tiles;
    const int t0 = blockIdx.y * TT, n0 = (is_a ? blockIdx.x : blockIdx.x - a_tiles) * LR_COLS;
    const int N = is_a ? mp.heads * mp.dim : mp.gate_cols, rank = is_a ? mp.ra : mp.rg;
    const float * z = is_a ? mp.za : mp.zg, * w = is_a ? mp.wa : mp.wg;
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    float acc[TT / 16][4];
#pragma unroll
    for (int i = 0; i < TT / 16; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) acc[i][j] = 0.f;
    LowrankFetch<TT> fa;
    LowrankFetch<LR_COLS> fb;
    for (int k0 = 0; k0 < rank; k0 += LR_K) {
        fa.load(z, mp.ldu, t0, T, k0, rank);
        fb.load(w, rank, n0, N, k0, rank);
        __syncthreads();
        fa.store(As);
        fb.store(Bs);
        __syncthreads();
        lowrank_tile<TT>(As, Bs, ty, tx, acc);
    }
    float rate[4], bias[4];
#pragma unroll
    for (int j = 0; j < 4; j++) {
        const int n = n0 + tx + 16 * j;
        rate[j] = is_a && n < N ? expf(mp.A_log[n / mp.dim]) : 0.f;
        bias[j] = is_a && n < N ? mp.dt_bias[n] : 0.f;
    }
#pragma unroll
    for (int i = 0; i < TT / 16; i++) {
        const int t = t0 + ty + 16 * i;
        if (t >= T) continue;
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int n = n0 + tx + 16 * j;
            if (n >= N) continue;
            if (is_a) mp.decay[(int64_t) t * mp.ldd + n] = expf(-rate[j] * softplus_f(acc[i][j] + bias[j]));
            else mp.gate[(int64_t) t * mp.ldg + n] = acc[i][j];
        }
    }
}

// ---- the recurrence at head sizes N = 32, 64, 128, 256 ----
//   y_t = S^T r_t + (r_t . u k_t) v_t,  then  S <- diag(w_t) S + k_t v_t^T
// CTA = one head x 16 value columns of one entry.  LN = N / 8 lanes share a pair of columns: a lane keeps S[n][2 columns] for 8 n (four
// consecutive ones in either half of the key size), so the 16-byte loads of a token's r, k, w rows from shared memory serve two columns.  Tokens arrive in chunks of 16 through two cp.async stages.
// The state's chain is one multiply-add per token; the sums S^T r leave it aside: a full chunk keeps its 32 partial sums (16 tokens x 2
// columns) in registers and reduces them together, halving the number of values with every exchange (31 shuffles instead of 32 log2(LN)).
constexpr int WS_CHUNK = 16, WS_COLS = 16, WS_STAGES = 2, WS_NREG = 8;
template <int N> constexpr int ws_stage_floats() { return WS_CHUNK * (3 * N + WS_COLS); }


template <int N>
__global__ void __launch_bounds__(WS_COLS / 2 * (N / WS_NREG)) k_wkv_scan(GatedLinIO io, const int32_t * __restrict__ slot, const int32_t * __restrict__ off,
                                                                      GatedLinParams p, float * __restrict__ state, int64_t slot_stride, float * __restrict__ y) {
    extern __shared__ __align__(16) float sm[];   // [stages][ r [16][N] | k [16][N] | w [16][N] | v [16][16] ], then the bonus products [16]
    constexpr int LN = N / WS_NREG, NT = WS_COLS / 2 * LN, STAGE = ws_stage_floats<N>();
    const int P = p.vdim, inner = p.heads * P, ptiles = (P + WS_COLS - 1) / WS_COLS;
    const int h = blockIdx.x / ptiles, pt = blockIdx.x - h * ptiles, e = blockIdx.y;
    const int hk = h / (p.heads / p.qk_heads);
    const int tid = threadIdx.x, lane = tid & 31, ng = tid % LN, cp = tid / LN;   // this thread: n = n_of(0..7), columns 2 cp, 2 cp + 1 of the tile
    auto n_of = [&](int j) { return (j >> 2) * (N / 2) + 4 * ng + (j & 3); };
    const int col = pt * WS_COLS + 2 * cp;
    const bool ok0 = col < P, ok1 = col + 1 < P;
    float * Bs = sm + WS_STAGES * STAGE;
    float * gst = state + (int64_t) slot[e] * slot_stride + (int64_t) h * N * P;
    const int t0 = off[e], n = off[e + 1] - t0;
    auto stage_in = [&](int c0, float * st) {
        const int nc = min(WS_CHUNK, n - c0);
        constexpr int Q = N / 4;                     // 16-byte pieces of a row
#pragma unroll 4
        for (int i = tid; i < 3 * WS_CHUNK * Q; i += NT) {
            const int which = i / (WS_CHUNK * Q), rem = i % (WS_CHUNK * Q), tt = rem / Q, q = rem % Q;
            const int64_t tok = t0 + c0 + min(tt, nc - 1);
            const float * src = which == 0 ? io.q + tok * io.ldq : which == 1 ? io.k + tok * io.ldk : io.decay + tok * io.ldd;
            cp_async16(st + which * WS_CHUNK * N + tt * N + 4 * q, src + (which == 2 ? h : hk) * N + 4 * q, tt < nc);
        }
        for (int i = tid; i < WS_CHUNK * (WS_COLS / 4); i += NT) {
            const int tt = i / (WS_COLS / 4), q = i % (WS_COLS / 4), c = pt * WS_COLS + 4 * q;
            const bool ok = tt < nc && c < P;        // P is a multiple of 4
            cp_async16(st + 3 * WS_CHUNK * N + tt * WS_COLS + 4 * q, ok ? io.v + (int64_t) (t0 + c0 + tt) * io.ldv + h * P + c : io.v, ok);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    if (n > 0) stage_in(0, sm);
    float S0[WS_NREG], S1[WS_NREG];
#pragma unroll
    for (int j = 0; j < WS_NREG; j++) {
        const float * g = gst + (int64_t) n_of(j) * P + col;
        S0[j] = ok0 ? g[0] : 0.f;
        S1[j] = ok1 ? g[1] : 0.f;
    }
    const float * ub = io.bonus + (int64_t) hk * N;
    for (int c0 = 0, it = 0; c0 < n; c0 += WS_CHUNK, it++) {
        const int nc = min(WS_CHUNK, n - c0);
        float * st = sm + (it & 1) * STAGE;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                             // the stage is complete, and everybody is done with the other one
        if (c0 + WS_CHUNK < n) stage_in(c0 + WS_CHUNK, sm + ((it + 1) & 1) * STAGE);
        const float * Rs = st, * Ks = st + WS_CHUNK * N, * Ws = st + 2 * WS_CHUNK * N, * Vs = st + 3 * WS_CHUNK * N;
        for (int tt = tid >> 5; tt < nc; tt += (NT + 31) / 32) {   // r . (u k) of every token, a warp each
            float b = 0.f;
#pragma unroll
            for (int nn = lane; nn < N; nn += 32) b = fmaf(Rs[tt * N + nn] * ub[nn], Ks[tt * N + nn], b);
            b = wsum(b);
            if (lane == 0) Bs[tt] = b;
        }
        __syncthreads();
        auto token = [&](int tt, float & a0, float & a1) {
            const float2 v = *reinterpret_cast<const float2 *>(Vs + tt * WS_COLS + 2 * cp);
            float x0 = 0.f, x1 = 0.f;
#pragma unroll
            for (int j = 0; j < WS_NREG; j += 4) {
                const int o = tt * N + n_of(j);
                const float4 r = *reinterpret_cast<const float4 *>(Rs + o), k = *reinterpret_cast<const float4 *>(Ks + o), w = *reinterpret_cast<const float4 *>(Ws + o);
                const float rr[4] = {r.x, r.y, r.z, r.w}, kk[4] = {k.x, k.y, k.z, k.w}, ww[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
                for (int i = 0; i < 4; i++) {
                    x0 = fmaf(S0[j + i], rr[i], x0);
                    x1 = fmaf(S1[j + i], rr[i], x1);
                    S0[j + i] = fmaf(ww[i], S0[j + i], kk[i] * v.x);
                    S1[j + i] = fmaf(ww[i], S1[j + i], kk[i] * v.y);
                }
            }
            a0 = x0;
            a1 = x1;
        };
        if (nc == WS_CHUNK) {
            constexpr int M = 2 * WS_CHUNK, KEEP = M / LN;   // partial sums, and how many whole ones a lane ends up with
            float acc[M];                                    // value token * 2 + column
#pragma unroll
            for (int tt = 0; tt < WS_CHUNK; tt++) token(tt, acc[2 * tt], acc[2 * tt + 1]);
            joint_sum<M, LN / 2>(acc, lane);
#pragma unroll
            for (int i = 0; i < KEEP; i++) {
                const int idx = ng * KEEP + i, tt = idx >> 1, c = idx & 1;
                if (c == 0 ? ok0 : ok1) y[(int64_t) (t0 + c0 + tt) * inner + h * P + col + c] = fmaf(Bs[tt], Vs[tt * WS_COLS + 2 * cp + c], acc[i]);
            }
        } else {
            for (int tt = 0; tt < nc; tt++) {
                float a0, a1;
                token(tt, a0, a1);
#pragma unroll
                for (int o = 1; o < LN; o <<= 1) {
                    a0 += __shfl_xor_sync(0xffffffffu, a0, o);
                    a1 += __shfl_xor_sync(0xffffffffu, a1, o);
                }
                if (ng == 0 && ok0) y[(int64_t) (t0 + c0 + tt) * inner + h * P + col] = fmaf(Bs[tt], Vs[tt * WS_COLS + 2 * cp], a0);
                if (ng == 0 && ok1) y[(int64_t) (t0 + c0 + tt) * inner + h * P + col + 1] = fmaf(Bs[tt], Vs[tt * WS_COLS + 2 * cp + 1], a1);
            }
        }
    }
#pragma unroll
    for (int j = 0; j < WS_NREG; j++) {
        float * g = gst + (int64_t) n_of(j) * P + col;
        if (ok0) g[0] = S0[j];
        if (ok1) g[1] = S1[j];
    }
}

template <int N>
int wkv_scan_launch(const GatedLinIO & io, const BatchView & b, const GatedLinParams & p, float * state, int64_t slot_stride, float * y, cudaStream_t st) {
    const size_t smem = ((size_t) WS_STAGES * ws_stage_floats<N>() + WS_CHUNK) * sizeof(float);
    const int rc = raise_smem(k_wkv_scan<N>, smem);
    if (rc) return rc;
    const dim3 grid((unsigned) (p.heads * ((p.vdim + WS_COLS - 1) / WS_COLS)), (unsigned) b.n_entries);
    return ck_launch([&] { k_wkv_scan<N><<<grid, WS_COLS / 2 * (N / WS_NREG), smem, st>>>(io, b.slot, b.off, p, state, slot_stride, y); });
}

}  // namespace

// 1: the kernel above takes this recurrence (bonus form, a head size it is built for, rows that 16-byte copies can read)
int wkv_scan_ok(const GatedLinIO & io, const GatedLinParams & p) {
    auto al = [](const float * q, int64_t ld) { return ((uintptr_t) q & 15) == 0 && ld % 4 == 0; };
    return p.bonus && (p.dim == 32 || p.dim == 64 || p.dim == 128 || p.dim == 256) && p.vdim % 4 == 0 && al(io.q, io.ldq) && al(io.k, io.ldk) && al(io.v, io.ldv) &&
           al(io.decay, io.ldd);
}
int launch_wkv_scan(const GatedLinIO & io, const BatchView & b, const GatedLinParams & p, float * state, int64_t slot_stride, float * y, cudaStream_t st) {
    if (p.dim == 32) return wkv_scan_launch<32>(io, b, p, state, slot_stride, y, st);
    if (p.dim == 64) return wkv_scan_launch<64>(io, b, p, state, slot_stride, y, st);
    if (p.dim == 128) return wkv_scan_launch<128>(io, b, p, state, slot_stride, y, st);
    if (p.dim == 256) return wkv_scan_launch<256>(io, b, p, state, slot_stride, y, st);
    return (int) cudaErrorInvalidValue;
}

int launch_lowrank_maps(const LowrankMaps & mp, int n_tokens, cudaStream_t st) {
    if (n_tokens <= 0) return 0;
    if (!mp.za || !mp.wa || mp.ra <= 0 || !mp.A_log || !mp.dt_bias || !mp.decay || mp.heads <= 0 || mp.dim <= 0 || mp.gate_cols < 0 ||
        (mp.gate_cols > 0 && (!mp.zg || !mp.wg || mp.rg <= 0 || !mp.gate)))
        return (int) cudaErrorInvalidValue;
    const int at = (mp.heads * mp.dim + LR_COLS - 1) / LR_COLS;
    const unsigned tiles = (unsigned) (at + (mp.gate_cols + LR_COLS - 1) / LR_COLS);
    return ck_launch([&] {
        if (n_tokens > 64) k_lowrank_maps<64><<<dim3(tiles, (unsigned) ((n_tokens + 63) / 64)), 256, 0, st>>>(mp, n_tokens, at);
        else k_lowrank_maps<16><<<dim3(tiles, (unsigned) ((n_tokens + 15) / 16)), 256, 0, st>>>(mp, n_tokens, at);
    });
}

int launch_lowrank_decay(const float * m, const float * w1, const float * w2, const float * w0, int n_tokens, int width, int rank, int channels, float * tmp,
                         float * decay, cudaStream_t st) {
    if (n_tokens <= 0 || channels <= 0) return 0;
    if (!m || !w1 || !w2 || !w0 || !tmp || !decay || width <= 0 || rank <= 0) return (int) cudaErrorInvalidValue;
    const unsigned rt = (unsigned) ((rank + LR_COLS - 1) / LR_COLS), ct = (unsigned) ((channels + LR_COLS - 1) / LR_COLS);
    if (n_tokens <= 4) {   // one or a few tokens: the weight-streaming product, the tanh at its reader
        const int rc = launch_dense(0 /* T_F32 */, m, width, w1, width, tmp, rank, n_tokens, rank, width, nullptr, nullptr, 0, 1.f, st);
        if (rc) return rc;
        return ck_launch([&] { k_lowrank_up<16, true><<<dim3(ct, 1), 256, 0, st>>>(tmp, w2, w0, decay, n_tokens, channels, rank); });
    }
    int rc = ck_launch([&] {
        if (n_tokens >= 1024) k_lowrank_down<64><<<dim3(rt, (unsigned) ((n_tokens + 63) / 64), LR_SPLIT), 256, 0, st>>>(m, w1, tmp, n_tokens, rank, width);
        else k_lowrank_down<16><<<dim3(rt, (unsigned) ((n_tokens + 15) / 16), LR_SPLIT), 256, 0, st>>>(m, w1, tmp, n_tokens, rank, width);
    });
    if (rc) return rc;
    return ck_launch([&] {
        if (n_tokens > 64) k_lowrank_up<64, false><<<dim3(ct, (unsigned) ((n_tokens + 63) / 64)), 256, 0, st>>>(tmp, w2, w0, decay, n_tokens, channels, rank);
        else k_lowrank_up<16, false><<<dim3(ct, (unsigned) ((n_tokens + 15) / 16)), 256, 0, st>>>(tmp, w2, w0, decay, n_tokens, channels, rank);
    });
}

}  // namespace pb
