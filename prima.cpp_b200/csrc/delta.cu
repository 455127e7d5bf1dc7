// prima.cpp_b200/csrc/delta.cu — the gated delta rule with a decay per head and key channel for the usual head sizes (declaration and semantics:
// layers.h, GatedLinParams; any other size runs through the kernels of gated.cu).  Keys, queries, decays, step sizes, values and the state are fp32
// in either compute type.
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include "layers.h"
#include "mixers.cuh"

namespace pb {
namespace {

// ---- head sizes N = 32, 64, 128, 256 ----
//   S <- diag(g_t) S,  u = beta_t (v_t - S^T k_t),  S <- S + k_t u^T,  y_t = S^T q_t
// CTA = one head x 16 value columns of one entry.  LN = N / 8 lanes share a pair of columns: a lane keeps S[n][2 columns] for 8 n (four
// consecutive ones in either half of the key size), so the 16-byte loads of a token's q, k, g rows from shared memory serve two columns.  Tokens
// arrive in chunks of 16 through two cp.async stages.  The chain from token to token is decay, product with the key, its sum over the lanes (the
// two columns' shuffles side by side) and the rank-one write; the read-out with the query leaves it aside: a full chunk keeps its 32 partial sums
// (16 tokens x 2 columns) in registers and sums them together (30 shuffles at most instead of 32 log2(LN)).
constexpr int DS_CHUNK = 16, DS_COLS = 16, DS_STAGES = 2, DS_NREG = 8;
template <int N> constexpr int ds_stage_floats() { return DS_CHUNK * (3 * N + DS_COLS + 1); }

template <int N>
__global__ void __launch_bounds__(DS_COLS / 2 * (N / DS_NREG)) k_delta_scan(GatedLinIO io, const int32_t * __restrict__ slot, const int32_t * __restrict__ off,
                                                                           GatedLinParams p, float * __restrict__ state, int64_t slot_stride, float * __restrict__ y) {
    extern __shared__ __align__(16) float sm[];   // [stages][ q [16][N] | k [16][N] | g [16][N] | v [16][16] | beta [16] ]
    constexpr int LN = N / DS_NREG, NT = DS_COLS / 2 * LN, STAGE = ds_stage_floats<N>();
    const int P = p.vdim, inner = p.heads * P, ptiles = (P + DS_COLS - 1) / DS_COLS;
    const int h = blockIdx.x / ptiles, pt = blockIdx.x - h * ptiles, e = blockIdx.y;
    const int hk = h / (p.heads / p.qk_heads);
    const int tid = threadIdx.x, lane = tid & 31, ng = tid % LN, cp = tid / LN;   // this thread: n = n_of(0..7), columns 2 cp, 2 cp + 1 of the tile
    auto n_of = [&](int j) { return (j >> 2) * (N / 2) + 4 * ng + (j & 3); };
    const int col = pt * DS_COLS + 2 * cp;
    const bool ok0 = col < P, ok1 = col + 1 < P;
    float * gst = state + (int64_t) slot[e] * slot_stride + (int64_t) h * N * P;
    const int t0 = off[e], n = off[e + 1] - t0;
    auto stage_in = [&](int c0, float * st) {
        const int nc = min(DS_CHUNK, n - c0);
        constexpr int Q = N / 4;                     // 16-byte pieces of a row
#pragma unroll 4
        for (int i = tid; i < 3 * DS_CHUNK * Q; i += NT) {
            const int which = i / (DS_CHUNK * Q), rem = i % (DS_CHUNK * Q), tt = rem / Q, q = rem % Q;
            const int64_t tok = t0 + c0 + min(tt, nc - 1);
            const float * src = which == 0 ? io.q + tok * io.ldq + hk * N : which == 1 ? io.k + tok * io.ldk + hk * N : io.decay + tok * io.ldd + h * N;
            cp_async16(st + which * DS_CHUNK * N + tt * N + 4 * q, src + 4 * q, tt < nc);
        }
        for (int i = tid; i < DS_CHUNK * (DS_COLS / 4); i += NT) {
            const int tt = i / (DS_COLS / 4), q = i % (DS_COLS / 4), c = pt * DS_COLS + 4 * q;
            const bool ok = tt < nc && c < P;        // P is a multiple of 4
            cp_async16(st + 3 * DS_CHUNK * N + tt * DS_COLS + 4 * q, ok ? io.v + (int64_t) (t0 + c0 + tt) * io.ldv + h * P + c : io.v, ok);
        }
        if (tid < DS_CHUNK) {
            const bool ok = tid < nc;
            cp_async4(st + DS_CHUNK * (3 * N + DS_COLS) + tid, ok ? io.beta + (int64_t) (t0 + c0 + tid) * io.ldb + h : io.beta, ok);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    if (n > 0) stage_in(0, sm);
    float S0[DS_NREG], S1[DS_NREG];
#pragma unroll
    for (int j = 0; j < DS_NREG; j++) {
        const float * g = gst + (int64_t) n_of(j) * P + col;
        S0[j] = ok0 ? g[0] : 0.f;
        S1[j] = ok1 ? g[1] : 0.f;
    }
    for (int c0 = 0, it = 0; c0 < n; c0 += DS_CHUNK, it++) {
        const int nc = min(DS_CHUNK, n - c0);
        float * st = sm + (it & 1) * STAGE;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                             // the stage is complete, and everybody is done with the other one
        if (c0 + DS_CHUNK < n) stage_in(c0 + DS_CHUNK, sm + ((it + 1) & 1) * STAGE);
        const float * Qs = st, * Ks = st + DS_CHUNK * N, * Gs = st + 2 * DS_CHUNK * N, * Vs = st + 3 * DS_CHUNK * N, * Bs = Vs + DS_CHUNK * DS_COLS;
        auto token = [&](int tt, float & y0, float & y1) {
            float kk[DS_NREG], x0 = 0.f, x1 = 0.f;
#pragma unroll
            for (int j = 0; j < DS_NREG; j += 4) {
                const int o = tt * N + n_of(j);
                const float4 k = *reinterpret_cast<const float4 *>(Ks + o), g = *reinterpret_cast<const float4 *>(Gs + o);
                const float gg[4] = {g.x, g.y, g.z, g.w};
                kk[j] = k.x; kk[j + 1] = k.y; kk[j + 2] = k.z; kk[j + 3] = k.w;
#pragma unroll
                for (int i = 0; i < 4; i++) {
                    S0[j + i] *= gg[i];
                    S1[j + i] *= gg[i];
                    x0 = fmaf(S0[j + i], kk[j + i], x0);
                    x1 = fmaf(S1[j + i], kk[j + i], x1);
                }
            }
#pragma unroll
            for (int o = 1; o < LN; o <<= 1) {
                x0 += __shfl_xor_sync(0xffffffffu, x0, o);
                x1 += __shfl_xor_sync(0xffffffffu, x1, o);
            }
            const float2 v = *reinterpret_cast<const float2 *>(Vs + tt * DS_COLS + 2 * cp);
            const float b = Bs[tt], u0 = b * (v.x - x0), u1 = b * (v.y - x1);
            y0 = y1 = 0.f;
#pragma unroll
            for (int j = 0; j < DS_NREG; j += 4) {
                const float4 q = *reinterpret_cast<const float4 *>(Qs + tt * N + n_of(j));
                const float qq[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
                for (int i = 0; i < 4; i++) {
                    S0[j + i] = fmaf(kk[j + i], u0, S0[j + i]);
                    S1[j + i] = fmaf(kk[j + i], u1, S1[j + i]);
                    y0 = fmaf(S0[j + i], qq[i], y0);
                    y1 = fmaf(S1[j + i], qq[i], y1);
                }
            }
        };
        if (nc == DS_CHUNK) {
            constexpr int M = 2 * DS_CHUNK, KEEP = M / LN;   // partial sums, and how many whole ones a lane ends up with
            float acc[M];                                    // value token * 2 + column
#pragma unroll
            for (int tt = 0; tt < DS_CHUNK; tt++) token(tt, acc[2 * tt], acc[2 * tt + 1]);
            joint_sum<M, LN / 2>(acc, lane);
#pragma unroll
            for (int i = 0; i < KEEP; i++) {
                const int idx = ng * KEEP + i, tt = idx >> 1, c = idx & 1;
                if (c == 0 ? ok0 : ok1) y[(int64_t) (t0 + c0 + tt) * inner + h * P + col + c] = acc[i];
            }
        } else {
            for (int tt = 0; tt < nc; tt++) {
                float y0, y1;
                token(tt, y0, y1);
#pragma unroll
                for (int o = 1; o < LN; o <<= 1) {
                    y0 += __shfl_xor_sync(0xffffffffu, y0, o);
                    y1 += __shfl_xor_sync(0xffffffffu, y1, o);
                }
                if (ng == 0 && ok0) y[(int64_t) (t0 + c0 + tt) * inner + h * P + col] = y0;
                if (ng == 0 && ok1) y[(int64_t) (t0 + c0 + tt) * inner + h * P + col + 1] = y1;
            }
        }
    }
#pragma unroll
    for (int j = 0; j < DS_NREG; j++) {
        float * g = gst + (int64_t) n_of(j) * P + col;
        if (ok0) g[0] = S0[j];
        if (ok1) g[1] = S1[j];
    }
}

template <int N>
int delta_scan_launch(const GatedLinIO & io, const BatchView & b, const GatedLinParams & p, float * state, int64_t slot_stride, float * y, cudaStream_t st) {
    const size_t smem = (size_t) DS_STAGES * ds_stage_floats<N>() * sizeof(float);
    const int rc = raise_smem(k_delta_scan<N>, smem);
    if (rc) return rc;
    const dim3 grid((unsigned) (p.heads * ((p.vdim + DS_COLS - 1) / DS_COLS)), (unsigned) b.n_entries);
    return ck_launch([&] { k_delta_scan<N><<<grid, DS_COLS / 2 * (N / DS_NREG), smem, st>>>(io, b.slot, b.off, p, state, slot_stride, y); });
}

}  // namespace

// 1: the kernel above takes this recurrence (a head size it is built for, rows that 16-byte copies can read)
int delta_scan_ok(const GatedLinIO & io, const GatedLinParams & p) {
    auto al = [](const float * q, int64_t ld) { return ((uintptr_t) q & 15) == 0 && ld % 4 == 0; };
    return p.delta && p.decay_per_channel && (p.dim == 32 || p.dim == 64 || p.dim == 128 || p.dim == 256) && p.vdim % 4 == 0 && al(io.q, io.ldq) &&
           al(io.k, io.ldk) && al(io.v, io.ldv) && al(io.decay, io.ldd);
}
int launch_delta_scan(const GatedLinIO & io, const BatchView & b, const GatedLinParams & p, float * state, int64_t slot_stride, float * y, cudaStream_t st) {
    if (p.dim == 32) return delta_scan_launch<32>(io, b, p, state, slot_stride, y, st);
    if (p.dim == 64) return delta_scan_launch<64>(io, b, p, state, slot_stride, y, st);
    if (p.dim == 128) return delta_scan_launch<128>(io, b, p, state, slot_stride, y, st);
    if (p.dim == 256) return delta_scan_launch<256>(io, b, p, state, slot_stride, y, st);
    return (int) cudaErrorInvalidValue;
}

}  // namespace pb
