// gtb_seq_recur.cuh -- recurrent token mixers whose decay depends on the token, for the layer-list sequence models:
//   * "mLSTM": S <- a_t S + w_t k_t [v_t | 1]^T per head, a and w from a capped exponential input gate and a logistic forget gate under a
//     running maximum; the column of ones is the normaliser, so it needs no kernel of its own
//   * gated delta rule: S decays by g_t, then moves by beta_t k_t (v_t - S^T k_t)^T, then is read with q_t; unit-length q and k
//   * selective scan (Mamba): every channel holds a row of numbers that decay by e^(step A) and gain step x B, read out with C
// Rows are walked one by one from the slot's state (decode rows, short portions, float mode); prompt portions in bf16 mode take the first two
// chunk-wise on tensor cores.
//
// Precision: gates, their logarithms and running sums, decays, step sizes, unit norms and the state are fp32 in both compute modes.  The tensor-core
// kernels carry every fp32 factor as the sum of two bf16 numbers ("planes" hi and lo) and multiply hi hi + hi lo + lo hi with fp32 accumulation
// (relative error 2^-17); the state itself stays in fp32 accumulators from chunk to chunk.
#pragma once
#include "gtb_seq_sandwich.cuh"

namespace gtb {
namespace seq {

constexpr int REC_MLSTM = 0, REC_DELTA = 1;
constexpr int REC_VS = 16;                   // value columns per CTA of the chunk scan

struct RecBranch {
    int heads, kv_heads, dim, vdim;          // kv_heads: heads of q and k (head h uses h / (heads / kv_heads))
    int vx, vxp;                             // state columns (vdim, and one more for the normaliser), row stride of the state
    int dp, vp;                              // plane widths per head: dim and vx rounded up to 16
    float cap, eps, qscale, out_scale;
    int q_off, k_off, v_off;                 // columns of q, k, v in the buffer X the kernels read them from
    int i_off, f_off;                        // columns of the gate pre-activations in the projection buffer: input / forget gate; decay / beta
    int g_off, a_off;                        // output gate columns; columns of the output in the out-projection operand
    const float *A_log, *dt_bias;            // [heads], delta rule
    const float* norm;                       // weight of the output norm: [heads * vdim] (mLSTM) or [vdim] (delta rule)
};

__device__ __forceinline__ float softplus_(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }
// the same with log(1 + u), u = exp(-|z|) in (0, 1], from the series of the inverse hyperbolic tangent: log(1 + u) = 2 atanh(s), s = u / (2 + u) <= 1/3
// (terms up to s^13: relative error 2e-8 beside fp32 rounding)
__device__ __forceinline__ float softplus_series(float z) {
    const float u = expf(-fabsf(z)), s = __fdividef(u, 2.0f + u), q = s * s;
    float p = fmaf(q, 1.0f / 13.0f, 1.0f / 11.0f);
    p = fmaf(q, p, 1.0f / 9.0f);
    p = fmaf(q, p, 1.0f / 7.0f);
    p = fmaf(q, p, 1.0f / 5.0f);
    p = fmaf(q, p, 1.0f / 3.0f);
    p = fmaf(q, p, 1.0f);
    return fmaxf(z, 0.0f) + 2.0f * s * p;
}
// two neighbouring values as packed hi and lo pairs
__device__ __forceinline__ void split2_pack(float a, float b, uint32_t& hi, uint32_t& lo) {
    hi = sa_pack(a, b);
    lo = sa_pack(a - __uint_as_float(hi << 16), b - __uint_as_float(hi & 0xffff0000u));
}

// ------------------------------------------------------------------------------------------------ gates
// log decay la and input weight w of one (row, head).  mLSTM: capped log input gate i and log forget gate f (their combination needs the
// running maximum); delta rule: la from the step size softplus(z + dt_bias), w = logistic
__device__ __forceinline__ void mlstm_gates(const RecBranch& b, const float* __restrict__ p, int h, float& i, float& f) {
    i = b.cap * tanhf(p[b.i_off + h] / b.cap);
    f = -softplus_(-b.cap * tanhf(p[b.f_off + h] / b.cap));
}
__device__ __forceinline__ void delta_gates(const RecBranch& b, const float* __restrict__ p, int h, float& la, float& w) {
    la = -expf(b.A_log[h]) * softplus_(p[b.i_off + h] + b.dt_bias[h]);
    w = sigmoidf_(p[b.f_off + h]);
}
// G [R][heads]: {log decay, w, m, 0}.  mLSTM: the running maximum goes from m' to m = max(f + m', i); the row's decay is e^(f + m' - m) and its
// input weight e^(i - m) times the query scale (w holds the logarithm; every factor is at most 1); delta rule: w = beta.
// Bp [R][heads] (or null): the sum of the log decays from the start of the row's chunk of C rows, as hi + lo (summed in double), so that
// differences of two sums keep their precision.  The running maximum is a max-plus scan: rows compose as (F, M) o (F', M') =
// (F + F', max(M + F', M')).  grid (segments, heads); blockDim a multiple of C (or 32 without Bp).
template <int KIND>
__global__ void __launch_bounds__(1024) k_rec_gates(PassTables t, RecBranch b, const float* __restrict__ P, int ldp, int C, float* __restrict__ mstate, float4* __restrict__ G,
                                                   float2* __restrict__ Bp) {
    __shared__ float sF[32], sM[32];
    __shared__ double sB[32];
    const int s = blockIdx.x, h = blockIdx.y, lane = threadIdx.x & 31, wid = threadIdx.x >> 5, nw = blockDim.x >> 5;
    const int slot = t.seg_slot[s], row0 = t.seg_row0[s], len = t.seg_len[s];
    float carry = KIND == REC_MLSTM ? mstate[(size_t)slot * b.heads + h] : 0.0f;
    const float lqs = KIND == REC_MLSTM ? logf(b.qscale) : 0.0f;
    for (int base = 0; base < len; base += blockDim.x) {
        const int n = base + threadIdx.x;
        const bool on = n < len;
        float la = 0.0f, w = 0.0f, m = 0.0f;
        if (KIND == REC_MLSTM) {
            float f = 0.0f, i = -INFINITY;
            if (on) mlstm_gates(b, P + (size_t)(row0 + n) * ldp, h, i, f);
            float F = f, M = i;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float pF = __shfl_up_sync(0xffffffffu, F, o), pM = __shfl_up_sync(0xffffffffu, M, o);
                if (lane >= o) { M = fmaxf(pM + F, M); F += pF; }
            }
            if (lane == 31) { sF[wid] = F; sM[wid] = M; }
            __syncthreads();
            float before = carry;
            for (int k = 0; k < wid; k++) before = fmaxf(before + sF[k], sM[k]);
            m = fmaxf(before + F, M);
            float prev = __shfl_up_sync(0xffffffffu, m, 1);
            if (lane == 0) prev = before;
            la = fminf(f + prev - m, 0.0f);
            w = i - m + lqs;
            for (int k = 0; k < nw; k++) carry = fmaxf(carry + sF[k], sM[k]);
        } else if (on) delta_gates(b, P + (size_t)(row0 + n) * ldp, h, la, w);
        if (Bp) {
            double acc = la;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const double p = __shfl_up_sync(0xffffffffu, acc, o);
                if (lane >= o) acc += p;
            }
            if (lane == 31) sB[wid] = acc;
            __syncthreads();
            for (int k = wid / (C / 32) * (C / 32); k < wid; k++) acc += sB[k];
            const float hi = (float)acc;
            if (on) Bp[(size_t)(row0 + n) * b.heads + h] = make_float2(hi, (float)(acc - (double)hi));
        }
        if (on) G[(size_t)(row0 + n) * b.heads + h] = make_float4(la, w, m, 0.0f);
        __syncthreads();                     // the shared sums are overwritten by the next block of rows
    }
    if (KIND == REC_MLSTM && threadIdx.x == 0 && !t.slots[slot].stopped) mstate[(size_t)slot * b.heads + h] = carry;
}

// unit length: every head of q and k (X columns q_off.. and k_off.., kv_heads each) divided by sqrt(sum of squares + 1e-6), q times qscale; in place
__global__ void __launch_bounds__(128) k_rec_unit(RecBranch b, float* __restrict__ X, int ldx) {
    const int r = blockIdx.x, lane = threadIdx.x & 31, wid = threadIdx.x >> 5, nw = blockDim.x >> 5;
    for (int u = blockIdx.y * nw + wid; u < 2 * b.kv_heads; u += gridDim.y * nw) {
        const bool is_q = u < b.kv_heads;
        float* v = X + (size_t)r * ldx + (is_q ? b.q_off + u * b.dim : b.k_off + (u - b.kv_heads) * b.dim);
        float ss = 0.0f;
        for (int i = lane; i < b.dim; i += 32) ss += v[i] * v[i];
        const float sc = (is_q ? b.qscale : 1.0f) / sqrtf(warp_sum(ss) + 1e-6f);
        for (int i = lane; i < b.dim; i += 32) v[i] *= sc;
    }
}

// ------------------------------------------------------------------------------------------------ rows one by one
// One CTA per (segment, head, 32 state columns) walks the segment's rows: eight warps split the rows of the state slice, RPT of them in each
// thread's registers (lane = column); the next row's q, k and v are in flight while the current one is computed.  Raw read-outs go to
// O [R][heads * vx].  The delta rule needs S^T k before it can write: with r = g S^T k and p = g S^T q from one sweep, u = beta (v - r) and
// the read-out after the write is p + (k . q) u.
// ONE: every segment is one row.  The gates are formed here from the projections P (the running maximum mstate is only read: its slices' CTAs share it, and
// k_rec_post moves it on), and q and k come as they left their convolution -- their lengths are linear factors of r, p, k . q and the write.
template <int KIND, int RPT, bool ONE>
__global__ void __launch_bounds__(256) k_rec_walk(PassTables t, RecBranch b, const float* __restrict__ X, int ldx, const float* __restrict__ P, int ldp, const float4* __restrict__ G,
                                                  const float* __restrict__ mstate, float* __restrict__ state, float* __restrict__ O) {
    constexpr int DP = RPT * 8, NPF = (DP + 255) / 256;
    __shared__ __align__(16) float sq[2][DP], sk[2][DP];
    __shared__ float part[2][2][8][32], skq[2][3][8];
    const int s = blockIdx.x, h = blockIdx.y, hk = h / (b.heads / b.kv_heads), lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
    const int slot = t.seg_slot[s], row0 = t.seg_row0[s], len = t.seg_len[s];
    const int c = blockIdx.z * 32 + lane;
    const bool ok = c < b.vx;
    float* gs = state + ((size_t)slot * b.heads + h) * (size_t)b.dim * b.vxp;
    float S[RPT];
#pragma unroll
    for (int j = 0; j < RPT; j++) { const int i = wid * RPT + j; S[j] = (ok && i < b.dim) ? gs[(size_t)i * b.vxp + c] : 0.0f; }
    float qn[NPF], kn[NPF], vn = 0.0f;
    float4 gn = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    auto fetch = [&](int n) {
        const float* x = X + (size_t)(row0 + n) * ldx;
#pragma unroll
        for (int j = 0; j < NPF; j++) {
            const int i = threadIdx.x + j * 256;
            qn[j] = i < b.dim ? x[b.q_off + hk * b.dim + i] : 0.0f;
            kn[j] = i < b.dim ? x[b.k_off + hk * b.dim + i] : 0.0f;
        }
        vn = c < b.vdim ? x[b.v_off + h * b.vdim + c] : 1.0f;
        if (!ONE) gn = G[(size_t)(row0 + n) * b.heads + h];
    };
    fetch(0);
    if (ONE) {
        if (KIND == REC_MLSTM) {
            float i, f;
            mlstm_gates(b, P + (size_t)row0 * ldp, h, i, f);
            const float m0 = mstate[(size_t)slot * b.heads + h], m = fmaxf(f + m0, i);
            gn = make_float4(fminf(f + m0 - m, 0.0f), i - m + logf(b.qscale), m, 0.0f);
        } else delta_gates(b, P + (size_t)row0 * ldp, h, gn.x, gn.y);
    }
    for (int n = 0; n < len; n++) {
        const int buf = n & 1;
#pragma unroll
        for (int j = 0; j < NPF; j++) { const int i = threadIdx.x + j * 256; if (i < DP) { sq[buf][i] = qn[j]; sk[buf][i] = kn[j]; } }
        const float v = vn, dec = expf(gn.x), w = KIND == REC_MLSTM ? expf(gn.y) : gn.y;
        __syncthreads();
        if (n + 1 < len) fetch(n + 1);
        float o = 0.0f;
        if (KIND == REC_MLSTM) {
            const float wv = w * v;
#pragma unroll
            for (int j = 0; j < RPT; j++) {
                S[j] = fmaf(dec, S[j], sk[buf][wid * RPT + j] * wv);
                o = fmaf(S[j], sq[buf][wid * RPT + j], o);
            }
            part[buf][0][wid][lane] = o;
            __syncthreads();
            if (wid == 0 && ok) {
                o = 0.0f;
#pragma unroll
                for (int k = 0; k < 8; k++) o += part[buf][0][k][lane];
                O[(size_t)(row0 + n) * (b.heads * b.vx) + h * b.vx + c] = o;
            }
        } else {
            float r = 0.0f, kq = 0.0f, k2 = 0.0f, q2 = 0.0f;
#pragma unroll
            for (int j = 0; j < RPT; j++) {
                const float kk = sk[buf][wid * RPT + j], qq = sq[buf][wid * RPT + j];
                S[j] *= dec;
                r = fmaf(S[j], kk, r);
                o = fmaf(S[j], qq, o);
                kq = fmaf(kk, qq, kq);
                if (ONE) { k2 = fmaf(kk, kk, k2); q2 = fmaf(qq, qq, q2); }
            }
            part[buf][0][wid][lane] = r;
            part[buf][1][wid][lane] = o;
            if (lane == 0) { skq[buf][0][wid] = kq; skq[buf][1][wid] = k2; skq[buf][2][wid] = q2; }
            __syncthreads();
            r = o = kq = k2 = q2 = 0.0f;
#pragma unroll
            for (int k = 0; k < 8; k++) {
                r += part[buf][0][k][lane]; o += part[buf][1][k][lane]; kq += skq[buf][0][k];
                if (ONE) { k2 += skq[buf][1][k]; q2 += skq[buf][2][k]; }
            }
            float u, ks = 1.0f;
            if (ONE) {
                ks = 1.0f / sqrtf(k2 + 1e-6f);
                const float qs = b.qscale / sqrtf(q2 + 1e-6f);
                r *= ks; o *= qs; kq *= ks * qs;
            }
            u = w * (v - r);
            const float ku = ks * u;
#pragma unroll
            for (int j = 0; j < RPT; j++) S[j] = fmaf(sk[buf][wid * RPT + j], ku, S[j]);
            if (wid == 0 && ok) O[(size_t)(row0 + n) * (b.heads * b.vx) + h * b.vx + c] = fmaf(kq, u, o);
        }
    }
    if (t.slots[slot].stopped) return;
#pragma unroll
    for (int j = 0; j < RPT; j++) { const int i = wid * RPT + j; if (ok && i < b.dim) gs[(size_t)i * b.vxp + c] = S[j]; }
}

// Output of a (row, head), a warp each: mLSTM o = O / (max(|n . q|, exp(-m)) + 1e-6); both: o / sqrt(mean(o^2) + eps) * norm * gate
// (mLSTM: logistic, delta rule: silu) -> out-projection operand.  G null (mLSTM, every segment one row): the running maximum is formed here and moved on.
template <typename OT, int KIND>
__global__ void __launch_bounds__(128) k_rec_post(PassTables t, RecBranch b, const float* __restrict__ O, const float4* __restrict__ G, float* __restrict__ mstate,
                                                  const float* __restrict__ P, int ldp, OT* __restrict__ out, int ld_out) {
    const int r = blockIdx.x, lane = threadIdx.x & 31, wid = threadIdx.x >> 5, nw = blockDim.x >> 5;
    for (int h = blockIdx.y * nw + wid; h < b.heads; h += gridDim.y * nw) {
        const float* o = O + (size_t)r * (b.heads * b.vx) + h * b.vx;
        float dn = 1.0f;
        if (KIND == REC_MLSTM) {
            float m;
            if (G) m = G[(size_t)r * b.heads + h].z;
            else {
                const int slot = t.seg_slot[t.row_seg[r]];
                float i, f;
                mlstm_gates(b, P + (size_t)r * ldp, h, i, f);
                float* ms = mstate + (size_t)slot * b.heads + h;
                m = fmaxf(f + *ms, i);
                __syncwarp();
                if (lane == 0 && !t.slots[slot].stopped) *ms = m;
            }
            dn = 1.0f / (fmaxf(fabsf(o[b.vdim]), expf(-m)) + 1e-6f);
        }
        float ss = 0.0f;
        for (int i = lane; i < b.vdim; i += 32) { const float v = o[i] * dn; ss += v * v; }
        const float sc = dn * b.out_scale / sqrtf(warp_sum(ss) / (float)b.vdim + b.eps);
        const float* w = b.norm + (KIND == REC_MLSTM ? h * b.vdim : 0);
        const float* g = P + (size_t)r * ldp + b.g_off + h * b.vdim;
        for (int i = lane; i < b.vdim; i += 32) out[(size_t)r * ld_out + b.a_off + h * b.vdim + i] = cvt<OT>(o[i] * sc * w[i] * (KIND == REC_MLSTM ? sigmoidf_(g[i]) : silu_(g[i])));
    }
}

// ================================================================================================ chunks on tensor cores
// With b_t = the sum of log decays from the chunk's start to row t, S0 the state before the chunk and rows t, s of one chunk of C rows:
//     o_t   = exp(b_t) S0^T q_t + sum_{s <= t} exp(b_t - b_s + w_s) (q_t . k_s) u_s
//     S_end = exp(b_L) S0 + sum_s exp(b_L - b_s + w_s) k_s u_s^T
// mLSTM: u = [v | 1].  Delta rule (w = 0): u = beta (v - S^T k) makes U = U' - W S0 with (I + A) [W | U'] = [beta e^b K | beta V], A the strictly
// lower part of beta_t exp(b_t - b_s) k_t . k_s -- a triangular system per chunk that does not know S0 (k_delta_wy, all chunks at once).
//   k_rec_prep    q, k (unit length for the delta rule) and v as planes, heads padded to multiples of 16
//   k_delta_wy    W (planes) and U' (fp32, over v) of every chunk
//   k_rec_scan    walks the chunks of a (segment, head, 16 columns): leaves the state before each chunk as planes, U as planes, the slot's state
//   k_rec_out     the rows of every chunk, all chunks at once
// Planes: [2][rows][heads * width], hi then lo, `ps` elements apart.
template <int KIND>
__global__ void __launch_bounds__(256) k_rec_prep(RecBranch b, const float* __restrict__ X, int ldx, bf16* __restrict__ QP, bf16* __restrict__ KP, size_t ps_qk,
                                                  bf16* __restrict__ VPn, size_t ps_v) {
    const int r = blockIdx.x, lane = threadIdx.x & 31, wid = threadIdx.x >> 5, nw = blockDim.x >> 5;
    const float* x = X + (size_t)r * ldx;
    const int units = 2 * b.kv_heads + b.heads;
    for (int u = blockIdx.y * nw + wid; u < units; u += gridDim.y * nw) {
        if (u >= 2 * b.kv_heads) {           // values, and the column of ones of a normaliser
            const int h = u - 2 * b.kv_heads;
            bf16* d = VPn + ((size_t)r * b.heads + h) * b.vp;
            for (int i = lane * 2; i < b.vp; i += 64) {
                float v[2];
#pragma unroll
                for (int e = 0; e < 2; e++) v[e] = i + e < b.vdim ? x[b.v_off + h * b.vdim + i + e] : i + e < b.vx ? 1.0f : 0.0f;
                uint32_t hi, lo;
                split2_pack(v[0], v[1], hi, lo);
                *reinterpret_cast<uint32_t*>(d + i) = hi;
                *reinterpret_cast<uint32_t*>(d + ps_v + i) = lo;
            }
            continue;
        }
        const bool is_q = u < b.kv_heads;
        const int hk = is_q ? u : u - b.kv_heads;
        const float* v = x + (is_q ? b.q_off : b.k_off) + hk * b.dim;
        bf16* d = (is_q ? QP : KP) + ((size_t)r * b.kv_heads + hk) * b.dp;
        float sc = 1.0f;
        if (KIND == REC_DELTA) {
            float ss = 0.0f;
            for (int i = lane; i < b.dim; i += 32) ss += v[i] * v[i];
            sc = (is_q ? b.qscale : 1.0f) / sqrtf(warp_sum(ss) + 1e-6f);
        }
        for (int i = lane * 2; i < b.dp; i += 64) {
            uint32_t hi, lo;
            split2_pack(i < b.dim ? v[i] * sc : 0.0f, i + 1 < b.dim ? v[i + 1] * sc : 0.0f, hi, lo);
            *reinterpret_cast<uint32_t*>(d + i) = hi;
            *reinterpret_cast<uint32_t*>(d + ps_qk + i) = lo;
        }
    }
}

// planes of rows [row0, row0 + C) (rows from L on: zeros), columns [0, w) of a head -> shared memory [2][C][ld]; w a multiple of 8
// (a warp covers 1, 2 or 4 rows at a time)
__device__ __forceinline__ void rec_stage(uint32_t dst, int ld, int C, const bf16* __restrict__ src, size_t ps, size_t row_ld, int L, int w) {
    const int per = w >> 3, sh = per <= 8 ? 3 : per <= 16 ? 4 : 5, lane = threadIdx.x & 31, piece = lane & ((1 << sh) - 1), rows = 32 >> sh;
    for (int r = (threadIdx.x >> 5) * rows + (lane >> sh); r < 2 * C; r += (blockDim.x >> 5) * rows) {
        const int pl = r >= C, rr = r - pl * C;
        const bool on = rr < L;
        for (int c = piece; c < per; c += 1 << sh)
            sa_cp16(dst + (uint32_t)((r * ld + c * 8) * 2), on ? (const void*)(src + pl * ps + (size_t)rr * row_ld + c * 8) : (const void*)src, on);
    }
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// grid (chunks, heads), 256 threads.  The chunk's A from k's planes on tensor cores; T = (I + A)^-1 in fp32 by blocks of 16 rows -- the diagonal blocks by
// forward substitution (a thread per column), T_ij = -T_ii sum_k A_ik T_kj below them, one block diagonal after the other; then W = (T diag(beta e^b)) K
// and U' = (T diag(beta)) V on tensor cores, T's scaled columns split into planes on the way into the A fragments.
// VPn: planes of v; U' goes to X's v columns.
template <int C>
__global__ void __launch_bounds__(256, 2) k_delta_wy(PassTables t, RecBranch b, int S, const bf16* __restrict__ KP, size_t ps_qk, const bf16* __restrict__ VPn, size_t ps_v,
                                                     const float4* __restrict__ G, const float2* __restrict__ Bp, float* __restrict__ X, int ldx, bf16* __restrict__ WP, size_t ps_w) {
    extern __shared__ __align__(16) unsigned char rc_raw[];
    __shared__ float sbeta[C], sbeb[C], sbh[C], sbl[C];
    constexpr int LA = C + 4, NB = C / 16;
    int seg, ck;
    if (!ret_find_chunk(t, S, C, blockIdx.x, seg, ck)) return;
    const int h = blockIdx.y, hk = h / (b.heads / b.kv_heads), LK = b.dp + 8, LV = b.vp + 8;
    const int row0 = t.seg_row0[seg] + ck * C, L = min(C, t.seg_len[seg] - ck * C);
    float* sA = reinterpret_cast<float*>(rc_raw);                // [C][LA]
    float* sT = sA + C * LA;                                     // [C][LA]; block (i, j) also holds sum_k A_ik T_kj on its way to T_ij
    bf16* sk = reinterpret_cast<bf16*>(sT + C * LA);             // [2][C][max(LK, LV)]: k, then v
    const uint32_t sk_a = (uint32_t)__cvta_generic_to_shared(sk);
    rec_stage(sk_a, LK, C, KP + ((size_t)row0 * b.kv_heads + hk) * b.dp, ps_qk, (size_t)b.kv_heads * b.dp, L, b.dp);
    cp_commit();
    for (int r = threadIdx.x; r < C; r += 256) {
        float2 bb = make_float2(0.0f, 0.0f);
        float be = 0.0f;
        if (r < L) { bb = Bp[(size_t)(row0 + r) * b.heads + h]; be = G[(size_t)(row0 + r) * b.heads + h].y; }
        sbeta[r] = be; sbh[r] = bb.x; sbl[r] = bb.y; sbeb[r] = be * expf(bb.x + bb.y);
    }
    cp_wait<0>();
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gq = lane >> 2, tq = lane & 3;
    for (int tile = warp; tile < NB * NB; tile += 8) {
        const int mt = tile / NB, nt = tile % NB;
        if (nt > mt) continue;                                   // above the diagonal nothing is read
        float acc[2][4] = {}, acx[2][4] = {};
        for (int kk = 0; kk < b.dp / 16; kk++) {
            uint32_t a[2][4], w[2][4];
#pragma unroll
            for (int pl = 0; pl < 2; pl++) {
                sa_ldsm_x4(sk_a + (uint32_t)(((pl * C + mt * 16 + (lane & 15)) * LK + kk * 16 + (lane >> 4) * 8) * 2), a[pl][0], a[pl][1], a[pl][2], a[pl][3]);
                sa_ldsm_x4(sk_a + (uint32_t)(((pl * C + nt * 16 + (lane & 7) + (lane >> 4) * 8) * LK + kk * 16 + ((lane >> 3) & 1) * 8) * 2), w[pl][0], w[pl][1], w[pl][2], w[pl][3]);
            }
#pragma unroll
            for (int n = 0; n < 2; n++) {
                sa_mma(acc[n], a[0], w[0][2 * n], w[0][2 * n + 1]);
                sa_mma(acx[n], a[0], w[1][2 * n], w[1][2 * n + 1]);
                sa_mma(acx[n], a[1], w[0][2 * n], w[0][2 * n + 1]);
            }
        }
#pragma unroll
        for (int n = 0; n < 2; n++)
#pragma unroll
            for (int x = 0; x < 4; x++) {
                const int tt = mt * 16 + gq + (x >= 2 ? 8 : 0), ss = nt * 16 + n * 8 + tq * 2 + (x & 1);
                sA[tt * LA + ss] = (ss < tt && tt < L) ? sbeta[tt] * expf((sbh[tt] - sbh[ss]) + (sbl[tt] - sbl[ss])) * (acc[n][x] + acx[n][x]) : 0.0f;
            }
    }
    __syncthreads();
    if (threadIdx.x < C) {                                       // diagonal blocks
        const int b0 = (threadIdx.x >> 4) * 16, col = threadIdx.x & 15;
        float x[16];
#pragma unroll
        for (int r = 0; r < 16; r++) {
            float a0 = r == col ? 1.0f : 0.0f;
#pragma unroll
            for (int q = 0; q < r; q++) a0 = fmaf(-sA[(b0 + r) * LA + b0 + q], x[q], a0);
            x[r] = a0;
            sT[(b0 + r) * LA + b0 + col] = a0;
        }
    }
    __syncthreads();
#pragma unroll
    for (int d = 1; d < NB; d++) {                               // blocks (j + d, j)
        const int r = threadIdx.x >> 4, c = threadIdx.x & 15;
#pragma unroll
        for (int j = 0; j + d < NB; j++) {
            const int i = j + d;
            float a0 = 0.0f, a1 = 0.0f;
            for (int k = j * 16; k < i * 16; k += 2) { a0 = fmaf(sA[(i * 16 + r) * LA + k], sT[k * LA + j * 16 + c], a0); a1 = fmaf(sA[(i * 16 + r) * LA + k + 1], sT[(k + 1) * LA + j * 16 + c], a1); }
            sT[(i * 16 + r) * LA + j * 16 + c] = a0 + a1;
        }
        __syncthreads();
        float v[NB];
#pragma unroll
        for (int j = 0; j + d < NB; j++) {
            const int i = j + d;
            float a0 = 0.0f;
#pragma unroll
            for (int k = 0; k < 16; k++) a0 = fmaf(sT[(i * 16 + r) * LA + i * 16 + k], sT[(i * 16 + k) * LA + j * 16 + c], a0);
            v[j] = -a0;
        }
        __syncthreads();
#pragma unroll
        for (int j = 0; j + d < NB; j++) sT[((j + d) * 16 + r) * LA + j * 16 + c] = v[j];
        __syncthreads();
    }
    const int mt = warp % NB, part = warp / NB, n_part = 8 / NB;  // this warp's 16 rows and its share of the columns
#pragma unroll
    for (int pass = 0; pass < 2; pass++) {                       // W, then U'
        const int LB = pass ? LV : LK, nw16 = (pass ? b.vp : b.dp) / 16;
        if (pass) {
            __syncthreads();                                     // k's planes have been read
            rec_stage(sk_a, LV, C, VPn + ((size_t)row0 * b.heads + h) * b.vp, ps_v, (size_t)b.heads * b.vp, L, b.vp);
            cp_commit();
        }
        uint32_t ah[NB][4], al[NB][4];
#pragma unroll
        for (int kk = 0; kk < NB; kk++) {
            if (kk > mt) continue;
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int rr = mt * 16 + gq + (e & 1) * 8, c = kk * 16 + tq * 2 + (e >> 1) * 8;
                const float* sc = pass ? sbeta : sbeb;
                const bool low = kk < mt || c <= rr, low1 = kk < mt || c + 1 <= rr;
                split2_pack(low ? sT[rr * LA + c] * sc[c] : 0.0f, low1 ? sT[rr * LA + c + 1] * sc[c + 1] : 0.0f, ah[kk][e], al[kk][e]);
            }
        }
        if (pass) { cp_wait<0>(); __syncthreads(); }
        for (int n2 = part; n2 < nw16; n2 += n_part) {
            float acc[2][4] = {}, acx[2][4] = {};
#pragma unroll
            for (int kk = 0; kk < NB; kk++) {
                if (kk > mt) continue;
                uint32_t w[2][4];
#pragma unroll
                for (int pl = 0; pl < 2; pl++)
                    sa_ldsm_x4_t(sk_a + (uint32_t)(((pl * C + kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LB + n2 * 16 + (lane >> 4) * 8) * 2), w[pl][0], w[pl][1], w[pl][2], w[pl][3]);
#pragma unroll
                for (int n = 0; n < 2; n++) {
                    sa_mma(acc[n], ah[kk], w[0][2 * n], w[0][2 * n + 1]);
                    sa_mma(acx[n], ah[kk], w[1][2 * n], w[1][2 * n + 1]);
                    sa_mma(acx[n], al[kk], w[0][2 * n], w[0][2 * n + 1]);
                }
            }
#pragma unroll
            for (int n = 0; n < 2; n++)
#pragma unroll
                for (int hf = 0; hf < 2; hf++) {
                    const int rr = mt * 16 + gq + hf * 8, c = n2 * 16 + n * 8 + tq * 2;
                    if (rr >= L) continue;
                    const float v0 = acc[n][2 * hf] + acx[n][2 * hf], v1 = acc[n][2 * hf + 1] + acx[n][2 * hf + 1];
                    if (pass == 0) {
                        uint32_t hi, lo;
                        split2_pack(v0, v1, hi, lo);
                        bf16* wd = WP + ((size_t)(row0 + rr) * b.heads + h) * b.dp + c;
                        *reinterpret_cast<uint32_t*>(wd) = hi;
                        *reinterpret_cast<uint32_t*>(wd + ps_w) = lo;
                    } else {
                        float* xv = X + (size_t)(row0 + rr) * ldx + b.v_off + h * b.vdim + c;
                        if (c < b.vdim) xv[0] = v0;
                        if (c + 1 < b.vdim) xv[1] = v1;
                    }
                }
        }
    }
}

// grid (segments, heads, groups of 16 state columns), 256 threads.  The slice of the state lives in the accumulators of S = K^T U (rows = dim, eight
// warps x MT tiles of 16); chunk by chunk: its planes to shared memory (and to SP for k_rec_out), the delta rule's U = U' - W S0, then
// S <- exp(b_L) S + K^T (exp(b_L - b_s + w_s) u_s).  K and W of the next chunk arrive while the current one is computed.
// SP [chunks][heads][2][dp][vp]; UP: planes of u (delta rule: written here).
template <int KIND, int C, int MT>
__global__ void __launch_bounds__(256) k_rec_scan(PassTables t, RecBranch b, const bf16* __restrict__ KP, size_t ps_qk, const bf16* __restrict__ WP, size_t ps_w,
                                                  const float4* __restrict__ G, const float2* __restrict__ Bp, const float* __restrict__ X, int ldx, bf16* __restrict__ UP, size_t ps_v,
                                                  bf16* __restrict__ SP, float* __restrict__ state) {
    extern __shared__ __align__(16) unsigned char rc_raw[];
    constexpr int LS = REC_VS + 8;
    const int LK = b.dp + 8;
    bf16* sk = reinterpret_cast<bf16*>(rc_raw);                              // [2 stages][2][C][LK]
    bf16* sw = sk + 4 * C * LK;                                              // the same for W (delta rule)
    bf16* sS = sw + (KIND == REC_DELTA ? 4 * C * LK : 0);                    // [2][dp][LS]
    bf16* sU = sS + 2 * b.dp * LS;                                           // [2][C][LS]
    __shared__ float sbh[2][C], sbl[2][C], slw[2][C];
    const int seg = blockIdx.x, h = blockIdx.y, hk = h / (b.heads / b.kv_heads), c0 = blockIdx.z * REC_VS;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gq = lane >> 2, tq = lane & 3;
    const int slot = t.seg_slot[seg], len = t.seg_len[seg], n_ck = (len + C - 1) / C;
    int first = 0;
    for (int s = 0; s < seg; s++) first += (t.seg_len[s] + C - 1) / C;
    float* gs = state + ((size_t)slot * b.heads + h) * (size_t)b.dim * b.vxp;
    const uint32_t sk_a = (uint32_t)__cvta_generic_to_shared(sk), sw_a = (uint32_t)__cvta_generic_to_shared(sw);
    const uint32_t sS_a = (uint32_t)__cvta_generic_to_shared(sS), sU_a = (uint32_t)__cvta_generic_to_shared(sU);
    const int nmt = b.dp / 16;                                               // tiles of 16 state rows; warp w owns w, w + 8, ...
    float acc[MT][2][4];
#pragma unroll
    for (int i = 0; i < MT; i++)
#pragma unroll
        for (int n = 0; n < 2; n++)
#pragma unroll
            for (int x = 0; x < 4; x++) {
                const int d = (warp + 8 * i) * 16 + gq + (x >= 2 ? 8 : 0), c = c0 + n * 8 + tq * 2 + (x & 1);
                acc[i][n][x] = (d < b.dim && c < b.vx) ? gs[(size_t)d * b.vxp + c] : 0.0f;
            }
    auto stage = [&](int st, int ck) {
        const int row0 = t.seg_row0[seg] + ck * C, L = min(C, len - ck * C);
        rec_stage(sk_a + (uint32_t)(st * 2 * C * LK * 2), LK, C, KP + ((size_t)row0 * b.kv_heads + hk) * b.dp, ps_qk, (size_t)b.kv_heads * b.dp, L, b.dp);
        if (KIND == REC_DELTA) rec_stage(sw_a + (uint32_t)(st * 2 * C * LK * 2), LK, C, WP + ((size_t)row0 * b.heads + h) * b.dp, ps_w, (size_t)b.heads * b.dp, L, b.dp);
        cp_commit();
    };
    // gates of one chunk and this thread's elements of u of the next one wait in registers: for the delta rule those of its U tile (warp -> 16 rows x 8
    // columns), otherwise rows of [v | 1]
    float2 gb = make_float2(0.0f, 0.0f);
    float glw = 0.0f, un[4];
    const int ut = (warp >> 1) * 16 + gq, uc = c0 + (warp & 1) * 8 + tq * 2;
    const bool has_u = (warp >> 1) * 16 < C;
    auto fetch_gates = [&](int ck) {
        const int r = ck * C + (int)threadIdx.x;
        if ((int)threadIdx.x >= C) return;
        gb = make_float2(0.0f, 0.0f);
        glw = 0.0f;
        if (r < len) { const size_t at = (size_t)(t.seg_row0[seg] + r) * b.heads + h; gb = Bp[at]; if (KIND == REC_MLSTM) glw = G[at].y; }
    };
    auto put_gates = [&](int st) { if ((int)threadIdx.x < C) { sbh[st][threadIdx.x] = gb.x; sbl[st][threadIdx.x] = gb.y; slw[st][threadIdx.x] = glw; } };
    auto fetch_u = [&](int ck) {
#pragma unroll
        for (int x = 0; x < 4; x++) {
            const int r = ck * C + ut + (x >= 2 ? 8 : 0), c = uc + (x & 1);
            un[x] = 0.0f;
            if (has_u && r < len) un[x] = c < b.vdim ? X[(size_t)(t.seg_row0[seg] + r) * ldx + b.v_off + h * b.vdim + c] : (c < b.vx ? 1.0f : 0.0f);
        }
    };
    stage(0, 0);
    fetch_gates(0);
    put_gates(0);
    fetch_gates(1);
    fetch_u(0);
    for (int ck = 0; ck < n_ck; ck++) {
        const int st = ck & 1, row0 = t.seg_row0[seg] + ck * C, L = min(C, len - ck * C);
        bf16* sp = SP + ((size_t)(first + ck) * b.heads + h) * 2 * b.dp * b.vp + c0;
#pragma unroll
        for (int i = 0; i < MT; i++) {
            if (warp + 8 * i >= nmt) continue;
#pragma unroll
            for (int n = 0; n < 2; n++)
#pragma unroll
                for (int hf = 0; hf < 2; hf++) {
                    const int d = (warp + 8 * i) * 16 + gq + hf * 8, c = n * 8 + tq * 2;
                    uint32_t hi, lo;
                    split2_pack(acc[i][n][2 * hf], acc[i][n][2 * hf + 1], hi, lo);
                    *reinterpret_cast<uint32_t*>(sS + d * LS + c) = hi;
                    *reinterpret_cast<uint32_t*>(sS + (b.dp + d) * LS + c) = lo;
                    *reinterpret_cast<uint32_t*>(sp + (size_t)d * b.vp + c) = hi;
                    *reinterpret_cast<uint32_t*>(sp + ((size_t)b.dp + d) * b.vp + c) = lo;
                }
        }
        float u[4] = {un[0], un[1], un[2], un[3]};
        cp_wait<0>();
        __syncthreads();
        if (ck + 1 < n_ck) {                                                 // its last readers passed the barrier above
            stage(st ^ 1, ck + 1);
            put_gates(st ^ 1);
            fetch_gates(ck + 2);
            fetch_u(ck + 1);
        }
        const float bLh = sbh[st][L - 1], bLl = sbl[st][L - 1];
        if (has_u) {
            if (KIND == REC_DELTA) {
                float ws[3][4] = {};
                const int m0 = (warp >> 1) * 16, n8 = (warp & 1) * 8;
                for (int kk = 0; kk < nmt; kk++) {
                    uint32_t a[2][4], s0[2], s1[2];
#pragma unroll
                    for (int pl = 0; pl < 2; pl++)
                        sa_ldsm_x4(sw_a + (uint32_t)((((st * 2 + pl) * C + m0 + (lane & 15)) * LK + kk * 16 + (lane >> 4) * 8) * 2), a[pl][0], a[pl][1], a[pl][2], a[pl][3]);
                    // hi and lo of the state's 16 rows at once: lanes 0 - 15 address the hi plane, 16 - 31 the lo plane
                    sa_ldsm_x4_t(sS_a + (uint32_t)((((lane >> 4) * b.dp + kk * 16 + (lane & 15)) * LS + n8) * 2), s0[0], s0[1], s1[0], s1[1]);
                    sa_mma(ws[0], a[0], s0[0], s0[1]);
                    sa_mma(ws[1], a[0], s1[0], s1[1]);
                    sa_mma(ws[2], a[1], s0[0], s0[1]);
                }
#pragma unroll
                for (int x = 0; x < 4; x++) u[x] = ut + (x >= 2 ? 8 : 0) < L ? u[x] - (ws[0][x] + (ws[1][x] + ws[2][x])) : 0.0f;
            }
#pragma unroll
            for (int hf = 0; hf < 2; hf++) {
                const int r = ut + hf * 8;
                uint32_t hi, lo;
                if (KIND == REC_DELTA && r < L) {
                    bf16* ud = UP + ((size_t)(row0 + r) * b.heads + h) * b.vp + uc;
                    split2_pack(u[2 * hf], u[2 * hf + 1], hi, lo);
                    *reinterpret_cast<uint32_t*>(ud) = hi;
                    *reinterpret_cast<uint32_t*>(ud + ps_v) = lo;
                }
                const float f = r < L ? expf((bLh - sbh[st][r]) + (bLl - sbl[st][r]) + slw[st][r]) : 0.0f;
                split2_pack(u[2 * hf] * f, u[2 * hf + 1] * f, hi, lo);
                *reinterpret_cast<uint32_t*>(sU + r * LS + uc - c0) = hi;
                *reinterpret_cast<uint32_t*>(sU + (C + r) * LS + uc - c0) = lo;
            }
        }
        __syncthreads();
        const float dec = expf(bLh + bLl);
        float acx[MT][2][4];                                                 // the products with a lo plane
#pragma unroll
        for (int i = 0; i < MT; i++)
#pragma unroll
            for (int n = 0; n < 2; n++)
#pragma unroll
                for (int x = 0; x < 4; x++) { acc[i][n][x] *= dec; acx[i][n][x] = 0.0f; }
#pragma unroll
        for (int kk = 0; kk < C / 16; kk++) {
            uint32_t w[2][4];
#pragma unroll
            for (int pl = 0; pl < 2; pl++)
                sa_ldsm_x4_t(sU_a + (uint32_t)(((pl * C + kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LS + (lane >> 4) * 8) * 2), w[pl][0], w[pl][1], w[pl][2], w[pl][3]);
#pragma unroll
            for (int i = 0; i < MT; i++) {
                if (warp + 8 * i >= nmt) continue;
                uint32_t a[2][4];
#pragma unroll
                for (int pl = 0; pl < 2; pl++)                               // K^T: rows of the tile are columns of k
                    sa_ldsm_x4_t(sk_a + (uint32_t)((((st * 2 + pl) * C + kk * 16 + (lane & 7) + (lane >> 4) * 8) * LK + (warp + 8 * i) * 16 + ((lane >> 3) & 1) * 8) * 2),
                                 a[pl][0], a[pl][1], a[pl][2], a[pl][3]);
#pragma unroll
                for (int n = 0; n < 2; n++) {
                    sa_mma(acc[i][n], a[0], w[0][2 * n], w[0][2 * n + 1]);
                    sa_mma(acx[i][n], a[0], w[1][2 * n], w[1][2 * n + 1]);
                    sa_mma(acx[i][n], a[1], w[0][2 * n], w[0][2 * n + 1]);
                }
            }
        }
#pragma unroll
        for (int i = 0; i < MT; i++)
#pragma unroll
            for (int n = 0; n < 2; n++)
#pragma unroll
                for (int x = 0; x < 4; x++) acc[i][n][x] += acx[i][n][x];
    }
    if (t.slots[slot].stopped) return;
#pragma unroll
    for (int i = 0; i < MT; i++)
#pragma unroll
        for (int n = 0; n < 2; n++)
#pragma unroll
            for (int x = 0; x < 4; x++) {
                const int d = (warp + 8 * i) * 16 + gq + (x >= 2 ? 8 : 0), c = c0 + n * 8 + tq * 2 + (x & 1);
                if (d < b.dim && c < b.vx) gs[(size_t)d * b.vxp + c] = acc[i][n][x];
            }
}

// grid (chunks, heads, groups of VP value columns), 2 C threads: warp w owns the chunk's rows 16 w .. 16 w + 15.  Q K^T and Q S0 are summed over
// the head size in steps of 64 (staged planes of q, k and the state); the scores under the causal decay weights are the A fragments
// of the product with u.
template <int VP, int C>
__global__ void __launch_bounds__(2 * C) k_rec_out(PassTables t, RecBranch b, int kind, int S, const bf16* __restrict__ QP, const bf16* __restrict__ KP, size_t ps_qk,
                                                   const bf16* __restrict__ UP, size_t ps_v, const bf16* __restrict__ SP, const float4* __restrict__ G, const float2* __restrict__ Bp,
                                                   float* __restrict__ O) {
    extern __shared__ __align__(16) unsigned char rc_raw[];
    constexpr int LQ = 64 + 8, LV = VP + 8;
    bf16* sq = reinterpret_cast<bf16*>(rc_raw);              // [2][C][LQ]
    bf16* sk = sq + 2 * C * LQ;                              // [2][C][LQ]
    bf16* ss = sk + 2 * C * LQ;                              // [2][64][LV] state; then [2][C][LV] u
    __shared__ float sbh[C], sbl[C], slw[C];
    int seg, ck;
    if (!ret_find_chunk(t, S, C, blockIdx.x, seg, ck)) return;
    const int h = blockIdx.y, hk = h / (b.heads / b.kv_heads), c0 = blockIdx.z * VP, nc = min(VP, b.vp - c0);       // nc: a multiple of 16
    const int row0 = t.seg_row0[seg] + ck * C, L = min(C, t.seg_len[seg] - ck * C);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gq = lane >> 2, tq = lane & 3;
    const uint32_t sq_a = (uint32_t)__cvta_generic_to_shared(sq), sk_a = (uint32_t)__cvta_generic_to_shared(sk), ss_a = (uint32_t)__cvta_generic_to_shared(ss);
    for (int r = threadIdx.x; r < C; r += 2 * C) {
        float2 bb = make_float2(0.0f, 0.0f);
        float lw = 0.0f;
        if (r < L) { bb = Bp[(size_t)(row0 + r) * b.heads + h]; if (kind == REC_MLSTM) lw = G[(size_t)(row0 + r) * b.heads + h].y; }
        sbh[r] = bb.x; sbl[r] = bb.y; slw[r] = lw;
    }
    float sc[C / 8][4], o[VP / 8][4];
#pragma unroll
    for (int n = 0; n < C / 8; n++) { sc[n][0] = sc[n][1] = sc[n][2] = sc[n][3] = 0.0f; }
#pragma unroll
    for (int n = 0; n < VP / 8; n++) { o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.0f; }
    const bf16* sp = SP + ((size_t)blockIdx.x * b.heads + h) * 2 * b.dp * b.vp + c0;
    for (int d0 = 0; d0 < b.dp; d0 += 64) {
        const int dw = min(64, b.dp - d0);
        if (d0) __syncthreads();
        rec_stage(sq_a, LQ, C, QP + ((size_t)row0 * b.kv_heads + hk) * b.dp + d0, ps_qk, (size_t)b.kv_heads * b.dp, L, dw);
        rec_stage(sk_a, LQ, C, KP + ((size_t)row0 * b.kv_heads + hk) * b.dp + d0, ps_qk, (size_t)b.kv_heads * b.dp, L, dw);
        rec_stage(ss_a, LV, 64, sp + (size_t)d0 * b.vp, (size_t)b.dp * b.vp, b.vp, dw, nc);
        cp_commit();
        cp_wait<0>();
        __syncthreads();
        for (int kk = 0; kk < dw / 16; kk++) {
            uint32_t a[2][4];
#pragma unroll
            for (int pl = 0; pl < 2; pl++)
                sa_ldsm_x4(sq_a + (uint32_t)(((pl * C + warp * 16 + (lane & 15)) * LQ + kk * 16 + (lane >> 4) * 8) * 2), a[pl][0], a[pl][1], a[pl][2], a[pl][3]);
#pragma unroll
            for (int n2 = 0; n2 < C / 16; n2++) {
                if (n2 > warp) continue;                         // keys after this warp's rows
                uint32_t w[2][4];
#pragma unroll
                for (int pl = 0; pl < 2; pl++)
                    sa_ldsm_x4(sk_a + (uint32_t)(((pl * C + n2 * 16 + (lane & 7) + (lane >> 4) * 8) * LQ + kk * 16 + ((lane >> 3) & 1) * 8) * 2), w[pl][0], w[pl][1], w[pl][2], w[pl][3]);
#pragma unroll
                for (int n = 0; n < 2; n++) {
                    sa_mma(sc[2 * n2 + n], a[0], w[0][2 * n], w[0][2 * n + 1]);
                    sa_mma(sc[2 * n2 + n], a[0], w[1][2 * n], w[1][2 * n + 1]);
                    sa_mma(sc[2 * n2 + n], a[1], w[0][2 * n], w[0][2 * n + 1]);
                }
            }
#pragma unroll
            for (int n2 = 0; n2 < VP / 16; n2++) {
                if (n2 * 16 >= nc) continue;
                uint32_t w[2][4];
#pragma unroll
                for (int pl = 0; pl < 2; pl++)
                    sa_ldsm_x4_t(ss_a + (uint32_t)(((pl * 64 + kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LV + n2 * 16 + (lane >> 4) * 8) * 2), w[pl][0], w[pl][1], w[pl][2], w[pl][3]);
#pragma unroll
                for (int n = 0; n < 2; n++) {
                    sa_mma(o[2 * n2 + n], a[0], w[0][2 * n], w[0][2 * n + 1]);
                    sa_mma(o[2 * n2 + n], a[0], w[1][2 * n], w[1][2 * n + 1]);
                    sa_mma(o[2 * n2 + n], a[1], w[0][2 * n], w[0][2 * n + 1]);
                }
            }
        }
    }
    __syncthreads();
    rec_stage(ss_a, LV, C, UP + ((size_t)row0 * b.heads + h) * b.vp + c0, ps_v, (size_t)b.heads * b.vp, L, nc);
    cp_commit();
    const int t_lo = warp * 16 + gq, t_hi = t_lo + 8;
    const float g_lo = expf(sbh[t_lo] + sbl[t_lo]), g_hi = expf(sbh[t_hi] + sbl[t_hi]);
#pragma unroll
    for (int n = 0; n < VP / 8; n++) { o[n][0] *= g_lo; o[n][1] *= g_lo; o[n][2] *= g_hi; o[n][3] *= g_hi; }
#pragma unroll
    for (int n = 0; n < C / 8; n++)
#pragma unroll
        for (int x = 0; x < 4; x++) {
            const int tt = x >= 2 ? t_hi : t_lo, s = n * 8 + tq * 2 + (x & 1);
            sc[n][x] = s <= tt ? sc[n][x] * expf((sbh[tt] - sbh[s]) + (sbl[tt] - sbl[s]) + slw[s]) : 0.0f;
        }
    cp_wait<0>();
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < C / 16; kk++) {
        if (kk > warp) continue;
        uint32_t a[2][4];
        split2_pack(sc[2 * kk][0], sc[2 * kk][1], a[0][0], a[1][0]);
        split2_pack(sc[2 * kk][2], sc[2 * kk][3], a[0][1], a[1][1]);
        split2_pack(sc[2 * kk + 1][0], sc[2 * kk + 1][1], a[0][2], a[1][2]);
        split2_pack(sc[2 * kk + 1][2], sc[2 * kk + 1][3], a[0][3], a[1][3]);
#pragma unroll
        for (int n2 = 0; n2 < VP / 16; n2++) {
            if (n2 * 16 >= nc) continue;
            uint32_t w[2][4];
#pragma unroll
            for (int pl = 0; pl < 2; pl++)
                sa_ldsm_x4_t(ss_a + (uint32_t)(((pl * C + kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LV + n2 * 16 + (lane >> 4) * 8) * 2), w[pl][0], w[pl][1], w[pl][2], w[pl][3]);
#pragma unroll
            for (int n = 0; n < 2; n++) {
                sa_mma(o[2 * n2 + n], a[0], w[0][2 * n], w[0][2 * n + 1]);
                sa_mma(o[2 * n2 + n], a[0], w[1][2 * n], w[1][2 * n + 1]);
                sa_mma(o[2 * n2 + n], a[1], w[0][2 * n], w[0][2 * n + 1]);
            }
        }
    }
#pragma unroll
    for (int n = 0; n < VP / 8; n++)
#pragma unroll
        for (int x = 0; x < 4; x++) {
            const int r = x >= 2 ? t_hi : t_lo, c = c0 + n * 8 + tq * 2 + (x & 1);
            if (n * 8 < nc && r < L && c < b.vx) O[(size_t)(row0 + r) * (b.heads * b.vx) + h * b.vx + c] = o[n][x];
        }
}

// ================================================================================================ selective scan
struct SsmBranch {
    int inner, state, dt_rank;
    int z_off, a_off;                        // gate columns in the projection buffer; columns of the output in the out-projection operand
    const float *A_log, *D;                  // [inner][state], [inner]
    float out_scale;
};
// Walks the rows of a segment for 128 / LANES channels.  Threads 0 .. 127 scan: LANES neighbouring ones share a channel, KS of its states in each
// thread's registers, so the chain per row is one multiply-add per state.  The other SSM_SERVE threads serve them, a tile of TILE rows ahead and one behind: step
// sizes and inputs, B and C of the next tile into shared memory, outputs of the previous tile out of it (one barrier per tile).
// XC [R][inner]: input behind its convolution; DT [R][inner]: step sizes before the softplus; BC [R][ld_bc]: columns dt_rank.. are B, then C.
constexpr int SSM_SERVE = 384;
template <typename OT, int LANES, int KS, int TILE>
__global__ void __launch_bounds__(128 + SSM_SERVE, 1) k_ssm_scan(PassTables t, SsmBranch b, const float* __restrict__ XC, const float* __restrict__ DT, const float* __restrict__ BC, int ld_bc,
                                                  const float* __restrict__ P, int ldp, float* __restrict__ state, OT* __restrict__ out, int ld_out) {
    constexpr int NCH = 128 / LANES, NSP = LANES * KS, NE = (TILE * NCH + SSM_SERVE - 1) / SSM_SERVE;      // NE: (row, channel) pairs of a tile per serving thread
    __shared__ __align__(16) float sB[2][TILE][NSP], sC[2][TILE][NSP];
    __shared__ float2 sdx[2][TILE][NCH];                  // {dt, dt x}
    __shared__ float sy[2][TILE][NCH + 1];
    const int s = blockIdx.x, ch0 = blockIdx.y * NCH;
    const int slot = t.seg_slot[s], row0 = t.seg_row0[s], len = t.seg_len[s], n_t = (len + TILE - 1) / TILE;
    if (threadIdx.x >= 128) {
        const int tid = threadIdx.x - 128;
        constexpr int NB = (TILE * NSP + SSM_SERVE - 1) / SSM_SERVE;
        // what a tile needs waits in registers while the tile before it is served: no load is waited for
        float fz[NE], fx[NE], fb[NB], fc[NB], dx[NE], dz[NE], dd[NE];
        int er[NE], ec[NE], br[NB], bn[NB];               // (row, channel) and (row, state) of this thread's entries of a tile; row TILE: none
#pragma unroll
        for (int i = 0; i < NE; i++) {
            const int e = tid + i * SSM_SERVE;
            ec[i] = e % NCH;
            er[i] = e < TILE * NCH && ch0 + ec[i] < b.inner ? e / NCH : TILE;
            dd[i] = er[i] < TILE ? b.D[ch0 + ec[i]] : 0.0f;
        }
#pragma unroll
        for (int i = 0; i < NB; i++) { const int e = tid + i * SSM_SERVE; bn[i] = e % NSP; br[i] = e < TILE * NSP && bn[i] < b.state ? e / NSP : TILE; }
        auto load_fill = [&](int it) {
            const int n0 = it * TILE, nt = min(TILE, len - n0);       // (it >= n_t: nothing is on)
            const float *z = DT + (size_t)(row0 + n0) * b.inner + ch0, *x = XC + (size_t)(row0 + n0) * b.inner + ch0, *p = BC + (size_t)(row0 + n0) * ld_bc + b.dt_rank;
#pragma unroll
            for (int i = 0; i < NE; i++) {
                const bool on = er[i] < nt;
                const int at = er[i] * b.inner + ec[i];
                fz[i] = on ? z[at] : 0.0f;
                fx[i] = on ? x[at] : 0.0f;
            }
#pragma unroll
            for (int i = 0; i < NB; i++) {
                const bool on = br[i] < nt;
                const int at = br[i] * ld_bc + bn[i];
                fb[i] = on ? p[at] : 0.0f;
                fc[i] = on ? p[at + b.state] : 0.0f;
            }
        };
        auto put_fill = [&](int it) {
            const int nt = min(TILE, len - it * TILE), buf = it & 1;
#pragma unroll
            for (int i = 0; i < NB; i++) {
                const int e = tid + i * SSM_SERVE;
                if (e < TILE * NSP) { (&sB[buf][0][0])[e] = fb[i]; (&sC[buf][0][0])[e] = fc[i]; }
            }
#pragma unroll
            for (int i = 0; i < NE; i++) {
                const int e = tid + i * SSM_SERVE;
                float dt = 0.0f;                              // rows behind the segment leave the state as it is
                if (er[i] < nt) dt = sizeof(OT) == 2 ? softplus_series(fz[i]) : softplus_(fz[i]);
                if (e < TILE * NCH) (&sdx[buf][0][0])[e] = make_float2(dt, dt * fx[i]);
            }
        };
        auto load_drain = [&](int it) {
            const int n0 = it * TILE, nt = min(TILE, len - n0);
            const float *x = XC + (size_t)(row0 + n0) * b.inner + ch0, *z = P + (size_t)(row0 + n0) * ldp + b.z_off + ch0;
#pragma unroll
            for (int i = 0; i < NE; i++) {
                const bool on = er[i] < nt;
                dx[i] = on ? x[er[i] * b.inner + ec[i]] : 0.0f;
                dz[i] = on ? z[er[i] * ldp + ec[i]] : 0.0f;
            }
        };
        auto put_drain = [&](int it) {
            const int n0 = it * TILE, nt = min(TILE, len - n0), buf = it & 1;
            OT* o = out + (size_t)(row0 + n0) * ld_out + b.a_off + ch0;
#pragma unroll
            for (int i = 0; i < NE; i++)
                if (er[i] < nt)
                    o[er[i] * ld_out + ec[i]] = cvt<OT>(fmaf(dd[i], dx[i], sy[buf][er[i]][ec[i]]) * (sizeof(OT) == 2 ? __fdividef(dz[i], 1.0f + __expf(-dz[i])) : silu_(dz[i])) * b.out_scale);
        };
        load_fill(0);
        put_fill(0);
        load_fill(1);
        __syncthreads();
        for (int it = 0; it < n_t; it++) {
            if (it + 1 < n_t) { put_fill(it + 1); load_fill(it + 2); }
            if (it > 0) put_drain(it - 1);
            load_drain(it);
            __syncthreads();
        }
        put_drain(n_t - 1);
        return;
    }
    const int ci = threadIdx.x / LANES, li = threadIdx.x % LANES, ch = ch0 + ci;
    const bool ok = ch < b.inner;
    float* gs = state + ((size_t)slot * b.inner + (ok ? ch : 0)) * b.state;
    float S[KS], A[KS];
#pragma unroll
    for (int k = 0; k < KS; k++) {
        const int n = li * KS + k;
        const bool in = ok && n < b.state;
        S[k] = in ? gs[n] : 0.0f;
        A[k] = in ? -expf(b.A_log[(size_t)ch * b.state + n]) : 0.0f;
        if (sizeof(OT) == 2) A[k] *= 1.4426950408889634f;
    }
    __syncthreads();
    // NR rows at a time: their loads and decays are independent of the state, and their read-outs are summed over the channel's lanes together (a lane
    // ends with NR / LANES of them)
    constexpr int NR = KS == 4 ? 8 : 4;
    for (int it = 0; it < n_t; it++) {
        const int nt = min(TILE, len - it * TILE), buf = it & 1;
        for (int r0 = 0; r0 < nt; r0 += NR) {
            float a[NR][KS], w[NR][KS], c[NR][KS], y[NR];
#pragma unroll
            for (int j = 0; j < NR; j++) {
                const float2 dx = sdx[buf][r0 + j][ci];
#pragma unroll
                for (int k = 0; k < KS; k += 4) {
                    const float4 b4 = *reinterpret_cast<const float4*>(&sB[buf][r0 + j][li * KS + k]), c4 = *reinterpret_cast<const float4*>(&sC[buf][r0 + j][li * KS + k]);
                    w[j][k] = dx.y * b4.x; w[j][k + 1] = dx.y * b4.y; w[j][k + 2] = dx.y * b4.z; w[j][k + 3] = dx.y * b4.w;
                    c[j][k] = c4.x; c[j][k + 1] = c4.y; c[j][k + 2] = c4.z; c[j][k + 3] = c4.w;
                }
#pragma unroll
                for (int k = 0; k < KS; k++) {
                    if (sizeof(OT) == 2) asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(a[j][k]) : "f"(dx.x * A[k]));
                    else a[j][k] = expf(dx.x * A[k]);
                }
            }
#pragma unroll
            for (int j = 0; j < NR; j++) {
                y[j] = 0.0f;
#pragma unroll
                for (int k = 0; k < KS; k++) { S[k] = fmaf(a[j][k], S[k], w[j][k]); y[j] = fmaf(S[k], c[j][k], y[j]); }
            }
            int rb = r0;
            bool first = true;                            // among the lanes that end with the same rows
#pragma unroll
            for (int o = LANES / 2, n = NR; o > 0; o >>= 1, n = n > 1 ? n / 2 : 1) {
                if (n > 1) {
                    const bool up = (li & o) != 0;
#pragma unroll
                    for (int j = 0; j < NR / 2; j++) {
                        if (j >= n / 2) continue;
                        const float give = up ? y[j] : y[j + n / 2], keep = up ? y[j + n / 2] : y[j];
                        y[j] = keep + __shfl_xor_sync(0xffffffffu, give, o);
                    }
                    rb += up ? n / 2 : 0;
                } else {
                    y[0] += __shfl_xor_sync(0xffffffffu, y[0], o);
                    first = first && (li & o) == 0;
                }
            }
            constexpr int LEFT = NR > LANES ? NR / LANES : 1;
#pragma unroll
            for (int j = 0; j < LEFT; j++) if (first) sy[buf][rb + j][ci] = y[j];
        }
        __syncthreads();
    }
    if (t.slots[slot].stopped) return;
#pragma unroll
    for (int k = 0; k < KS; k++) { const int n = li * KS + k; if (ok && n < b.state) gs[n] = S[k]; }
}
// columns [0, n) of an fp32 block as a product operand, zero-padded to ld_out
template <typename OT>
__global__ void k_cols_operand(const float* __restrict__ A, int lda, int n, OT* __restrict__ out, int ld_out) {
    const int r = blockIdx.x;
    for (int c = threadIdx.x; c < ld_out; c += blockDim.x) out[(size_t)r * ld_out + c] = cvt<OT>(c < n ? A[(size_t)r * lda + c] : 0.0f);
}

}  // namespace seq
}  // namespace gtb
