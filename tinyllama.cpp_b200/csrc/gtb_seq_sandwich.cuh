// gtb_seq_sandwich.cuh -- mechanisms of the sandwich layer style of the layer-list sequence models (a norm in front of and behind each
// sublayer):
//   * layer norm / RMS norm with a weight (and bias) as an operand producer, and the residual update x += norm_b(sublayer output) that
//     also writes the NEXT sublayer's normalised input
//   * one RMS norm over a whole query / key projection (its scale per row), for softmax attention with qk_norm 3
//   * differential attention: the combination of a head's two score maps, its unit-RMS norm and gate
//   * retention with SiLU-activated inputs, an RMS norm over the concatenated heads and a logistic gate
//   * a sigmoid router whose choice is limited to the best groups of experts, and a router that weights the largest outputs with their own softmax
//   * two branches with out projections and norms of their own, joined in the residual update
//   * a short causal convolution right behind the query and key projections, with the cache append behind it (recurrent mixers: with a bias, silu and
//     an operand copy)
//   * the erf form of GELU as the activation of an ungated feed-forward
// The attention and retention kernels themselves are those of gtb_seq_mixers*.cuh and gtb_seq_kernels.cuh.
//
// Precision follows gtb_seq_kernels.cuh: everything below is fp32 except operands of matrix products (type OT).
#pragma once
#include "gtb_seq_latent.cuh"

namespace gtb {
namespace seq {

constexpr int SW_NORM_LAYER = 2;            // NormArgs::kind of a layer norm (GTB_NORM_LAYER); anything else here: RMS with a plain weight.  b null: no bias

// Sum over the block with ONE barrier: every warp leaves its partial sum in `slot` (32 floats that no other reduction of the kernel uses, so
// nothing has to wait for earlier readers) and every thread adds the partial sums itself, in the same order.
__device__ __forceinline__ float sw_block_sum(float v, float* slot) {
    const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
    v = warp_sum(v);
    if (lane == 0) slot[wid] = v;
    __syncthreads();
    float t = 0.0f;
    for (int w = 0; w < nw; w++) t += slot[w];
    return t;
}
// mean and 1 / sqrt(variance + eps) of a row (layer norm), or 0 and 1 / sqrt(mean square + eps) (RMS); a thread holds the values of columns
// (threadIdx.x + i blockDim.x) * 4 .. + 3 in v[4 i ..].  The mean first, then the squared deviations: no cancellation between two large sums.
// red: 64 floats of shared memory of this call's own.
template <int N4>
__device__ __forceinline__ void sw_stats(const float (&v)[4 * N4], int width, int center, float eps, float* red, float& mean, float& rstd) {
    mean = 0.0f;
    if (center) {
        float s = 0.0f;
#pragma unroll
        for (int i = 0; i < N4; i++)
            if ((int)(threadIdx.x + i * blockDim.x) * 4 < width) s += (v[4 * i] + v[4 * i + 1]) + (v[4 * i + 2] + v[4 * i + 3]);
        mean = sw_block_sum(s, red) / (float)width;
    }
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < N4; i++)
        if ((int)(threadIdx.x + i * blockDim.x) * 4 < width) {
            const float d0 = v[4 * i] - mean, d1 = v[4 * i + 1] - mean, d2 = v[4 * i + 2] - mean, d3 = v[4 * i + 3] - mean;
            ss += (d0 * d0 + d1 * d1) + (d2 * d2 + d3 * d3);
        }
    rstd = 1.0f / sqrtf(sw_block_sum(ss, red + 32) / (float)width + eps);
}

// out = out_scale * norm(x[rows[o]]) as a product operand.  rows: optional gather.
template <typename OT>
__global__ void __launch_bounds__(256) k_norm_rows(const float* __restrict__ x, int width, NormArgs nrm, const int* __restrict__ rows, OT* __restrict__ out, int ld_out,
                                                   float out_scale) {
    __shared__ float red[33];
    const int o = blockIdx.x, r = rows ? rows[o] : o, center = nrm.kind == SW_NORM_LAYER;
    const float* xr = x + (size_t)r * width;
    float mean = 0.0f;
    if (center) {
        float s = 0.0f;
        for (int c = threadIdx.x; c < width; c += blockDim.x) s += xr[c];
        mean = block_sum(s, red) / (float)width;
    }
    float ss = 0.0f;
    for (int c = threadIdx.x; c < width; c += blockDim.x) { const float d = xr[c] - mean; ss += d * d; }
    const float rstd = 1.0f / sqrtf(block_sum(ss, red) / (float)width + nrm.eps);
    for (int c = threadIdx.x; c < width; c += blockDim.x)
        out[(size_t)o * ld_out + c] = cvt<OT>(((xr[c] - mean) * rstd * nrm.w[c] + (nrm.b ? nrm.b[c] : 0.0f)) * out_scale);
}

// ------------------------------------------------------------------------------------------------ group-limited sigmoid router
// One warp routes one row from its router outputs z [n_exp]: s = logistic(z).  The experts form n_groups equal groups of neighbours; a
// group ranks by the sum of its two largest s (its only s when it has one expert); experts outside the `keep` best groups (ties to the
// lower group) cannot be chosen.  The `top` largest s among the rest are chosen (ties to the lower index) with weight scale * s.  Choices
// top .. top + n_always - 1 are the experts n_exp .. n_exp + n_always - 1 with weight 1 (parts of an expert that every row uses).
// sel_idx / sel_w: the row's top + n_always entries.  s, ch: n_exp floats of shared memory each; gr: n_groups floats.
__device__ __forceinline__ void route_grouped_row(const float* __restrict__ z, int n_exp, int n_groups, int keep, int top, float scale, int n_always,
                                                  int* __restrict__ sel_idx, float* __restrict__ sel_w, float* s, float* ch, float* gr, int lane) {
    for (int i = lane; i < n_exp; i += 32) { const float v = sigmoidf_(z[i]); s[i] = v; ch[i] = v; }
    __syncwarp();
    if (n_groups > 1 && keep < n_groups) {
        const int size = n_exp / n_groups;
        for (int g = lane; g < n_groups; g += 32) {
            float m1 = -INFINITY, m2 = -INFINITY;
            for (int i = 0; i < size; i++) { const float v = s[g * size + i]; if (v > m1) { m2 = m1; m1 = v; } else if (v > m2) m2 = v; }
            gr[g] = size > 1 ? m1 + m2 : m1;
        }
        __syncwarp();
        // `keep` rounds of arg-max over the groups; a kept group's rank becomes +inf, and what is finite afterwards is closed
        for (int k = 0; k < keep; k++) {
            float best = -INFINITY;
            int arg = 0x7fffffff;
            for (int g = lane; g < n_groups; g += 32) { const float v = gr[g]; if (v != INFINITY && v > best) { best = v; arg = g; } }
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) {
                const float ov = __shfl_xor_sync(0xffffffffu, best, o);
                const int oi = __shfl_xor_sync(0xffffffffu, arg, o);
                if (ov > best || (ov == best && oi < arg)) { best = ov; arg = oi; }
            }
            if (arg != 0x7fffffff && lane == 0) gr[arg] = INFINITY;
            __syncwarp();
        }
        for (int i = lane; i < n_exp; i += 32) if (gr[i / size] != INFINITY) ch[i] = -INFINITY;
        __syncwarp();
    }
    for (int k = 0; k < top; k++) {
        float best = -INFINITY;
        int arg = 0x7fffffff;
        for (int i = lane; i < n_exp; i += 32) { const float v = ch[i]; if (v > best) { best = v; arg = i; } }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, best, o);
            const int oi = __shfl_xor_sync(0xffffffffu, arg, o);
            if (ov > best || (ov == best && oi < arg)) { best = ov; arg = oi; }
        }
        if (arg == 0x7fffffff) { arg = 0; best = 0.0f; }
        if (lane == 0) { sel_idx[k] = arg; sel_w[k] = best * scale; ch[arg] = -INFINITY; }
        __syncwarp();
    }
    for (int k = lane; k < n_always; k += 32) { sel_idx[top + k] = n_exp + k; sel_w[top + k] = 1.0f; }
}
// rows of router logits Z -> choices; sel_idx / sel_w [rows][top + n_always].  Shared memory: 2 n_exp + n_groups floats.
__global__ void __launch_bounds__(32) k_moe_route_grouped(const float* __restrict__ Z, int ldz, int n_exp, int n_groups, int keep, int top, float scale,
                                                          int n_always, int* __restrict__ sel_idx, float* __restrict__ sel_w) {
    extern __shared__ float rsm[];
    const int r = blockIdx.x, tt = top + n_always;
    route_grouped_row(Z + (size_t)r * ldz, n_exp, n_groups, keep, top, scale, n_always, sel_idx + (size_t)r * tt, sel_w + (size_t)r * tt, rsm, rsm + n_exp,
                      rsm + 2 * n_exp, threadIdx.x);
}
// One warp routes one row from its router outputs z [n_exp]: the `top` largest are chosen (ties to the lower index), their weights are the softmax
// over the chosen outputs alone.  ch: n_exp floats of shared memory.
__device__ __forceinline__ void route_top_softmax_row(const float* __restrict__ z, int n_exp, int top, int* __restrict__ sel_idx, float* __restrict__ sel_w, float* ch, int lane) {
    for (int i = lane; i < n_exp; i += 32) ch[i] = z[i];
    __syncwarp();
    float first = 0.0f, sum = 0.0f, e0 = 0.0f, e1 = 0.0f;        // lane k % 32 keeps exp(z_k - z_0) of choice k (at most 64 choices)
    for (int k = 0; k < top; k++) {
        float best = -INFINITY;
        int arg = 0x7fffffff;
        for (int i = lane; i < n_exp; i += 32) { const float v = ch[i]; if (v > best) { best = v; arg = i; } }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, best, o);
            const int oi = __shfl_xor_sync(0xffffffffu, arg, o);
            if (ov > best || (ov == best && oi < arg)) { best = ov; arg = oi; }
        }
        if (k == 0) first = best;
        float e = expf(best - first);
        if (arg == 0x7fffffff) { arg = 0; e = 0.0f; }            // every remaining output is -inf or NaN
        sum += e;
        if (lane == (k & 31)) { if (k < 32) e0 = e; else e1 = e; }
        if (lane == 0) { sel_idx[k] = arg; ch[arg] = -INFINITY; }
        __syncwarp();
    }
    const float inv = 1.0f / sum;
    if (lane < top) sel_w[lane] = e0 * inv;
    if (lane + 32 < top) sel_w[lane + 32] = e1 * inv;
}
__global__ void __launch_bounds__(32) k_moe_route_softmax(const float* __restrict__ Z, int ldz, int n_exp, int top, int* __restrict__ sel_idx, float* __restrict__ sel_w) {
    extern __shared__ float rsm[];
    const int r = blockIdx.x;
    route_top_softmax_row(Z + (size_t)r * ldz, n_exp, top, sel_idx + (size_t)r * top, sel_w + (size_t)r * top, rsm, threadIdx.x);
}
// The router of the NEXT sublayer inside the residual update (few rows): what k_sandwich_add appends when it is given a router
struct GroupRouteNext {
    int kind;                  // 0: group-limited logistic; 1: softmax over the chosen outputs (groups, scale and n_always unused)
    const bf16* w;             // [n_exp][ldw] router matrix, or null: no routing here
    int ldw, n_exp, n_groups, keep, top, n_always;
    float scale;
    int* sel_idx;              // [rows][top + n_always]
    float* sel_w;
};
// router logits of row r from the feed-forward's input sx [width] (shared memory; already rounded like the product's operand) -- a warp
// per output -- and the row's choices.  sx is followed by n_exp logits, 2 n_exp work floats and n_groups ranks.
__device__ __forceinline__ void sandwich_route(const GroupRouteNext& rn, float* sx, int width, int r) {
    float* sl = sx + width;
    const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5, nw = blockDim.x >> 5;
    __syncthreads();
    for (int j = wid; j < rn.n_exp; j += nw) {
        const bf16* wr = rn.w + (size_t)j * rn.ldw;
        float a = 0.0f;
        const int w8 = width & ~7;                   // rows of the router matrix start on 16-byte boundaries: eight weights per load
        for (int c = lane * 8; c < w8; c += 256) {
            const uint4 wv = __ldg(reinterpret_cast<const uint4*>(wr + c));
            const uint32_t ww[4] = {wv.x, wv.y, wv.z, wv.w};
#pragma unroll
            for (int i = 0; i < 4; i++) {
                a = fmaf(sx[c + 2 * i], __uint_as_float(ww[i] << 16), a);
                a = fmaf(sx[c + 2 * i + 1], __uint_as_float(ww[i] & 0xffff0000u), a);
            }
        }
        for (int c = w8 + lane; c < width; c += 32) a = fmaf(sx[c], __bfloat162float(wr[c]), a);
        a = warp_sum(a);
        if (lane == 0) sl[j] = a;
    }
    __syncthreads();
    const int tt = rn.top + rn.n_always;
    if (wid == 0 && rn.kind == 1) route_top_softmax_row(sl, rn.n_exp, rn.top, rn.sel_idx + (size_t)r * rn.top, rn.sel_w + (size_t)r * rn.top, sl + rn.n_exp, lane);
    else if (wid == 0)
        route_grouped_row(sl, rn.n_exp, rn.n_groups, rn.keep, rn.top, rn.scale, rn.n_always, rn.sel_idx + (size_t)r * tt, rn.sel_w + (size_t)r * tt, sl + rn.n_exp,
                          sl + 2 * rn.n_exp, sl + 3 * rn.n_exp, lane);
}

// x = scale * embed[tok] and op = norm(x) in one kernel: the first layer's input (models without a bigram table)
template <typename OT>
__global__ void __launch_bounds__(256) k_embed_norm(PassTables t, const bf16* __restrict__ embed, int width, float scale, NormArgs nrm, float* __restrict__ x,
                                                    OT* __restrict__ op, int ld_op) {
    __shared__ float red[33];
    const int r = blockIdx.x, center = nrm.kind == SW_NORM_LAYER;
    const bf16* e = embed + (size_t)t.tok[r] * width;
    float* xr = x + (size_t)r * width;
    float s = 0.0f;
    for (int c = threadIdx.x; c < width; c += blockDim.x) { const float v = __bfloat162float(e[c]) * scale; xr[c] = v; s += v; }
    const float mean = center ? block_sum(s, red) / (float)width : 0.0f;
    float ss = 0.0f;
    for (int c = threadIdx.x; c < width; c += blockDim.x) { const float d = xr[c] - mean; ss += d * d; }      // a thread re-reads what it wrote
    const float rstd = 1.0f / sqrtf(block_sum(ss, red) / (float)width + nrm.eps);
    for (int c = threadIdx.x; c < width; c += blockDim.x) op[(size_t)r * ld_op + c] = cvt<OT>((xr[c] - mean) * rstd * nrm.w[c] + (nrm.b ? nrm.b[c] : 0.0f));
}

// Residual update of the sandwich style: y = Y (+ Y2), or the sum of rows pair_dst[r * top + k] >= 0 of Yg (grouped experts, in order of k);
// x += post(y); when next.w is set, op = next(x) is the operand of the following matrix product.  Rows of up to 4 * SW_KEEP * 256 values
// stay in registers between the passes (16-byte accesses); wider or unaligned rows walk the row again.  With a router (rn.w; few rows) the
// kernel also forms the next sublayer's router logits from the operand row it has just written and picks the experts; dynamic shared
// memory: width + 3 n_exp + n_groups floats.
// JOIN: Y and Y2 are two branches, y = scale (Y / rms(Y) w1 + Y2 / rms(Y2) w2), each norm over the row with its own weight.
// SW_KEEP: float4 groups a thread keeps per array (1, 2 or 4: rows up to 1024, 2048, 4096 wide); fewer kept values, fewer registers, more rows
// in flight per SM -- the kernel is bound by the latency of a row's load / reduce / store chain, not by bandwidth.
struct JoinArgs { const float *w1, *w2; float scale, eps; };
template <typename OT, int SW_KEEP, bool JOIN = false>
__global__ void __launch_bounds__(256, JOIN ? (SW_KEEP == 4 ? 2 : 4) : SW_KEEP == 4 ? 4 : SW_KEEP == 2 ? 6 : 8) k_sandwich_add(const float* __restrict__ Y, const float* __restrict__ Y2, const float* __restrict__ Yg,
                                                      const int* __restrict__ pair_dst, int top, int width, NormArgs post, float* __restrict__ x,
                                                      NormArgs next, OT* __restrict__ op, int ld_op, GroupRouteNext rn, JoinArgs jn) {
    __shared__ float red[JOIN ? 192 : 128];           // four reductions (two more to join branches), each with 32 floats of its own (the walking path uses the first 33)
    __shared__ int sdst[PN_MAX_TOP];
    extern __shared__ float srt[];
    const int r = blockIdx.x;
    const int cp = post.kind == SW_NORM_LAYER, cn = next.kind == SW_NORM_LAYER;
    if (Yg && threadIdx.x < top) sdst[threadIdx.x] = pair_dst[(size_t)r * top + threadIdx.x];
    __syncthreads();
    float* xr = x + (size_t)r * width;
    if (width % 4 == 0 && width <= 4 * SW_KEEP * (int)blockDim.x && ld_op % 4 == 0) {
        float vy[4 * SW_KEEP], vx[4 * SW_KEEP];
#pragma unroll
        for (int i = 0; i < SW_KEEP; i++) {
            const int c = (threadIdx.x + i * blockDim.x) * 4;
            if (c < width) {
                float4 y = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                if (Y) y = *reinterpret_cast<const float4*>(Y + (size_t)r * width + c);
                if (!JOIN && Y2) { const float4 t4 = *reinterpret_cast<const float4*>(Y2 + (size_t)r * width + c); y.x += t4.x; y.y += t4.y; y.z += t4.z; y.w += t4.w; }
                if (!JOIN && Yg)
                    for (int k = 0; k < top; k++)
                        if (sdst[k] >= 0) { const float4 t4 = *reinterpret_cast<const float4*>(Yg + (size_t)sdst[k] * width + c); y.x += t4.x; y.y += t4.y; y.z += t4.z; y.w += t4.w; }
                const float4 xv = *reinterpret_cast<const float4*>(xr + c);
                vy[4 * i] = y.x; vy[4 * i + 1] = y.y; vy[4 * i + 2] = y.z; vy[4 * i + 3] = y.w;
                vx[4 * i] = xv.x; vx[4 * i + 1] = xv.y; vx[4 * i + 2] = xv.z; vx[4 * i + 3] = xv.w;
            }
        }
        float mean, rstd;
        if constexpr (JOIN) {
            float v2[4 * SW_KEEP], r1, r2;
#pragma unroll
            for (int i = 0; i < SW_KEEP; i++) {
                const int c = (threadIdx.x + i * blockDim.x) * 4;
                if (c < width) { const float4 t4 = *reinterpret_cast<const float4*>(Y2 + (size_t)r * width + c); v2[4 * i] = t4.x; v2[4 * i + 1] = t4.y; v2[4 * i + 2] = t4.z; v2[4 * i + 3] = t4.w; }
            }
            sw_stats<SW_KEEP>(vy, width, 0, jn.eps, red + 128 - 32, mean, r1);       // (RMS uses the second 32 floats it is given)
            sw_stats<SW_KEEP>(v2, width, 0, jn.eps, red + 160 - 32, mean, r2);
            r1 *= jn.scale; r2 *= jn.scale;
#pragma unroll
            for (int i = 0; i < SW_KEEP; i++) {
                const int c = (threadIdx.x + i * blockDim.x) * 4;
                if (c < width) {
                    const float4 a4 = *reinterpret_cast<const float4*>(jn.w1 + c), b4 = *reinterpret_cast<const float4*>(jn.w2 + c);
                    vy[4 * i] = vy[4 * i] * r1 * a4.x + v2[4 * i] * r2 * b4.x; vy[4 * i + 1] = vy[4 * i + 1] * r1 * a4.y + v2[4 * i + 1] * r2 * b4.y;
                    vy[4 * i + 2] = vy[4 * i + 2] * r1 * a4.z + v2[4 * i + 2] * r2 * b4.z; vy[4 * i + 3] = vy[4 * i + 3] * r1 * a4.w + v2[4 * i + 3] * r2 * b4.w;
                }
            }
        }
        sw_stats<SW_KEEP>(vy, width, cp, post.eps, red, mean, rstd);
#pragma unroll
        for (int i = 0; i < SW_KEEP; i++) {
            const int c = (threadIdx.x + i * blockDim.x) * 4;
            if (c < width) {
                const float4 w4 = *reinterpret_cast<const float4*>(post.w + c);
                const float4 b4 = post.b ? *reinterpret_cast<const float4*>(post.b + c) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                vx[4 * i] += (vy[4 * i] - mean) * rstd * w4.x + b4.x; vx[4 * i + 1] += (vy[4 * i + 1] - mean) * rstd * w4.y + b4.y;
                vx[4 * i + 2] += (vy[4 * i + 2] - mean) * rstd * w4.z + b4.z; vx[4 * i + 3] += (vy[4 * i + 3] - mean) * rstd * w4.w + b4.w;
                *reinterpret_cast<float4*>(xr + c) = make_float4(vx[4 * i], vx[4 * i + 1], vx[4 * i + 2], vx[4 * i + 3]);
            }
        }
        if (!next.w) return;
        sw_stats<SW_KEEP>(vx, width, cn, next.eps, red + 64, mean, rstd);
#pragma unroll
        for (int i = 0; i < SW_KEEP; i++) {
            const int c = (threadIdx.x + i * blockDim.x) * 4;
            if (c < width) {
                const float4 w4 = *reinterpret_cast<const float4*>(next.w + c);
                const float4 b4 = next.b ? *reinterpret_cast<const float4*>(next.b + c) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                const float h0 = (vx[4 * i] - mean) * rstd * w4.x + b4.x, h1 = (vx[4 * i + 1] - mean) * rstd * w4.y + b4.y;
                const float h2 = (vx[4 * i + 2] - mean) * rstd * w4.z + b4.z, h3 = (vx[4 * i + 3] - mean) * rstd * w4.w + b4.w;
                store4(op + (size_t)r * ld_op + c, h0, h1, h2, h3);
                if (rn.w) { srt[c] = ldf<OT>(op + (size_t)r * ld_op + c); srt[c + 1] = ldf<OT>(op + (size_t)r * ld_op + c + 1);      // as the product would read them
                            srt[c + 2] = ldf<OT>(op + (size_t)r * ld_op + c + 2); srt[c + 3] = ldf<OT>(op + (size_t)r * ld_op + c + 3); }
            }
        }
        if (rn.w) sandwich_route(rn, srt, width, r);
        return;
    }
    float j1 = 0.0f, j2 = 0.0f;
    if (JOIN) {
        for (int c = threadIdx.x; c < width; c += blockDim.x) { const float a = Y[(size_t)r * width + c], q = Y2[(size_t)r * width + c]; j1 += a * a; j2 += q * q; }
        j1 = jn.scale / sqrtf(block_sum(j1, red) / (float)width + jn.eps);
        j2 = jn.scale / sqrtf(block_sum(j2, red) / (float)width + jn.eps);
    }
    auto sub = [&](int c) {
        if (JOIN) return Y[(size_t)r * width + c] * j1 * jn.w1[c] + Y2[(size_t)r * width + c] * j2 * jn.w2[c];
        float a = Y ? Y[(size_t)r * width + c] : 0.0f;
        if (Y2) a += Y2[(size_t)r * width + c];
        if (Yg)
            for (int k = 0; k < top; k++)
                if (sdst[k] >= 0) a += Yg[(size_t)sdst[k] * width + c];
        return a;
    };
    float mean = 0.0f, s = 0.0f;
    if (cp) {
        for (int c = threadIdx.x; c < width; c += blockDim.x) s += sub(c);
        mean = block_sum(s, red) / (float)width;
    }
    s = 0.0f;
    for (int c = threadIdx.x; c < width; c += blockDim.x) { const float d = sub(c) - mean; s += d * d; }
    float rstd = 1.0f / sqrtf(block_sum(s, red) / (float)width + post.eps);
    for (int c = threadIdx.x; c < width; c += blockDim.x) xr[c] += (sub(c) - mean) * rstd * post.w[c] + (post.b ? post.b[c] : 0.0f);     // a thread re-reads only what it wrote
    if (!next.w) return;
    mean = 0.0f; s = 0.0f;
    if (cn) {
        for (int c = threadIdx.x; c < width; c += blockDim.x) s += xr[c];
        mean = block_sum(s, red) / (float)width;
    }
    s = 0.0f;
    for (int c = threadIdx.x; c < width; c += blockDim.x) { const float d = xr[c] - mean; s += d * d; }
    rstd = 1.0f / sqrtf(block_sum(s, red) / (float)width + next.eps);
    for (int c = threadIdx.x; c < width; c += blockDim.x) {
        const OT h = cvt<OT>((xr[c] - mean) * rstd * next.w[c] + (next.b ? next.b[c] : 0.0f));
        op[(size_t)r * ld_op + c] = h;
        if (rn.w) srt[c] = ldf<OT>(&h);
    }
    if (rn.w) sandwich_route(rn, srt, width, r);
}

// sc[r][0] = 1 / sqrt(mean(q_r^2) + eps) over the nq entries of row r's query projection, sc[r][1] the same for its nk key entries (nk may be 0)
__global__ void __launch_bounds__(256) k_proj_rms(const float* __restrict__ P, int ldp, int q_off, int nq, int k_off, int nk, float eps, float* __restrict__ sc) {
    __shared__ float red[33];
    const int r = blockIdx.x;
    const float* p = P + (size_t)r * ldp;
    float a = 0.0f, b = 0.0f;
    for (int i = threadIdx.x; i < nq; i += blockDim.x) { const float v = p[q_off + i]; a += v * v; }
    for (int i = threadIdx.x; i < nk; i += blockDim.x) { const float v = p[k_off + i]; b += v * v; }
    a = block_sum(a, red);
    b = block_sum(b, red);
    if (threadIdx.x == 0) {
        sc[(size_t)r * 2] = 1.0f / sqrtf(a / (float)nq + eps);
        sc[(size_t)r * 2 + 1] = nk > 0 ? 1.0f / sqrtf(b / (float)nk + eps) : 0.0f;
    }
}

// ------------------------------------------------------------------------------------------------ differential attention
struct DiffArgs {
    int heads, dim, vdim;
    float diff, eps, out_scale;
    const float *lq1, *lk1, *lq2, *lk2;     // [dim]
    int gate, g_off, a_off;                  // gate 0: none; 3: logistic of column g_off + head of P
};
// A [R][heads * 2 * vdim]: the two maps' outputs per head.  o = a1 - lambda a2, lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff;
// o / sqrt(mean(o^2) + eps) * (1 - diff), gate, weight -> operand.  A warp per (row, head).
template <typename OT>
__global__ void __launch_bounds__(128) k_diff_combine(DiffArgs b, const float* __restrict__ A, const float* __restrict__ P, int ldp, OT* __restrict__ out, int ld_out) {
    const int r = blockIdx.x, lane = threadIdx.x & 31, wid = threadIdx.x >> 5, nw = blockDim.x >> 5;
    float d1 = 0.0f, d2 = 0.0f;
    for (int i = lane; i < b.dim; i += 32) { d1 = fmaf(b.lq1[i], b.lk1[i], d1); d2 = fmaf(b.lq2[i], b.lk2[i], d2); }
    const float lambda = expf(warp_sum(d1)) - expf(warp_sum(d2)) + b.diff;
    for (int h = blockIdx.y * nw + wid; h < b.heads; h += gridDim.y * nw) {
        const float* a1 = A + ((size_t)r * b.heads + h) * 2 * b.vdim;
        const float* a2 = a1 + b.vdim;
        float ss = 0.0f;
        for (int i = lane; i < b.vdim; i += 32) { const float o = a1[i] - lambda * a2[i]; ss += o * o; }
        ss = warp_sum(ss);
        float sc = (1.0f - b.diff) * b.out_scale / sqrtf(ss / (float)b.vdim + b.eps);
        if (b.gate) sc *= sigmoidf_(P[(size_t)r * ldp + b.g_off + h]);
        for (int i = lane; i < b.vdim; i += 32) out[(size_t)r * ld_out + b.a_off + h * b.vdim + i] = cvt<OT>((a1[i] - lambda * a2[i]) * sc);
    }
}

// ------------------------------------------------------------------------------------------------ retention: activation, joint norm
// q, k, v <- silu(.) in place: columns [c0, c0 + n) of the projection buffer (q | k | v are neighbours)
__global__ void k_silu_cols(float* __restrict__ P, int ldp, int c0, int n, int R) {
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (size_t)R * n) return;
    float* p = P + (i / n) * ldp + c0 + (i % n);
    const float z = *p;
    *p = z * sigmoidf_(z);
}
// per row: o (all heads together) / sqrt(mean(o^2) + eps) * w, times the gate (1: silu, 2: logistic of P's column g_off + c), times out_scale
template <typename OT>
__global__ void __launch_bounds__(256) k_ret_post_all(RetBranch b, const float* __restrict__ w, const float* __restrict__ O, const float* __restrict__ P, int ldp,
                                                      OT* __restrict__ out, int ld_out) {
    __shared__ float red[33];
    const int r = blockIdx.x, n = b.heads * b.vdim;
    const float* o = O + (size_t)r * n;
    float ss = 0.0f;
    for (int c = threadIdx.x; c < n; c += blockDim.x) ss += o[c] * o[c];
    const float sc = b.out_scale / sqrtf(block_sum(ss, red) / (float)n + b.eps);
    for (int c = threadIdx.x; c < n; c += blockDim.x) {
        float v = o[c] * sc * w[c];
        if (b.gated) { const float g = P[(size_t)r * ldp + b.g_off + c]; v *= b.gated == 2 ? sigmoidf_(g) : g * sigmoidf_(g); }
        out[(size_t)r * ld_out + b.a_off + c] = cvt<OT>(v);
    }
}

// ------------------------------------------------------------------------------------------------ convolution behind the projections
struct ConvArgs {
    int nq, nk, nv;              // channels: queries, keys (both convolved), values (appended as they are; 0: the values are the keys)
    int off;                     // column of the first query channel in P; keys and values follow
    int taps;
    const float* w;              // [nq + nk][taps]
    int max_ctx, k_ld, v_ld;     // cache rows
    const float* bias;           // [nq + nk] added behind the convolution, or null
    int silu;                    // 1: silu on the result
    void* op;                    // the convolved "queries" once more as a product operand [R][ld_op], or null
    int ld_op;
};
// y_t = sum_j w[c][j] u_(t - taps + 1 + j) of every query and key channel of P; queries -> Q [R][nq] (fp32), keys -> the slot's key cache.
// Rows before the segment come from the slot's history `tail` [n_slots][taps - 1][nq + nk] (zeros after a reset = zeros before the
// sequence).  A thread owns V neighbouring channels of `rows_per` consecutive rows and slides its window of `taps` values along them (TAPS 0:
// any number of taps, read back from memory instead).  P keeps the projected values: other rows' windows and the history update read them.
// every_one: each segment is one row, so the thread that has read a channel's history also writes its update.
template <int V> __device__ __forceinline__ void cv_load(const float* __restrict__ p, float (&v)[V]) {
    if (V == 4) { const float4 t = *reinterpret_cast<const float4*>(p); v[0] = t.x; v[V > 1 ? 1 : 0] = t.y; v[V > 2 ? 2 : 0] = t.z; v[V > 3 ? 3 : 0] = t.w; }
    else v[0] = *p;
}
template <typename T> __device__ __forceinline__ void cv_store(T* p, const float (&v)[4]) { store4(p, v[0], v[1], v[2], v[3]); }
template <typename T> __device__ __forceinline__ void cv_store(T* p, const float (&v)[1]) { *p = cvt<T>(v[0]); }
template <typename OT, int V, int TAPS>
__global__ void __launch_bounds__(128) k_qk_conv(PassTables t, ConvArgs b, const float* __restrict__ P, int ldp, int R, int rows_per, float* __restrict__ tail,
                                                 float* __restrict__ Q, OT* __restrict__ kc, OT* __restrict__ vc, int every_one) {
    const int nc = b.nq + b.nk, c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
    if (c >= nc + b.nv) return;
    const int r0 = blockIdx.x * rows_per, r1 = min(R, r0 + rows_per);
    const float* p = P + b.off + c;
    if (c >= nc) {
        for (int r = r0; r < r1; r++) {
            float u[V];
            cv_load<V>(p + (size_t)r * ldp, u);
            cv_store(vc + ((size_t)t.seg_slot[t.row_seg[r]] * b.max_ctx + t.row_pos[r]) * b.v_ld + (c - nc), u);
        }
        return;
    }
    constexpr int NT = TAPS > 0 ? TAPS : 1;
    float w[NT][V], u[NT][V];
    if (TAPS > 0) {
#pragma unroll
        for (int j = 0; j < NT; j++)
#pragma unroll
            for (int i = 0; i < V; i++) w[j][i] = b.w[(size_t)(c + i) * NT + j];
    }
    int seg = -1, row0 = 0, slot = 0;
    for (int r = r0; r < r1; r++) {
        float y[V];
        const bool fresh = t.row_seg[r] != seg;
        if (fresh) { seg = t.row_seg[r]; row0 = t.seg_row0[seg]; slot = t.seg_slot[seg]; }
        float* tl = tail + (size_t)slot * (b.taps - 1) * nc + c;
        if (TAPS > 0) {
            if (fresh) {
#pragma unroll
                for (int j = 0; j < NT - 1; j++) {
                    const int src = r - (NT - 1) + j;
                    if (src >= row0) cv_load<V>(p + (size_t)src * ldp, u[j]);
                    else {
#pragma unroll
                        for (int i = 0; i < V; i++) u[j][i] = tl[(size_t)(src - row0 + NT - 1) * nc + i];
                    }
                }
            }
            cv_load<V>(p + (size_t)r * ldp, u[NT - 1]);
#pragma unroll
            for (int i = 0; i < V; i++) y[i] = 0.0f;
#pragma unroll
            for (int j = 0; j < NT; j++)
#pragma unroll
                for (int i = 0; i < V; i++) y[i] = fmaf(w[j][i], u[j][i], y[i]);
#pragma unroll
            for (int j = 0; j < NT - 1; j++)
#pragma unroll
                for (int i = 0; i < V; i++) u[j][i] = u[j + 1][i];
            if (every_one && !t.slots[slot].stopped) {
#pragma unroll
                for (int j = 0; j < NT - 1; j++)
#pragma unroll
                    for (int i = 0; i < V; i++) tl[(size_t)j * nc + i] = u[j][i];
            }
        } else {
#pragma unroll
            for (int i = 0; i < V; i++) y[i] = 0.0f;
            for (int j = 0; j < b.taps; j++) {
                const int src = r - (b.taps - 1) + j;
#pragma unroll
                for (int i = 0; i < V; i++)
                    y[i] = fmaf(b.w[(size_t)(c + i) * b.taps + j], src >= row0 ? p[(size_t)src * ldp + i] : tl[(size_t)(src - row0 + b.taps - 1) * nc + i], y[i]);
            }
        }
        if (b.bias) {
#pragma unroll
            for (int i = 0; i < V; i++) y[i] += b.bias[c + i];
        }
        if (b.silu) {
#pragma unroll
            for (int i = 0; i < V; i++) y[i] = silu_(y[i]);
        }
        if (b.op && c < b.nq) cv_store(reinterpret_cast<OT*>(b.op) + (size_t)r * b.ld_op + c, y);
        if (c < b.nq) cv_store(Q + (size_t)r * b.nq + c, y);
        else cv_store(kc + ((size_t)slot * b.max_ctx + t.row_pos[r]) * b.k_ld + (c - b.nq), y);
    }
}

// ------------------------------------------------------------------------------------------------ ungated feed-forward
// act = gelu(G) -> operand [R][ld_out], zero-padded (grid: rows x column groups; few rows spread their columns over many CTAs)
template <typename OT>
__global__ void k_gelu_rows(const float* __restrict__ G, int ff, OT* __restrict__ out, int ld_out) {
    const int r = blockIdx.x;
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < ld_out; c += gridDim.y * blockDim.x)
        out[(size_t)r * ld_out + c] = cvt<OT>(c < ff ? gelu_erf(G[(size_t)r * ff + c]) : 0.0f);
}

}  // namespace seq
}  // namespace gtb
