// Mixture of experts: the router's choice and the experts' activation.
//
// moe_route: per row, scores s = softmax(z) over all experts in fp32, the `top` largest chosen (of equal
// scores the lower index first), weights s / (sum of the chosen s + renorm_eps).  The weights are left
// twice: as a dense row [experts] with zeros for the experts not chosen, which is what the stacked
// products of a step of many rows multiply by, and as `top` (index, weight) pairs for a step of few rows
// that reads only the chosen experts' matrices.
//
// With a correction an expert is chosen by its score plus a learned number and weighed by the score; with groups only
// experts of the best groups of neighbours (by the sum of a group's two largest choice scores, or by its largest) can be chosen.
//
// moe_act: act[r, e * ff + i] = weight[r, e] * relu(up[r, e * ff + i])^2: the activation of every expert's
// hidden layer with the row's weight for that expert folded in, so that one product with the experts' down
// matrices side by side gives the weighted sum of the chosen experts' outputs (an expert that was not
// chosen contributes exact zeros).
//
// moe_up_rows / moe_down_rows: the same feed-forward for a step of few rows, reading only the chosen
// experts' matrices (a warp a hidden unit, or an output column, of one (row, choice) pair).
//
// moe_up_grouped / moe_down_grouped: the same with the pairs sorted by expert, so an expert's matrices are read once; on the
// tensor cores where rows are aligned.
//
// moe_group / moe_gather / relu2 / moe_combine: a step of many rows sorts its (row, choice) pairs by expert
// (counts, offsets, and each pair's place in the sorted order), gathers the rows in that order so that every
// expert's rows lie together for one product an expert, squares the positive part between the two products, and
// adds each row's `top` results up with their weights in the order of the choices.  Where a pair lands inside its
// expert's group may differ from run to run; a row's result does not depend on it.
#include "api.h"
#include "common.cuh"
#include "mma.cuh"

#include <math.h>

namespace {

constexpr int MAX_EXPERTS_PER_LANE = 16;   // experts up to 512

// Which experts may be chosen: with groups, `key` (the warp's choice scores in shared memory) is scanned by a lane a group
// for the group's two largest (which count together, or with `largest` the first alone), and a group is kept if fewer than keep_groups groups come before it (a larger sum, or an
// equal one and a lower number).  Scores of the other groups become -inf.
__device__ __forceinline__ void drop_groups(float* key, float* strength, int E, int groups, int keep, int largest, int lane) {
    const int per = E / groups;
    for (int g = lane; g < groups; g += 32) {
        float a = -INFINITY, b = -INFINITY;
        for (int i = 0; i < per; i++) {
            const float v = key[g * per + i];
            if (v > a) {
                b = a;
                a = v;
            } else if (v > b) {
                b = v;
            }
        }
        strength[g] = per > 1 && !largest ? a + b : a;
    }
    __syncwarp();
    for (int g = lane; g < groups; g += 32) {
        const float mine = strength[g];
        int before = 0;
        for (int o = 0; o < groups; o++) before += strength[o] > mine || (strength[o] == mine && o < g);
        if (before >= keep)
            for (int i = 0; i < per; i++) key[g * per + i] = -INFINITY;
    }
    __syncwarp();
}

// CORRECTED: the choice goes by score + correction and, with groups, inside the best of them
template <bool CORRECTED>
__global__ void __launch_bounds__(128) moe_route_kernel(MoeRouteParams p) {
    __shared__ float key_s[CORRECTED ? 4 : 1][CORRECTED ? 32 * MAX_EXPERTS_PER_LANE : 1];
    __shared__ float group_s[CORRECTED ? 4 : 1][CORRECTED ? 32 * MAX_EXPERTS_PER_LANE : 1];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int64_t row = (int64_t)blockIdx.x * 4 + warp;
    if (row >= p.rows) return;
    const int E = p.experts;
    const float* z = p.logits + row * p.logits_stride;
    float s[MAX_EXPERTS_PER_LANE];
    float mx = -INFINITY;
#pragma unroll
    for (int e = 0; e < MAX_EXPERTS_PER_LANE; e++) {
        const int i = lane + 32 * e;
        s[e] = i < E ? z[i] : -INFINITY;
        mx = fmaxf(mx, s[e]);
    }
    mx = warp_max(mx);
    float sum = 0.f;
#pragma unroll
    for (int e = 0; e < MAX_EXPERTS_PER_LANE; e++) {
        const int i = lane + 32 * e;
        // the key an expert is chosen by: its softmax numerator, or, for sigmoid scores, the logit itself (the
        // sigmoid grows with it, and two large logits stay apart where their sigmoids both round to 1);
        // -inf marks what is absent or taken
        s[e] = i < E ? (p.score_kind == 1 ? s[e] : expf(s[e] - mx)) : -INFINITY;
        if (i < E && p.score_kind != 1) sum += s[e];
    }
    sum = warp_sum(sum);
    const float inv = p.score_kind == 1 ? 1.f : 1.f / sum;     // a sigmoid score stands by itself
    if (CORRECTED) {
#pragma unroll
        for (int e = 0; e < MAX_EXPERTS_PER_LANE; e++) {
            const int i = lane + 32 * e;
            if (i >= E) continue;
            s[e] = (p.score_kind == 1 ? 1.f / (1.f + expf(-s[e])) : s[e] * inv) + (p.correction ? p.correction[i] : 0.f);
            if (p.groups > 1) key_s[warp][i] = s[e];
        }
        if (p.groups > 1) {
            __syncwarp();
            drop_groups(key_s[warp], group_s[warp], E, p.groups, p.keep_groups, p.group_largest, lane);
#pragma unroll
            for (int e = 0; e < MAX_EXPERTS_PER_LANE; e++)
                if (lane + 32 * e < E) s[e] = key_s[warp][lane + 32 * e];
        }
    }
    float* dense = p.dense + row * E;
    for (int i = lane; i < E; i += 32) dense[i] = 0.f;
    float chosen_sum = 0.f;
    float my_w = 0.f;      // lane k keeps the k-th choice
    int my_i = 0;
    for (int k = 0; k < p.top; k++) {
        float best = -INFINITY;
        int best_i = 0x7fffffff;
#pragma unroll
        for (int e = 0; e < MAX_EXPERTS_PER_LANE; e++) {
            const int i = lane + 32 * e;
            if (s[e] > best) best = s[e], best_i = i;     // within a lane indices grow with e: the first of equals stays
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ob = __shfl_xor_sync(0xffffffffu, best, o);
            const int oi = __shfl_xor_sync(0xffffffffu, best_i, o);
            if (ob > best || (ob == best && oi < best_i)) best = ob, best_i = oi;
        }
#pragma unroll
        for (int e = 0; e < MAX_EXPERTS_PER_LANE; e++)
            if (lane + 32 * e == best_i) s[e] = -INFINITY;
        if (best_i >= E) best_i = k;       // no number compares (NaN logits): any expert, but one that exists
        float sc;
        if (CORRECTED) {       // the score again, without its correction
            const float zc = z[best_i];
            sc = p.score_kind == 1 ? 1.f / (1.f + expf(-zc)) : expf(zc - mx) * inv;
        } else {
            sc = p.score_kind == 1 ? 1.f / (1.f + expf(-best)) : best * inv;
        }
        chosen_sum += sc;
        if (lane == (k & 31)) my_w = sc, my_i = best_i;
        if (k >= 32 && lane == 0) {}   // more than 32 choices are refused on the host
    }
    const float norm = p.renorm ? 1.f / (chosen_sum + p.renorm_eps) : 1.f;
    __syncwarp();
    if (lane < p.top) {
        const float w = my_w * norm;
        dense[my_i] = w;
        p.index[row * p.top + lane] = my_i;
        p.weight[row * p.top + lane] = w;
    }
}

// What an expert's hidden unit makes of its product(s) z (and, for a gated expert, u) and the pair's weight w:
// kind 0: relu(z)^2; kind 1: silu(z) * u; kind 2: g sigmoid(slope g) (v + 1) with g = min(z, limit) and
// v = clamp(u, -limit, limit).  The weight multiplies the result, or (weight_input) the expert's
// input, which for products without biases is the same as multiplying z and u.
__device__ __forceinline__ float expert_act(float z, float u, float w, int kind, int weight_input, float limit = 0.f, float slope = 1.f) {
    if (weight_input) z *= w, u *= w;
    float a;
    if (kind == 1) {
        a = z / (1.f + expf(-z)) * u;
    } else if (kind == 2) {
        const float g = fminf(z, limit), v = fminf(fmaxf(u, -limit), limit);
        a = g / (1.f + expf(-slope * g)) * (v + 1.f);
    } else {
        const float r = fmaxf(z, 0.f);
        a = r * r;
    }
    return weight_input ? a : w * a;
}

// up: [rows, experts * (kind 1: 2 ff, gate rows then up rows of each expert; else ff)]; dense null: every weight is 1
template <typename T>
__global__ void moe_act_kernel(const T* __restrict__ up, int64_t up_stride, const float* __restrict__ dense, T* __restrict__ act,
                               int64_t act_stride, int rows, int experts, int ff, int kind, int weight_input, float limit, float slope) {
    const int64_t n = (int64_t)experts * ff;
    const int64_t idx = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= rows * n) return;
    const int64_t r = idx / n, c = idx % n;
    const int64_t e = c / ff, i = c - e * ff;
    const float w = dense ? dense[r * experts + e] : 1.f;
    float z, u = 0.f;
    if (kind != 0) {
        z = to_f32<T>(up[r * up_stride + e * 2 * ff + i]);
        u = to_f32<T>(up[r * up_stride + e * 2 * ff + ff + i]);
    } else {
        z = to_f32<T>(up[r * up_stride + c]);
    }
    act[r * act_stride + c] = from_f32<T>(expert_act(z, u, w, kind, weight_input, limit, slope));
}

// a warp's share of the dot product of a weight row and a row of activations, 16 bytes a lane where both allow it
template <typename T, typename TW>
__device__ __forceinline__ float warp_dot(const TW* __restrict__ w, const T* __restrict__ x, int n, int lane) {
    float a = 0.f;
    for (int c = lane; c < n; c += 32) a = fmaf(to_f32<TW>(w[c]), to_f32<T>(x[c]), a);
    return a;
}
template <>
__device__ __forceinline__ float warp_dot<__nv_bfloat16, __nv_bfloat16>(const __nv_bfloat16* __restrict__ w, const __nv_bfloat16* __restrict__ x,
                                                                        int n, int lane) {
    float a = 0.f;
    if (!(n & 7) && !((uintptr_t)w & 15) && !((uintptr_t)x & 15)) {
        for (int c = lane * 8; c < n; c += 256) {
            const uint4 wv = *reinterpret_cast<const uint4*>(w + c), xv = *reinterpret_cast<const uint4*>(x + c);
            const __nv_bfloat162* wh = reinterpret_cast<const __nv_bfloat162*>(&wv);
            const __nv_bfloat162* xh = reinterpret_cast<const __nv_bfloat162*>(&xv);
#pragma unroll
            for (int e = 0; e < 4; e++) {
                a = fmaf(__low2float(wh[e]), __low2float(xh[e]), a);
                a = fmaf(__high2float(wh[e]), __high2float(xh[e]), a);
            }
        }
        return a;
    }
    for (int c = lane; c < n; c += 32) a = fmaf(__bfloat162float(w[c]), __bfloat162float(x[c]), a);
    return a;
}

// few rows: act[r, k, i] = weight[r, k] * relu(W_up[index[r, k]][i, :] . x[r])^2, a warp a hidden unit
template <typename T, typename TW>
__global__ void __launch_bounds__(128) moe_up_rows_kernel(MoeRowsParams p) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int i = blockIdx.x * 4 + warp;
    const int pair = blockIdx.y;            // row * top + k
    if (i >= p.ff) return;
    const int r = pair / p.top;
    const int e = p.index[pair];
    const int per = p.act_kind != 0 ? 2 : 1;      // a gated expert holds its gate rows, then its up rows
    const TW* w = (const TW*)p.up + ((int64_t)e * per * p.ff + i) * p.hidden;
    const T* x = (const T*)p.x + (int64_t)r * p.x_stride;
    const float a = warp_sum(warp_dot<T, TW>(w, x, p.hidden, lane));
    const float b = p.act_kind != 0 ? warp_sum(warp_dot<T, TW>(w + (int64_t)p.ff * p.hidden, x, p.hidden, lane)) : 0.f;
    if (lane == 0) {
        // the same roundings as the stacked path: the product in the activation dtype, then the activation
        ((T*)p.act)[(int64_t)pair * p.ff + i] =
            from_f32<T>(expert_act(to_f32<T>(from_f32<T>(a)), to_f32<T>(from_f32<T>(b)), p.weight[pair], p.act_kind, p.weight_input, p.limit, p.slope));
    }
}

// out[r, c] = sum_k W_down[index[r, k]][c, :] . act[r, k, :], a warp an output column of a row
template <typename T, typename TW>
__global__ void __launch_bounds__(128) moe_down_rows_kernel(MoeRowsParams p) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int c = blockIdx.x * 4 + warp;
    const int r = blockIdx.y;
    if (c >= p.hidden) return;
    float a = 0.f;
    for (int k = 0; k < p.top; k++) {
        const int pair = r * p.top + k;
        const int e = p.index[pair];
        const TW* w = (const TW*)p.down + ((int64_t)c * p.experts + e) * p.ff;      // the down matrices side by side: [hidden, experts * ff]
        a += warp_dot<T, TW>(w, (const T*)p.act + (int64_t)pair * p.ff, p.ff, lane);
    }
    a = warp_sum(a);
    if (lane == 0) p.out[(int64_t)r * p.out_stride + c] = a;
}

// The same two products with the pairs sorted by expert (moe_group): a warp takes a hidden unit (an output column) of
// ONE expert and walks that expert's pairs, so an expert's matrices are read from memory once however many rows chose
// it (the row of the matrix stays in the first-level cache from pair to pair).  act[p, i] = relu(up_e[i] . x[src_row[p]])^2
// at the pair's sorted place p, ys[p, c] = down_e[c] . act[p]; the weights are applied when the rows are added up.
template <typename T, typename TW>
__global__ void __launch_bounds__(128) moe_up_grouped_kernel(MoeRowsParams p, const int* __restrict__ offsets, const int* __restrict__ src_row) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int i = blockIdx.x * 4 + warp, e = blockIdx.y;
    const int lo = offsets[e], hi = offsets[e + 1];
    if (i >= p.ff || lo == hi) return;
    const int per = p.act_kind != 0 ? 2 : 1;
    const TW* w = (const TW*)p.up + ((int64_t)e * per * p.ff + i) * p.hidden;
    for (int at = lo; at < hi; at++) {
        const T* x = (const T*)p.x + (int64_t)src_row[at] * p.x_stride;
        const float a = warp_sum(warp_dot<T, TW>(w, x, p.hidden, lane));
        const float b = p.act_kind != 0 ? warp_sum(warp_dot<T, TW>(w + (int64_t)p.ff * p.hidden, x, p.hidden, lane)) : 0.f;
        if (lane == 0) {
            // a weight on the expert's input is applied here (p.weight: the pairs' weights in sorted order), one on its
            // output when the rows are added up
            const float pw = p.weight_input ? p.weight[at] : 1.f;
            ((T*)p.act)[(int64_t)at * p.ff + i] =
                from_f32<T>(expert_act(to_f32<T>(from_f32<T>(a)), to_f32<T>(from_f32<T>(b)), pw, p.act_kind, p.weight_input, p.limit, p.slope));
        }
    }
}

template <typename T, typename TW>
__global__ void __launch_bounds__(128) moe_down_grouped_kernel(MoeRowsParams p, const int* __restrict__ offsets, float* __restrict__ ys) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int c = blockIdx.x * 4 + warp, e = blockIdx.y;
    const int lo = offsets[e], hi = offsets[e + 1];
    if (c >= p.hidden || lo == hi) return;
    const TW* w = (const TW*)p.down + ((int64_t)c * p.experts + e) * p.ff;
    for (int at = lo; at < hi; at++) {
        const float a = warp_sum(warp_dot<T, TW>(w, (const T*)p.act + (int64_t)at * p.ff, p.ff, lane));
        if (lane == 0) ys[(int64_t)at * p.hidden + c] = a;
    }
}

// The same two products in bfloat16 on the tensor cores: a CTA takes 16 rows of ONE expert's matrix (16 hidden units, or 16
// output columns), streams them once from global memory straight into mma.sync fragments (the fragment's k order is the
// memory's: see gemm_skinny.cu) and multiplies them with eight of the expert's pairs at a time; its warps split K and
// meet in shared memory, added in warp order, so a pair's sums do not depend on what else the step holds.
constexpr int MG_WARPS = 8;

// W: this lane's two rows (g and g + 8 of the tile) at its place in a 32-wide step, X: its pair's row at the same place
__device__ __forceinline__ void stream_product(float (&acc)[4], const __nv_bfloat16* __restrict__ w_lo, const __nv_bfloat16* __restrict__ w_hi,
                                               const __nv_bfloat16* __restrict__ x, int k, int k_end, int t) {
    const int k_full = k + (k_end - k) / 32 * 32;
    constexpr int U = 4;
    for (; k + U * 32 <= k_full; k += U * 32) {      // the loads of four steps are in flight before the first product needs one
        uint4 a_lo[U], a_hi[U], b[U];
#pragma unroll
        for (int u = 0; u < U; u++) {
            a_lo[u] = ld_stream16(w_lo + k + u * 32);
            a_hi[u] = ld_stream16(w_hi + k + u * 32);
        }
#pragma unroll
        for (int u = 0; u < U; u++) b[u] = *reinterpret_cast<const uint4*>(x + k + u * 32);
#pragma unroll
        for (int u = 0; u < U; u++) {
            mma_bf16_16816(acc, a_lo[u].x, a_hi[u].x, a_lo[u].y, a_hi[u].y, b[u].x, b[u].y);
            mma_bf16_16816(acc, a_lo[u].z, a_hi[u].z, a_lo[u].w, a_hi[u].w, b[u].z, b[u].w);
        }
    }
    for (; k < k_full; k += 32) {
        const uint4 a_lo = ld_stream16(w_lo + k), a_hi = ld_stream16(w_hi + k), b = *reinterpret_cast<const uint4*>(x + k);
        mma_bf16_16816(acc, a_lo.x, a_hi.x, a_lo.y, a_hi.y, b.x, b.y);
        mma_bf16_16816(acc, a_lo.z, a_hi.z, a_lo.w, a_hi.w, b.z, b.w);
    }
    if (k < k_end) {      // K is a multiple of 8: a lane's piece is wholly inside or wholly outside
        const bool in = k + t * 8 < k_end;
        const uint4 z = make_uint4(0, 0, 0, 0);
        const uint4 a_lo = in ? ld_stream16(w_lo + k) : z, a_hi = in ? ld_stream16(w_hi + k) : z, b = in ? *reinterpret_cast<const uint4*>(x + k) : z;
        mma_bf16_16816(acc, a_lo.x, a_hi.x, a_lo.y, a_hi.y, b.x, b.y);
        mma_bf16_16816(acc, a_lo.z, a_hi.z, a_lo.w, a_hi.w, b.z, b.w);
    }
}

__device__ __forceinline__ void leave_fragment(float* __restrict__ mine, const float (&acc)[4], int g, int t) {
    mine[g * 8 + 2 * t] = acc[0];
    mine[g * 8 + 2 * t + 1] = acc[1];
    mine[(g + 8) * 8 + 2 * t] = acc[2];
    mine[(g + 8) * 8 + 2 * t + 1] = acc[3];
}

template <bool GATED>
__global__ void __launch_bounds__(32 * MG_WARPS) moe_up_grouped_mma_kernel(MoeRowsParams p, const int* __restrict__ offsets,
                                                                           const int* __restrict__ src_row) {
    __shared__ float red[GATED ? 2 : 1][MG_WARPS][16 * 8];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const int n0 = blockIdx.x * 16, e = blockIdx.y, K = p.hidden;
    const int lo = offsets[e], hi = offsets[e + 1];
    if (lo == hi) return;
    const int i_lo = min(n0 + g, p.ff - 1), i_hi = min(n0 + g + 8, p.ff - 1);      // rows past the end repeat the last one and are dropped
    const __nv_bfloat16* w = (const __nv_bfloat16*)p.up + (int64_t)e * (GATED ? 2 : 1) * p.ff * K + t * 8;
    const __nv_bfloat16 *w_lo = w + (int64_t)i_lo * K, *w_hi = w + (int64_t)i_hi * K;
    const int per = ((K + 31) / 32 + MG_WARPS - 1) / MG_WARPS * 32;
    const int k0 = warp * per, k1 = min(k0 + per, K);
    for (int p0 = lo; p0 < hi; p0 += 8) {
        const __nv_bfloat16* x = (const __nv_bfloat16*)p.x + (int64_t)src_row[min(p0 + g, hi - 1)] * p.x_stride + t * 8;
        float acc[4] = {0.f, 0.f, 0.f, 0.f}, acc2[4] = {0.f, 0.f, 0.f, 0.f};
        if (k0 < k1) stream_product(acc, w_lo, w_hi, x, k0, k1, t);
        if (GATED && k0 < k1) stream_product(acc2, w_lo + (int64_t)p.ff * K, w_hi + (int64_t)p.ff * K, x, k0, k1, t);
        leave_fragment(red[0][warp], acc, g, t);
        if (GATED) leave_fragment(red[GATED ? 1 : 0][warp], acc2, g, t);
        __syncthreads();
        if (threadIdx.x < 128) {
            const int b = threadIdx.x >> 4, i = threadIdx.x & 15, at = p0 + b;
            if (at < hi && n0 + i < p.ff) {
                float s = 0.f, u = 0.f;
#pragma unroll
                for (int ww = 0; ww < MG_WARPS; ww++) {
                    s += red[0][ww][i * 8 + b];
                    if (GATED) u += red[GATED ? 1 : 0][ww][i * 8 + b];
                }
                // the same roundings as the kernel above
                s = __bfloat162float(__float2bfloat16_rn(s));
                u = __bfloat162float(__float2bfloat16_rn(u));
                ((__nv_bfloat16*)p.act)[(int64_t)at * p.ff + n0 + i] =
                    __float2bfloat16_rn(expert_act(s, u, p.weight_input ? p.weight[at] : 1.f, p.act_kind, p.weight_input, p.limit, p.slope));
            }
        }
        __syncthreads();
    }
}

__global__ void __launch_bounds__(32 * MG_WARPS) moe_down_grouped_mma_kernel(MoeRowsParams p, const int* __restrict__ offsets, float* __restrict__ ys) {
    __shared__ float red[MG_WARPS][16 * 8];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const int n0 = blockIdx.x * 16, e = blockIdx.y, K = p.ff;
    const int lo = offsets[e], hi = offsets[e + 1];
    if (lo == hi) return;
    const int64_t ldw = (int64_t)p.experts * K;
    const int c_lo = min(n0 + g, p.hidden - 1), c_hi = min(n0 + g + 8, p.hidden - 1);
    const __nv_bfloat16* w = (const __nv_bfloat16*)p.down + (int64_t)e * K + t * 8;
    const __nv_bfloat16 *w_lo = w + c_lo * ldw, *w_hi = w + c_hi * ldw;
    const int per = ((K + 31) / 32 + MG_WARPS - 1) / MG_WARPS * 32;
    const int k0 = warp * per, k1 = min(k0 + per, K);
    for (int p0 = lo; p0 < hi; p0 += 8) {
        const __nv_bfloat16* x = (const __nv_bfloat16*)p.act + (int64_t)min(p0 + g, hi - 1) * K + t * 8;
        float acc[4] = {0.f, 0.f, 0.f, 0.f};
        if (k0 < k1) stream_product(acc, w_lo, w_hi, x, k0, k1, t);
        leave_fragment(red[warp], acc, g, t);
        __syncthreads();
        if (threadIdx.x < 128) {
            const int b = threadIdx.x >> 4, i = threadIdx.x & 15, at = p0 + b;
            if (at < hi && n0 + i < p.hidden) {
                float s = 0.f;
#pragma unroll
                for (int ww = 0; ww < MG_WARPS; ww++) s += red[ww][i * 8 + b];
                ys[(int64_t)at * p.hidden + n0 + i] = s;
            }
        }
        __syncthreads();
    }
}

constexpr int GROUP_THREADS = 1024;
constexpr int GROUP_MAX_EXPERTS = 512;

// one CTA: counts of the pairs of each expert, offsets of the experts' groups, and a place in its group for every pair
__global__ void __launch_bounds__(GROUP_THREADS) moe_group_kernel(const int* __restrict__ index, int pairs, int top, int experts,
                                                                 int* __restrict__ offsets, int* __restrict__ place, int* __restrict__ src_row,
                                                                 const float* __restrict__ weight, float* __restrict__ sorted_weight) {
    __shared__ int count[GROUP_MAX_EXPERTS], cursor[GROUP_MAX_EXPERTS];
    const int tid = threadIdx.x;
    for (int e = tid; e < experts; e += GROUP_THREADS) count[e] = 0;
    __syncthreads();
    for (int i = tid; i < pairs; i += GROUP_THREADS) atomicAdd(&count[index[i]], 1);
    __syncthreads();
    if (tid == 0) {
        int at = 0;
        for (int e = 0; e < experts; e++) {
            offsets[e] = at;
            cursor[e] = at;
            at += count[e];
        }
        offsets[experts] = at;
    }
    __syncthreads();
    for (int i = tid; i < pairs; i += GROUP_THREADS) {
        const int at = atomicAdd(&cursor[index[i]], 1);
        place[i] = at;
        src_row[at] = i / top;
        if (sorted_weight) sorted_weight[at] = weight[i];
    }
}

// xs[p, :] = x[src_row[p], :], 16 bytes a thread where rows allow it
template <typename T>
__global__ void moe_gather_kernel(const T* __restrict__ x, int64_t x_stride, const int* __restrict__ src_row, T* __restrict__ xs, int hidden) {
    const int64_t p = blockIdx.x;
    const T* src = x + (int64_t)src_row[p] * x_stride;
    T* dst = xs + p * hidden;
    constexpr int V = 16 / sizeof(T);
    if (!(hidden % V) && !(x_stride % V) && !((uintptr_t)x & 15) && !((uintptr_t)xs & 15)) {
        for (int c = threadIdx.x; c < hidden / V; c += blockDim.x)
            reinterpret_cast<uint4*>(dst)[c] = reinterpret_cast<const uint4*>(src)[c];
    } else {
        for (int c = threadIdx.x; c < hidden; c += blockDim.x) dst[c] = src[c];
    }
}

// z times the normal law's distribution function at z
__device__ __forceinline__ float gelu_erf(float z) { return 0.5f * z * (1.f + erff(z * 0.70710678118654752f)); }

// V elements a thread: 16 bytes where rows allow it
template <typename T, int V>
__global__ void gelu_kernel(T* __restrict__ z, int64_t n) {
    pdl_wait();
    pdl_trigger();
    const int64_t i = ((int64_t)blockIdx.x * blockDim.x + threadIdx.x) * V;
    if (i >= n) return;
    if constexpr (V > 1) {
        uint4 raw = *reinterpret_cast<const uint4*>(z + i);
        T* t = reinterpret_cast<T*>(&raw);
#pragma unroll
        for (int u = 0; u < V; u++) t[u] = from_f32<T>(gelu_erf(to_f32<T>(t[u])));
        *reinterpret_cast<uint4*>(z + i) = raw;
    } else {
        z[i] = from_f32<T>(gelu_erf(to_f32<T>(z[i])));
    }
}

template <typename T>
__global__ void relu2_kernel(T* __restrict__ z, int64_t n) {
    const int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    const float v = fmaxf(to_f32<T>(z[i]), 0.f);
    z[i] = from_f32<T>(v * v);
}

// out[r, :] = sum_k weight[r, k] * ys[place[r * top + k], :], in the order of k
__global__ void moe_combine_kernel(const float* __restrict__ ys, const int* __restrict__ place, const float* __restrict__ weight,
                                   float* __restrict__ out, int64_t out_stride, int top, int hidden) {
    const int64_t r = blockIdx.x;
    for (int c = threadIdx.x; c < hidden; c += blockDim.x) {
        float a = 0.f;
        for (int k = 0; k < top; k++) a = fmaf(weight ? weight[r * top + k] : 1.f, ys[(int64_t)place[r * top + k] * hidden + c], a);
        out[r * out_stride + c] = a;
    }
}

}  // namespace

GB_API int gb_moe_group(const int* index, int rows, int top, int experts, int* offsets, int* place, int* src_row, cudaStream_t stream) {
    return gb_moe_group_weights(index, rows, top, experts, offsets, place, src_row, nullptr, nullptr, stream);
}

// The same, and the pairs' weights in sorted order beside them (sorted_weight[place[i]] = weight[i]) if both are given.
GB_API int gb_moe_group_weights(const int* index, int rows, int top, int experts, int* offsets, int* place, int* src_row, const float* weight,
                                float* sorted_weight, cudaStream_t stream) {
    if (rows <= 0) return 0;
    if (experts <= 0 || experts > GROUP_MAX_EXPERTS || top <= 0) GB_REFUSE("moe_group: %d experts, %d a token", experts, top);
    if ((weight != nullptr) != (sorted_weight != nullptr)) GB_REFUSE("moe_group: weights in and out go together");
    moe_group_kernel<<<1, GROUP_THREADS, 0, stream>>>(index, rows * top, top, experts, offsets, place, src_row, weight, sorted_weight);
    GB_CHECK_LAUNCH("moe_group");
    return 0;
}

GB_API int gb_moe_gather(const void* x, int64_t x_stride, const int* src_row, void* xs, int pairs, int hidden, int dtype, cudaStream_t stream) {
    if (pairs <= 0) return 0;
    if (dtype == GB_F32)
        moe_gather_kernel<float><<<pairs, 128, 0, stream>>>((const float*)x, x_stride, src_row, (float*)xs, hidden);
    else if (dtype == GB_BF16)
        moe_gather_kernel<__nv_bfloat16><<<pairs, 128, 0, stream>>>((const __nv_bfloat16*)x, x_stride, src_row, (__nv_bfloat16*)xs, hidden);
    else
        GB_REFUSE("moe_gather: unknown dtype %d", dtype);
    GB_CHECK_LAUNCH("moe_gather");
    return 0;
}

GB_API int gb_relu2(void* z, int64_t n, int dtype, cudaStream_t stream) {
    if (n <= 0) return 0;
    const unsigned blocks = (unsigned)((n + 255) / 256);
    if (dtype == GB_F32)
        relu2_kernel<float><<<blocks, 256, 0, stream>>>((float*)z, n);
    else if (dtype == GB_BF16)
        relu2_kernel<__nv_bfloat16><<<blocks, 256, 0, stream>>>((__nv_bfloat16*)z, n);
    else
        GB_REFUSE("relu2: unknown dtype %d", dtype);
    GB_CHECK_LAUNCH("relu2");
    return 0;
}

GB_API int gb_gelu(void* z, int64_t n, int dtype, cudaStream_t stream) {
    if (n <= 0) return 0;
    const int v = dtype == GB_BF16 ? 8 : 4;
    const bool vec = !(n % v) && !((uintptr_t)z & 15);
    const int64_t threads = vec ? n / v : n, blocks = (threads + 255) / 256;
    if (blocks > 0x7fffffff) GB_REFUSE("gelu: %lld elements are too many for one launch", (long long)n);
    const dim3 grid((unsigned)blocks), block(256);
    if (dtype == GB_F32) {
        if (vec) launch_pdl(gelu_kernel<float, 4>, grid, block, 0, stream, (float*)z, n);
        else launch_pdl(gelu_kernel<float, 1>, grid, block, 0, stream, (float*)z, n);
    } else if (dtype == GB_BF16) {
        if (vec) launch_pdl(gelu_kernel<__nv_bfloat16, 8>, grid, block, 0, stream, (__nv_bfloat16*)z, n);
        else launch_pdl(gelu_kernel<__nv_bfloat16, 1>, grid, block, 0, stream, (__nv_bfloat16*)z, n);
    } else {
        GB_REFUSE("gelu: unknown dtype %d", dtype);
    }
    GB_CHECK_LAUNCH("gelu");
    return 0;
}

GB_API int gb_moe_combine(const float* ys, const int* place, const float* weight, float* out, int64_t out_stride, int rows, int top, int hidden,
                          cudaStream_t stream) {
    if (rows <= 0) return 0;
    moe_combine_kernel<<<rows, 256, 0, stream>>>(ys, place, weight, out, out_stride, top, hidden);
    GB_CHECK_LAUNCH("moe_combine");
    return 0;
}

GB_API int gb_moe_route(const MoeRouteParams* pp, cudaStream_t stream) {
    MoeRouteParams p = *pp;
    if (p.rows <= 0) return 0;
    if (p.experts <= 0 || p.experts > 32 * MAX_EXPERTS_PER_LANE) GB_REFUSE("moe_route: %d experts; 1 to %d", p.experts, 32 * MAX_EXPERTS_PER_LANE);
    if (p.top <= 0 || p.top > p.experts || p.top > 32) GB_REFUSE("moe_route: %d of %d experts a token; at most 32", p.top, p.experts);
    if (!p.logits || !p.dense || !p.index || !p.weight) GB_REFUSE("moe_route: a tensor is missing");
    if (p.groups > 1 && (p.experts % p.groups || p.keep_groups <= 0 || p.keep_groups > p.groups || p.experts / p.groups * p.keep_groups < p.top))
        GB_REFUSE("moe_route: %d of %d experts a token out of the best %d of %d groups", p.top, p.experts, p.keep_groups, p.groups);
    if (p.correction || p.groups > 1)
        moe_route_kernel<true><<<(p.rows + 3) / 4, 128, 0, stream>>>(p);
    else
        moe_route_kernel<false><<<(p.rows + 3) / 4, 128, 0, stream>>>(p);
    GB_CHECK_LAUNCH("moe_route");
    return 0;
}

GB_API int gb_moe_act(const void* up, int64_t up_stride, const float* dense, void* act, int64_t act_stride, int rows, int experts, int ff,
                      int dtype, cudaStream_t stream) {
    return gb_moe_act_kind(up, up_stride, dense, act, act_stride, rows, experts, ff, 0, 0, dtype, stream);
}

// kind 0: weight * relu(up)^2; kind 1: gated, silu(gate) * up with each expert's gate columns ahead of its up columns.
// weight_input 1: the weight multiplies the expert's input instead of its output.  dense null: weights of 1.
GB_API int gb_moe_act_kind(const void* up, int64_t up_stride, const float* dense, void* act, int64_t act_stride, int rows, int experts, int ff,
                           int kind, int weight_input, int dtype, cudaStream_t stream) {
    return gb_moe_act_clamped(up, up_stride, dense, act, act_stride, rows, experts, ff, kind, weight_input, 0.f, 1.f, dtype, stream);
}

// kind 2 as well: g sigmoid(slope g) (v + 1), g = min(gate, limit), v = clamp(up, -limit, limit), columns laid out as for kind 1.
GB_API int gb_moe_act_clamped(const void* up, int64_t up_stride, const float* dense, void* act, int64_t act_stride, int rows, int experts, int ff,
                              int kind, int weight_input, float limit, float slope, int dtype, cudaStream_t stream) {
    if (rows <= 0) return 0;
    if (experts <= 0 || ff <= 0) GB_REFUSE("moe_act: %d experts of %d", experts, ff);
    if (kind < 0 || kind > 2) GB_REFUSE("moe_act: unknown activation %d", kind);
    const int64_t total = (int64_t)rows * experts * ff;
    const unsigned blocks = (unsigned)((total + 255) / 256);
    if (dtype == GB_F32)
        moe_act_kernel<float><<<blocks, 256, 0, stream>>>((const float*)up, up_stride, dense, (float*)act, act_stride, rows, experts, ff, kind, weight_input, limit, slope);
    else if (dtype == GB_BF16)
        moe_act_kernel<__nv_bfloat16><<<blocks, 256, 0, stream>>>((const __nv_bfloat16*)up, up_stride, dense, (__nv_bfloat16*)act, act_stride,
                                                                  rows, experts, ff, kind, weight_input, limit, slope);
    else
        GB_REFUSE("moe_act: unknown dtype %d", dtype);
    GB_CHECK_LAUNCH("moe_act");
    return 0;
}

GB_API int gb_moe_rows(const MoeRowsParams* pp, int dtype, int w_dtype, cudaStream_t stream) {
    MoeRowsParams p = *pp;
    if (p.rows <= 0) return 0;
    if (p.experts <= 0 || p.top <= 0 || p.ff <= 0 || p.hidden <= 0) GB_REFUSE("moe_rows: %d experts, %d a token, %d x %d", p.experts, p.top, p.ff, p.hidden);
    if (!p.x || !p.up || !p.down || !p.act || !p.out || !p.index || !p.weight) GB_REFUSE("moe_rows: a tensor is missing");
    dim3 ugrid((p.ff + 3) / 4, p.rows * p.top), dgrid((p.hidden + 3) / 4, p.rows);
    if (ugrid.y > 65535) GB_REFUSE("moe_rows: %d rows exceed one launch", p.rows);
    if (dtype == GB_BF16 && w_dtype == GB_BF16) {
        moe_up_rows_kernel<__nv_bfloat16, __nv_bfloat16><<<ugrid, 128, 0, stream>>>(p);
        moe_down_rows_kernel<__nv_bfloat16, __nv_bfloat16><<<dgrid, 128, 0, stream>>>(p);
    } else if (dtype == GB_F32 && w_dtype == GB_F32) {
        moe_up_rows_kernel<float, float><<<ugrid, 128, 0, stream>>>(p);
        moe_down_rows_kernel<float, float><<<dgrid, 128, 0, stream>>>(p);
    } else {
        GB_REFUSE("moe_rows: activations of dtype %d with weights of dtype %d", dtype, w_dtype);
    }
    GB_CHECK_LAUNCH("moe_rows");
    return 0;
}

// The few-row feed-forward with the pairs sorted by expert: `offsets` and `src_row` as moe_group left them, `ys`
// float32 [rows * top, hidden] receives every pair's output at its sorted place (moe_combine adds them up).
GB_API int gb_moe_rows_grouped(const MoeRowsParams* pp, const int* offsets, const int* src_row, float* ys, int dtype, int w_dtype,
                               cudaStream_t stream) {
    MoeRowsParams p = *pp;
    if (p.rows <= 0) return 0;
    if (p.experts <= 0 || p.experts > 65535 || p.top <= 0 || p.ff <= 0 || p.hidden <= 0) GB_REFUSE("moe_rows: %d experts, %d a token, %d x %d", p.experts, p.top, p.ff, p.hidden);
    if (!p.x || !p.up || !p.down || !p.act || !offsets || !src_row || !ys || (p.weight_input && !p.weight)) GB_REFUSE("moe_rows: a tensor is missing");
    dim3 ugrid((p.ff + 3) / 4, p.experts), dgrid((p.hidden + 3) / 4, p.experts);
    const bool aligned = !(p.hidden & 7) && !(p.ff & 7) && !(p.x_stride & 7) &&
                         !(((uintptr_t)p.x | (uintptr_t)p.up | (uintptr_t)p.down | (uintptr_t)p.act) & 15);
    if (dtype == GB_BF16 && w_dtype == GB_BF16 && aligned) {
        dim3 um((p.ff + 15) / 16, p.experts), dm((p.hidden + 15) / 16, p.experts);
        if (p.act_kind != 0)
            moe_up_grouped_mma_kernel<true><<<um, 32 * MG_WARPS, 0, stream>>>(p, offsets, src_row);
        else
            moe_up_grouped_mma_kernel<false><<<um, 32 * MG_WARPS, 0, stream>>>(p, offsets, src_row);
        moe_down_grouped_mma_kernel<<<dm, 32 * MG_WARPS, 0, stream>>>(p, offsets, ys);
    } else if (dtype == GB_BF16 && w_dtype == GB_BF16) {
        moe_up_grouped_kernel<__nv_bfloat16, __nv_bfloat16><<<ugrid, 128, 0, stream>>>(p, offsets, src_row);
        moe_down_grouped_kernel<__nv_bfloat16, __nv_bfloat16><<<dgrid, 128, 0, stream>>>(p, offsets, ys);
    } else if (dtype == GB_F32 && w_dtype == GB_F32) {
        moe_up_grouped_kernel<float, float><<<ugrid, 128, 0, stream>>>(p, offsets, src_row);
        moe_down_grouped_kernel<float, float><<<dgrid, 128, 0, stream>>>(p, offsets, ys);
    } else {
        GB_REFUSE("moe_rows: activations of dtype %d with weights of dtype %d", dtype, w_dtype);
    }
    GB_CHECK_LAUNCH("moe_rows_grouped");
    return 0;
}
