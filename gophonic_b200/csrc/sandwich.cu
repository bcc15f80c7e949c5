// Row-wise kernels of blocks that norm in front of and behind their sublayers, convolve what a mixer reads over a few
// tokens and weigh the results of all layers so far into what goes on; and the cap on a head's logits.
//
// sandwich_rows:  between two sublayers, one pass over a row of the float32 residual: the sublayer's output (or the sum of two
//                 outputs side by side, each over its own root mean square and times a weight) over its root
//                 mean square and times its weight joins the residual (the sum may be stored: a layer's result), the planes
//                 of the earlier results and this one are summed with one weight each (stored if asked), and the sum is
//                 normed for whoever reads it next.  For single tokens the normed row also passes the convolution, whose
//                 earlier inputs are in the sequence's state, and the state moves on.  A CTA owns a row; a thread keeps its
//                 share of the row in registers from the first load to the last store.
// conv_rows:      the convolution for packed rows of prompts: a tap reaches back into the step's own rows of the sequence
//                 and, before its first row, into the state; conv_rows_state then moves the state on.
// soft_cap:       z <- cap tanh(z / cap).
//
// Everything is float32; a row's result depends on that row (and its sequence's earlier rows) alone, and the order of every
// sum is fixed by the row's width.
#include "api.h"
#include "common.cuh"

#include <math.h>

namespace {

constexpr int MAX_TAPS = 16;

template <int THREADS>
__device__ __forceinline__ float block_sum(float v, float* part) {
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.f;
#pragma unroll
    for (int i = 0; i < THREADS / 32; i++) t += part[i];   // every thread adds the warp sums in the same order
    return t;
}

// the same for two values at once
template <int THREADS>
__device__ __forceinline__ void block_sum2(float& a, float& b, float* part_a, float* part_b) {
    a = warp_sum(a);
    b = warp_sum(b);
    if ((threadIdx.x & 31) == 0) part_a[threadIdx.x >> 5] = a, part_b[threadIdx.x >> 5] = b;
    __syncthreads();
    a = b = 0.f;
#pragma unroll
    for (int i = 0; i < THREADS / 32; i++) a += part_a[i], b += part_b[i];
}

template <int V>
__device__ __forceinline__ void load_v(const float* __restrict__ src, float* v) {
    if (V == 4) {
        const float4 a = *reinterpret_cast<const float4*>(src);
        v[0] = a.x, v[V == 4 ? 1 : 0] = a.y, v[V == 4 ? 2 : 0] = a.z, v[V == 4 ? 3 : 0] = a.w;
    } else {
        v[0] = *src;
    }
}
template <int V>
__device__ __forceinline__ void store_v(float* dst, const float* v) {
    if (V == 4)
        *reinterpret_cast<float4*>(dst) = make_float4(v[0], v[V == 4 ? 1 : 0], v[V == 4 ? 2 : 0], v[V == 4 ? 3 : 0]);
    else
        *dst = v[0];
}
template <int V>
__device__ __forceinline__ void store_v(__nv_bfloat16* dst, const float* v) {
    if (V == 4) {
        const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[V == 4 ? 1 : 0]), b = __floats2bfloat162_rn(v[V == 4 ? 2 : 0], v[V == 4 ? 3 : 0]);
        uint2 u;
        u.x = *reinterpret_cast<const uint32_t*>(&a);
        u.y = *reinterpret_cast<const uint32_t*>(&b);
        *reinterpret_cast<uint2*>(dst) = u;
    } else {
        *dst = __float2bfloat16_rn(v[0]);
    }
}

// V neighbouring elements a piece, P pieces a thread, V * THREADS elements apart.  PAIR: the sublayer left two outputs, y and y2
template <typename TO, int V, int P, int THREADS, bool PAIR>
__global__ void __launch_bounds__(THREADS) sandwich_rows_kernel(SandwichParams p) {
    pdl_wait();
    pdl_trigger();
    __shared__ float part[PAIR ? 4 : 2][THREADS / 32];
    const int n = p.width;
    const int64_t out_row = blockIdx.x;
    const int64_t row = p.row_index ? p.row_index[out_row] : out_row;
    const int c0 = threadIdx.x * V;
    constexpr int STEP = THREADS * V;

    float x[P][V];       // the weighted sum of the earlier results
#pragma unroll
    for (int k = 0; k < P; k++)
#pragma unroll
        for (int u = 0; u < V; u++) x[k][u] = 0.f;
    if (p.average) {
        const float* plane = p.planes + row * n;
        int j = 0;
        for (; j + 3 < p.n_planes; j += 4) {      // four planes' loads are in flight together
#pragma unroll
            for (int k = 0; k < P; k++) {
                const int c = c0 + k * STEP;
                if (c >= n) continue;
                float t[4][V];
#pragma unroll
                for (int q = 0; q < 4; q++) load_v<V>(plane + (j + q) * p.plane_stride + c, t[q]);
#pragma unroll
                for (int q = 0; q < 4; q++)
#pragma unroll
                    for (int u = 0; u < V; u++) x[k][u] = fmaf(p.average[j + q], t[q][u], x[k][u]);
            }
        }
        for (; j < p.n_planes; j++) {
#pragma unroll
            for (int k = 0; k < P; k++) {
                const int c = c0 + k * STEP;
                if (c >= n) continue;
                float t[V];
                load_v<V>(plane + j * p.plane_stride + c, t);
#pragma unroll
                for (int u = 0; u < V; u++) x[k][u] = fmaf(p.average[j], t[u], x[k][u]);
            }
        }
    }
    float v[P][V];
#pragma unroll
    for (int k = 0; k < P; k++) {
#pragma unroll
        for (int u = 0; u < V; u++) v[k][u] = 0.f;
        const int c = c0 + k * STEP;
        if (c < n) load_v<V>(p.base + row * n + c, v[k]);
    }
    if (p.y) {
        float y[P][V];
        float ss = 0.f;
#pragma unroll
        for (int k = 0; k < P; k++) {
#pragma unroll
            for (int u = 0; u < V; u++) y[k][u] = 0.f;
            const int c = c0 + k * STEP;
            if (c < n) load_v<V>(p.y + row * n + c, y[k]);
#pragma unroll
            for (int u = 0; u < V; u++) ss += y[k][u] * y[k][u];
        }
        if (PAIR) {
            float y2[P][V];
            float s2 = 0.f;
#pragma unroll
            for (int k = 0; k < P; k++) {
#pragma unroll
                for (int u = 0; u < V; u++) y2[k][u] = 0.f;
                const int c = c0 + k * STEP;
                if (c < n) load_v<V>(p.y2 + row * n + c, y2[k]);
#pragma unroll
                for (int u = 0; u < V; u++) s2 += y2[k][u] * y2[k][u];
            }
            block_sum2<THREADS>(ss, s2, part[PAIR ? 2 : 0], part[PAIR ? 3 : 0]);
            const float i1 = 1.0f / sqrtf(ss / (float)n + p.pair_eps), i2 = 1.0f / sqrtf(s2 / (float)n + p.pair_eps);
            ss = 0.f;
#pragma unroll
            for (int k = 0; k < P; k++) {
                const int c = c0 + k * STEP;
                if (c >= n) continue;
                float w1[V], w2[V];
                load_v<V>(p.pair_w + c, w1);
                load_v<V>(p.pair_w2 + c, w2);
#pragma unroll
                for (int u = 0; u < V; u++) {
                    y[k][u] = fmaf(y[k][u] * i1, w1[u], y2[k][u] * i2 * w2[u]);
                    ss += y[k][u] * y[k][u];
                }
            }
        }
        const float inv = 1.0f / sqrtf(block_sum<THREADS>(ss, part[0]) / (float)n + p.y_eps);
#pragma unroll
        for (int k = 0; k < P; k++) {
            const int c = c0 + k * STEP;
            if (c >= n) continue;
            float w[V];
            load_v<V>(p.y_w + c, w);
#pragma unroll
            for (int u = 0; u < V; u++) v[k][u] += y[k][u] * inv * w[u];
        }
    }
    const float own = p.average ? p.average[p.n_planes] : 1.f;
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < P; k++) {
        const int c = c0 + k * STEP;
        if (c >= n) continue;
        if (p.result) store_v<V>(p.result + row * n + c, v[k]);
#pragma unroll
        for (int u = 0; u < V; u++) {
            x[k][u] = p.average ? fmaf(own, v[k][u], x[k][u]) : v[k][u];
            ss += x[k][u] * x[k][u];
        }
        if (p.x_out) store_v<V>(p.x_out + row * n + c, x[k]);
    }
    const float inv = 1.0f / sqrtf(block_sum<THREADS>(ss, part[1]) / (float)n + p.norm_eps);
    float* st = nullptr;
    if (p.conv_w && p.taps > 1) {
        int slot = p.seq_slot[p.row_seq[row]];
        if (!gb_check(slot, p.max_slots, GB_CHECK_SLOT)) slot = 0;
        st = p.state + (int64_t)slot * p.state_slot_stride;
    }
#pragma unroll
    for (int k = 0; k < P; k++) {
        const int c = c0 + k * STEP;
        if (c >= n) continue;
        float w[V], h[V];
        load_v<V>(p.norm_w + c, w);
#pragma unroll
        for (int u = 0; u < V; u++) h[u] = x[k][u] * inv * w[u];
        if (p.conv_w) {
            float a[V], cw[V];
#pragma unroll
            for (int u = 0; u < V; u++) a[u] = 0.f;
            for (int j = 0; j + 1 < p.taps; j++) {
                float s[V];
                load_v<V>(st + (int64_t)j * n + c, s);
                load_v<V>(p.conv_w + (int64_t)j * n + c, cw);
#pragma unroll
                for (int u = 0; u < V; u++) a[u] = fmaf(cw[u], s[u], a[u]);
                if (j > 0) store_v<V>(st + (int64_t)(j - 1) * n + c, s);
            }
            if (p.taps > 1) store_v<V>(st + (int64_t)(p.taps - 2) * n + c, h);
            load_v<V>(p.conv_w + (int64_t)(p.taps - 1) * n + c, cw);
#pragma unroll
            for (int u = 0; u < V; u++) h[u] += fmaf(cw[u], h[u], a[u]);
        }
        store_v<V>((TO*)p.out + out_row * n + c, h);
    }
}

template <typename TO, int V, int P, int THREADS>
int launch_rows(const SandwichParams& p, cudaStream_t stream) {
    if (p.y2)
        launch_pdl(sandwich_rows_kernel<TO, V, P, THREADS, true>, dim3(p.rows), dim3(THREADS), 0, stream, p);
    else
        launch_pdl(sandwich_rows_kernel<TO, V, P, THREADS, false>, dim3(p.rows), dim3(THREADS), 0, stream, p);
    GB_CHECK_LAUNCH("sandwich_rows");
    return 0;
}

constexpr int MANY_ROWS = 592;     // from this many rows on, CTAs of 256 threads fill the GPU; below, 512 threads share a row's latency

template <typename TO>
int dispatch_rows(const SandwichParams& p, cudaStream_t stream) {
    const int n = p.width;
    const uintptr_t all = (uintptr_t)p.base | (uintptr_t)p.y | (uintptr_t)p.y_w | (uintptr_t)p.result | (uintptr_t)p.planes | (uintptr_t)p.x_out |
                          (uintptr_t)p.norm_w | (uintptr_t)p.out | (uintptr_t)p.conv_w | (uintptr_t)p.state |
                          (uintptr_t)p.y2 | (uintptr_t)p.pair_w | (uintptr_t)p.pair_w2;
    if (!(n & 3) && !(all & 15) && !(p.plane_stride & 3) && !(p.state_slot_stride & 3)) {
        if (p.rows < MANY_ROWS && n > 1024) {
            if (n <= 2048) return launch_rows<TO, 4, 1, 512>(p, stream);
            if (n <= 4096) return launch_rows<TO, 4, 2, 512>(p, stream);
            if (n <= 8192) return launch_rows<TO, 4, 4, 512>(p, stream);
        }
        if (n <= 1024) return launch_rows<TO, 4, 1, 256>(p, stream);
        if (n <= 2048) return launch_rows<TO, 4, 2, 256>(p, stream);
        if (n <= 4096) return launch_rows<TO, 4, 4, 256>(p, stream);
        if (n <= 8192) return launch_rows<TO, 4, 8, 256>(p, stream);
        if (n <= 16384) return launch_rows<TO, 4, 16, 256>(p, stream);
    } else {
        if (n <= 512) return launch_rows<TO, 1, 2, 256>(p, stream);
        if (n <= 4096) return launch_rows<TO, 1, 16, 256>(p, stream);
        if (n <= 16384) return launch_rows<TO, 1, 64, 256>(p, stream);
    }
    GB_REFUSE("sandwich_rows: rows of %d; at most 16384", n);
}

template <typename TO, int V>
__global__ void __launch_bounds__(256) conv_rows_kernel(const float* __restrict__ h, const float* __restrict__ conv_w, int taps,
                                                        const float* __restrict__ state, int64_t state_slot_stride, int max_slots,
                                                        TO* __restrict__ out, int n, const int* __restrict__ row_seq,
                                                        const int* __restrict__ seq_slot, const int* __restrict__ seq_q_start) {
    const int64_t row = blockIdx.x;
    const int seq = row_seq[row];
    const int local = (int)(row - seq_q_start[seq]);     // the row's place in its sequence's portion
    int slot = seq_slot[seq];
    if (taps > 1 && !gb_check(slot, max_slots, GB_CHECK_SLOT)) slot = 0;      // one tap reaches nothing back: there is no state
    const float* st = state + (int64_t)slot * state_slot_stride;
    for (int c = threadIdx.x * V; c < n; c += 256 * V) {
        float a[V], x[V], cw[V];
#pragma unroll
        for (int u = 0; u < V; u++) a[u] = 0.f;
        for (int j = 0; j < taps; j++) {
            const int back = taps - 1 - j;
            load_v<V>(back <= local ? h + (row - back) * n + c : st + (int64_t)(taps - 1 + local - back) * n + c, x);
            load_v<V>(conv_w + (int64_t)j * n + c, cw);
#pragma unroll
            for (int u = 0; u < V; u++) a[u] = fmaf(cw[u], x[u], a[u]);
        }
        // the last tap's row is this one
#pragma unroll
        for (int u = 0; u < V; u++) x[u] += a[u];
        store_v<V>(out + row * n + c, x);
    }
}

// The same for convolutions of few taps on rows that vectors fit: a thread owns four channels of CONV_ROWS consecutive
// packed rows and loads them, and the TAPS - 1 rows ahead of them, once; a tap that reaches ahead of its sequence's portion
// takes the state instead.
constexpr int CONV_ROWS = 8;

template <typename TO, int TAPS>
__global__ void __launch_bounds__(256) conv_rows_window_kernel(const float* __restrict__ h, const float* __restrict__ conv_w,
                                                               const float* __restrict__ state, int64_t state_slot_stride, int max_slots,
                                                               TO* __restrict__ out, int rows, int n, const int* __restrict__ row_seq,
                                                               const int* __restrict__ seq_slot, const int* __restrict__ seq_q_start) {
    pdl_wait();
    pdl_trigger();
    const int c = (blockIdx.y * 256 + threadIdx.x) * 4;
    const int64_t r0 = (int64_t)blockIdx.x * CONV_ROWS;
    if (c >= n) return;
    float x[CONV_ROWS + TAPS - 1][4], w[TAPS][4];
    int seq[CONV_ROWS];
#pragma unroll
    for (int i = 0; i < CONV_ROWS + TAPS - 1; i++) {
        const int64_t r = r0 + i - (TAPS - 1);
        if (r >= 0 && r < rows) load_v<4>(h + r * n + c, x[i]);
    }
#pragma unroll
    for (int j = 0; j < TAPS; j++) load_v<4>(conv_w + (int64_t)j * n + c, w[j]);
#pragma unroll
    for (int i = 0; i < CONV_ROWS; i++) seq[i] = r0 + i < rows ? row_seq[r0 + i] : 0;
#pragma unroll
    for (int i = 0; i < CONV_ROWS; i++) {
        if (r0 + i >= rows) continue;
        const int local = (int)(r0 + i - seq_q_start[seq[i]]);
        float a[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int j = 0; j < TAPS; j++) {
            const int back = TAPS - 1 - j;
            float t[4];
#pragma unroll
            for (int u = 0; u < 4; u++) t[u] = x[i + j][u];
            if (back > local) {
                int slot = seq_slot[seq[i]];
                if (!gb_check(slot, max_slots, GB_CHECK_SLOT)) slot = 0;
                load_v<4>(state + (int64_t)slot * state_slot_stride + (int64_t)(TAPS - 1 + local - back) * n + c, t);
            }
#pragma unroll
            for (int u = 0; u < 4; u++) a[u] = fmaf(w[j][u], t[u], a[u]);
        }
        float o[4];
#pragma unroll
        for (int u = 0; u < 4; u++) o[u] = x[i + TAPS - 1][u] + a[u];
        store_v<4>(out + (r0 + i) * n + c, o);
    }
}

// the last taps - 1 rows of every sequence's portion into its state; a portion shorter than that pushes the older rows on
__global__ void conv_rows_state_kernel(const float* __restrict__ h, int taps, float* __restrict__ state, int64_t state_slot_stride, int max_slots,
                                       int n, const int* __restrict__ seq_slot, const int* __restrict__ seq_q_start,
                                       const int* __restrict__ seq_q_len) {
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    const int seq = blockIdx.y;
    if (c >= n) return;
    const int len = seq_q_len[seq];
    if (len <= 0) return;
    const int64_t start = seq_q_start[seq];
    int slot = seq_slot[seq];
    if (!gb_check(slot, max_slots, GB_CHECK_SLOT)) slot = 0;
    float* st = state + (int64_t)slot * state_slot_stride;
    for (int s = 0; s + 1 < taps; s++) {      // ascending: a place is read before it is written
        const int at = len - (taps - 1) + s;
        st[(int64_t)s * n + c] = at >= 0 ? h[(start + at) * n + c] : st[(int64_t)(s + len) * n + c];
    }
}

__global__ void soft_cap_kernel(float* __restrict__ z, int64_t n, float cap) {
    const int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) z[i] = cap * tanhf(z[i] / cap);
}

}  // namespace

GB_API int gb_sandwich_rows(const SandwichParams* pp, int out_dtype, cudaStream_t stream) {
    SandwichParams p = *pp;
    if (p.rows <= 0) return 0;
    if (p.width <= 0 || p.n_planes < 0) GB_REFUSE("sandwich_rows: rows of %d, %d planes", p.width, p.n_planes);
    if (!p.base || !p.out || !p.norm_w || (p.y && !p.y_w) || (p.average && p.n_planes > 0 && !p.planes)) GB_REFUSE("sandwich_rows: a tensor is missing");
    if (p.y2 && (!p.y || !p.pair_w || !p.pair_w2)) GB_REFUSE("sandwich_rows: two outputs side by side need both and their weights");
    if (p.row_index && (p.result || p.x_out || p.conv_w)) GB_REFUSE("sandwich_rows: gathered rows are only read");
    if (p.conv_w && (p.taps <= 0 || p.taps > MAX_TAPS)) GB_REFUSE("sandwich_rows: %d taps; 1 to %d", p.taps, MAX_TAPS);
    if (p.conv_w && (!p.row_seq || !p.seq_slot || (p.taps > 1 && (!p.state || p.state_slot_stride < (int64_t)(p.taps - 1) * p.width))))
        GB_REFUSE("sandwich_rows: the state has no room for %d rows of %d", p.taps - 1, p.width);
    if (out_dtype == GB_F32) return dispatch_rows<float>(p, stream);
    if (out_dtype == GB_BF16) return dispatch_rows<__nv_bfloat16>(p, stream);
    GB_REFUSE("sandwich_rows: unknown dtype %d", out_dtype);
}

GB_API int gb_conv_rows(const float* h, const float* conv_w, int taps, float* state, int64_t state_slot_stride, int max_slots, void* out, int out_dtype,
                        int rows, int width, int nseq, const int* row_seq, const int* seq_slot, const int* seq_q_start, const int* seq_q_len,
                        cudaStream_t stream) {
    if (rows <= 0) return 0;
    if (taps <= 0 || taps > MAX_TAPS) GB_REFUSE("conv_rows: %d taps; 1 to %d", taps, MAX_TAPS);
    if (taps > 1 && (!state || state_slot_stride < (int64_t)(taps - 1) * width)) GB_REFUSE("conv_rows: the state has no room for %d rows of %d", taps - 1, width);
    if (nseq > 65535) GB_REFUSE("conv_rows: %d sequences exceed one launch", nseq);
    const bool vec = !(width & 3) && !(((uintptr_t)h | (uintptr_t)conv_w | (uintptr_t)state | (uintptr_t)out) & 15) && !(state_slot_stride & 3);
#define GB_WINDOW(TO, TAPS)                                                                                                                          \
    launch_pdl(conv_rows_window_kernel<TO, TAPS>, dim3(ceil_div(rows, CONV_ROWS), ceil_div(width, 1024)), dim3(256), 0, stream, h, conv_w,            \
               (const float*)state, state_slot_stride, max_slots, (TO*)out, rows, width, row_seq, seq_slot, seq_q_start)
#define GB_WINDOWS(TO)                       \
    switch (taps) {                          \
        case 2: GB_WINDOW(TO, 2); break;     \
        case 3: GB_WINDOW(TO, 3); break;     \
        default: GB_WINDOW(TO, 4); break;    \
    }
#define GB_CONV(TO, V) \
    conv_rows_kernel<TO, V><<<rows, 256, 0, stream>>>(h, conv_w, taps, state, state_slot_stride, max_slots, (TO*)out, width, row_seq, seq_slot, seq_q_start)
    const bool window = vec && taps >= 2 && taps <= 4 && rows >= 64 && ceil_div(width, 1024) <= 65535;
    if (out_dtype != GB_F32 && out_dtype != GB_BF16) GB_REFUSE("conv_rows: unknown dtype %d", out_dtype);
    if (window) {
        if (out_dtype == GB_F32) GB_WINDOWS(float) else GB_WINDOWS(__nv_bfloat16)
    } else if (out_dtype == GB_F32) {
        if (vec) GB_CONV(float, 4); else GB_CONV(float, 1);
    } else {
        if (vec) GB_CONV(__nv_bfloat16, 4); else GB_CONV(__nv_bfloat16, 1);
    }
#undef GB_CONV
#undef GB_WINDOWS
#undef GB_WINDOW
    GB_CHECK_LAUNCH("conv_rows");
    if (taps > 1) {
        conv_rows_state_kernel<<<dim3(ceil_div(width, 256), nseq), 256, 0, stream>>>(h, taps, state, state_slot_stride, max_slots, width, seq_slot,
                                                                                    seq_q_start, seq_q_len);
        GB_CHECK_LAUNCH("conv_rows_state");
    }
    return 0;
}

GB_API int gb_soft_cap(float* z, int64_t n, float cap, cudaStream_t stream) {
    if (n <= 0) return 0;
    if (!(cap > 0.f)) GB_REFUSE("soft_cap: a cap of %g", (double)cap);
    soft_cap_kernel<<<(unsigned)((n + 255) / 256), 256, 0, stream>>>(z, n, cap);
    GB_CHECK_LAUNCH("soft_cap");
    return 0;
}

// the checked build's record of the first index this file's kernels found out of bounds
GB_CHECK_READER(gb_checked_status_sandwich)
