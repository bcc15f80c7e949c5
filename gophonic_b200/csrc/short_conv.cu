// The short causal convolution over time on projected heads, and what follows it up to the mixer's arithmetic, in one pass.
//
// Rows hold q heads, then k heads (both d wide), then v heads (dv wide).  Per channel, with an optional bias b in the
// projection and the activation act (none, or silu):
//
//     u_t = projected_t + b,   y_t = act( sum_j w[j] u_(t - taps + 1 + j) )         (no weights: y_t = act(u_t))
//
// then, per q and k head: a rotation of its first `rot` channels (neighbouring channels together, or channel i with i + rot / 2),
// a norm behind it (x / sqrt(mean x^2 + eps), or the unit vector x / sqrt(sum x^2 + eps)), and on q a factor.  The heads go
// either where attention reads them (q into a buffer, k and v into the paged cache) or, in float32 whatever the activation
// dtype, into packed rows for a recurrence.  All arithmetic is float32.
//
// A tap reaches back into the step's own rows of the same sequence and, before its first row, into the sequence's state: its
// last taps - 1 rows u, oldest first, zero at the start.  In a step of single tokens the same kernel moves the state on;
// otherwise a second kernel does when the first is through, so that a prompt cut into steps sees the same inputs as a whole one.
//
// A warp owns one head of ROWS consecutive packed rows and two neighbouring channels a lane (and 64 further on): it loads the
// rows and the taps - 1 ahead of them once, all loads in flight together.
#include "api.h"
#include "common.cuh"

#include <math.h>

namespace {

constexpr int MAX_TAPS = 16;
constexpr int MAX_HEAD = 256;
constexpr int WARPS = 4;

__device__ __forceinline__ float silu_f(float x) { return __fdividef(x, 1.f + expf(-x)); }     // a quotient good to two units in the last place

struct Pair {
    float a, b;
};

template <typename T>
__device__ __forceinline__ Pair load_pair(const T* p, int n, bool vec);   // n: channels that are there (0, 1 or 2)
template <>
__device__ __forceinline__ Pair load_pair<float>(const float* p, int n, bool vec) {
    if (vec && n == 2) {
        const float2 v = *reinterpret_cast<const float2*>(p);
        return {v.x, v.y};
    }
    return {n > 0 ? p[0] : 0.f, n > 1 ? p[1] : 0.f};
}
template <>
__device__ __forceinline__ Pair load_pair<__nv_bfloat16>(const __nv_bfloat16* p, int n, bool vec) {
    if (vec && n == 2) {
        const __nv_bfloat162 v = *reinterpret_cast<const __nv_bfloat162*>(p);
        return {__low2float(v), __high2float(v)};
    }
    return {n > 0 ? __bfloat162float(p[0]) : 0.f, n > 1 ? __bfloat162float(p[1]) : 0.f};
}
template <typename T>
__device__ __forceinline__ void store_pair(T* p, Pair v, int n, bool vec);
template <>
__device__ __forceinline__ void store_pair<float>(float* p, Pair v, int n, bool vec) {
    if (vec && n == 2) {
        *reinterpret_cast<float2*>(p) = make_float2(v.a, v.b);
        return;
    }
    if (n > 0) p[0] = v.a;
    if (n > 1) p[1] = v.b;
}
template <>
__device__ __forceinline__ void store_pair<__nv_bfloat16>(__nv_bfloat16* p, Pair v, int n, bool vec) {
    if (vec && n == 2) {
        *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v.a, v.b);
        return;
    }
    if (n > 0) p[0] = __float2bfloat16_rn(v.a);
    if (n > 1) p[1] = __float2bfloat16_rn(v.b);
}

// two channels that are there, at an even place of an aligned row
template <typename T>
__device__ __forceinline__ Pair load_two(const T* p);
template <>
__device__ __forceinline__ Pair load_two<float>(const float* p) {
    const float2 v = __ldg(reinterpret_cast<const float2*>(p));
    return {v.x, v.y};
}
template <>
__device__ __forceinline__ Pair load_two<__nv_bfloat16>(const __nv_bfloat16* p) {
    const unsigned raw = __ldg(reinterpret_cast<const unsigned*>(p));
    const __nv_bfloat162 v = *reinterpret_cast<const __nv_bfloat162*>(&raw);
    return {__low2float(v), __high2float(v)};
}

__device__ __forceinline__ int64_t page_at(const ShortConvParams& p, int slot, int pos) {
    return page_of(block_table_row(p.block_table, p.bt_stride, slot, p.max_slots), pos, p.bt_stride, p.pages);
}

// which head of the row: kind 0 q, 1 k, 2 v; c0 its first channel, n its width, at its number among its kind
struct Head {
    int kind, c0, n, at;
};
__device__ __forceinline__ Head head_of(const ShortConvParams& p, int hh) {
    if (hh < p.q_heads) return {0, hh * p.d, p.d, hh};
    if (hh < p.q_heads + p.k_heads) return {1, hh * p.d, p.d, hh - p.q_heads};
    const int v = hh - p.q_heads - p.k_heads;
    return {2, (p.q_heads + p.k_heads) * p.d + v * p.dv, p.dv, v};
}

// activation, rotation, norm and store of one row of one head, two channels a lane and piece.  CACHE: q into the buffer, k and v
// into the cache (`page`: the page of the row's position); else float32 rows.  HALF: channels i and i + rot / 2 may turn together
template <typename T, int NE, bool CACHE, bool HALF>
__device__ __forceinline__ void finish_head(const ShortConvParams& p, const Head& hd, int64_t row, int pos, int64_t page, Pair (&y)[NE], float* sh, int lane,
                                            bool vec) {
    if (p.silu) {
#pragma unroll
        for (int e = 0; e < NE; e++) y[e] = {silu_f(y[e].a), silu_f(y[e].b)};
    }
    if (hd.kind != 2) {
        if (p.rot > 0) {
            const int half = p.rot / 2;
            const int tpos = gb_check(pos, p.table_positions, GB_CHECK_ROPE_POSITION) ? pos : 0;
            const float* ct = p.cos_t + (int64_t)tpos * half;
            const float* st = p.sin_t + (int64_t)tpos * half;
            if (!HALF || p.pairs) {
#pragma unroll
                for (int e = 0; e < NE; e++) {
                    const int j = lane + 32 * e;       // channels 2j and 2j + 1
                    if (j < half) {
                        const float c = __ldg(ct + j), s = __ldg(st + j);
                        y[e] = {y[e].a * c - y[e].b * s, y[e].b * c + y[e].a * s};
                    }
                }
            } else if constexpr (HALF) {
                __syncwarp();
#pragma unroll
                for (int e = 0; e < NE; e++) {
                    const int i = 2 * (lane + 32 * e);
                    if (i < hd.n) sh[i] = y[e].a;
                    if (i + 1 < hd.n) sh[i + 1] = y[e].b;
                }
                __syncwarp();
                auto turned = [&](int i, float own) {
                    if (i >= p.rot) return own;
                    const int j = i < half ? i : i - half;
                    return i < half ? own * ct[j] - sh[i + half] * st[j] : own * ct[j] + sh[i - half] * st[j];
                };
#pragma unroll
                for (int e = 0; e < NE; e++) {
                    const int i = 2 * (lane + 32 * e);
                    y[e] = {turned(i, y[e].a), turned(i + 1, y[e].b)};
                }
            }
        }
        if (p.norm) {
            float ss = 0.f;
#pragma unroll
            for (int e = 0; e < NE; e++) ss = fmaf(y[e].a, y[e].a, fmaf(y[e].b, y[e].b, ss));
            ss = warp_sum(ss);
            float inv = 1.0f / sqrtf((p.norm == 1 ? ss / (float)hd.n : ss) + p.eps);
            if (hd.kind == 0) inv *= p.q_scale;
#pragma unroll
            for (int e = 0; e < NE; e++) y[e] = {y[e].a * inv, y[e].b * inv};
        } else if (hd.kind == 0 && p.q_scale != 1.f) {
#pragma unroll
            for (int e = 0; e < NE; e++) y[e] = {y[e].a * p.q_scale, y[e].b * p.q_scale};
        }
    }
    if constexpr (CACHE) {
        T* dst = (T*)p.out + row * p.out_stride + hd.c0;
        if (hd.kind != 0) {
            const int heads = hd.kind == 1 ? p.k_heads : p.v_heads;
            dst = (T*)(hd.kind == 1 ? p.k_plane : p.v_plane) + ((page * heads + hd.at) * GB_PAGE + (pos % GB_PAGE)) * (int64_t)hd.n;
        }
#pragma unroll
        for (int e = 0; e < NE; e++) {
            const int i = 2 * (lane + 32 * e);
            store_pair<T>(dst + i, y[e], min(2, hd.n - i), vec);
        }
    } else {
        float* dst = (float*)p.out + row * p.out_stride + hd.c0;
#pragma unroll
        for (int e = 0; e < NE; e++) {
            const int i = 2 * (lane + 32 * e);
            store_pair<float>(dst + i, y[e], min(2, hd.n - i), vec);
        }
    }
}

// one row of one head with any number of taps: what the portion does not hold comes from the state
template <typename T, int NE>
__device__ __forceinline__ void convolve_row(const ShortConvParams& p, const Head& hd, int64_t row, int local, int slot, Pair (&y)[NE], int lane, bool vec) {
    const bool move = p.taps > 1 && p.max_q_len == 1;
    const T* base = (const T*)p.src + hd.c0;
    float* st = p.state ? p.state + (int64_t)slot * p.state_slot_stride + hd.c0 : nullptr;
#pragma unroll
    for (int e = 0; e < NE; e++) {
        const int c = 2 * (lane + 32 * e), m = min(2, hd.n - c);
        Pair bias = {0.f, 0.f};
        if (p.bias) bias = load_pair<float>(p.bias + hd.c0 + c, m, false);
        Pair own = load_pair<T>(base + row * p.row_stride + c, m, vec);
        own = {own.a + bias.a, own.b + bias.b};
        y[e] = {0.f, 0.f};
#pragma unroll 4
        for (int j = 0; j + 1 < p.taps; j++) {
            const int back = p.taps - 1 - j;
            Pair u;
            if (back <= local) {
                u = load_pair<T>(base + (row - back) * p.row_stride + c, m, vec);
                u = {u.a + bias.a, u.b + bias.b};
            } else {
                u = load_pair<float>(st + (int64_t)(p.taps - 1 + local - back) * p.channels + c, m, false);
            }
            const Pair w = load_pair<float>(p.conv_w + (int64_t)j * p.channels + hd.c0 + c, m, false);
            y[e] = {fmaf(w.a, u.a, y[e].a), fmaf(w.b, u.b, y[e].b)};
            if (move && j > 0) store_pair<float>(st + (int64_t)(j - 1) * p.channels + c, u, m, false);
        }
        if (move) store_pair<float>(st + (int64_t)(p.taps - 2) * p.channels + c, own, m, false);
        Pair w = {1.f, 1.f};
        if (p.conv_w) w = load_pair<float>(p.conv_w + (int64_t)(p.taps - 1) * p.channels + hd.c0 + c, m, false);
        y[e] = {fmaf(w.a, own.a, y[e].a), fmaf(w.b, own.b, y[e].b)};
    }
}

// Prompts of few taps whose heads take two-channel accesses: a warp's ROWS rows through a window of registers, every load issued
// ahead of the arithmetic (lanes beyond a narrower head repeat its last two channels and store nothing).  Rows whose taps all lie in their own portion, nearly
// all of them, take straight code; a warp that holds a portion's first rows goes row by row.
template <typename T, int ROWS, int TAPS, int NE, bool CACHE>
__global__ void __launch_bounds__(32 * WARPS) short_conv_window_kernel(ShortConvParams p) {
    pdl_wait();
    pdl_trigger();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int hh = blockIdx.y * WARPS + warp;
    if (hh >= p.q_heads + p.k_heads + p.v_heads) return;
    const Head hd = head_of(p, hh);
    const int64_t r0 = (int64_t)blockIdx.x * ROWS;
    const int n = p.rows - r0 < ROWS ? (int)(p.rows - r0) : ROWS;
    const T* base = (const T*)p.src + hd.c0;
    int at[NE];
#pragma unroll
    for (int e = 0; e < NE; e++) at[e] = min(2 * (lane + 32 * e), hd.n - 2);
    Pair x[ROWS + TAPS - 1][NE];
#pragma unroll
    for (int i = 0; i < ROWS + TAPS - 1; i++) {
        int64_t r = r0 + i - (TAPS - 1);
        r = r < 0 ? 0 : (r < p.rows ? r : p.rows - 1);      // rows outside are not used
#pragma unroll
        for (int e = 0; e < NE; e++) x[i][e] = load_two<T>(base + r * p.row_stride + at[e]);
    }
    const int seq0 = p.row_seq[r0];
    const bool plain = p.row_seq[r0 + n - 1] == seq0 && r0 - p.seq_q_start[seq0] >= TAPS - 1;
    if (!plain) {
        for (int i = 0; i < n; i++) {
            const int64_t row = r0 + i;
            const int seq = p.row_seq[row];
            int slot = p.seq_slot[seq];
            if (!gb_check(slot, p.max_slots, GB_CHECK_SLOT)) slot = 0;
            Pair y[NE];
            convolve_row<T, NE>(p, hd, row, (int)(row - p.seq_q_start[seq]), slot, y, lane, true);
            const int pos = CACHE || p.rot > 0 ? p.row_pos[row] : 0;
            finish_head<T, NE, CACHE, false>(p, hd, row, pos, CACHE && hd.kind != 0 ? page_at(p, slot, pos) : 0, y, nullptr, lane, true);
        }
        return;
    }
    Pair w[TAPS][NE];
#pragma unroll
    for (int e = 0; e < NE; e++) {
#pragma unroll
        for (int j = 0; j < TAPS; j++) {
            w[j][e] = {1.f, 1.f};
            if (p.conv_w) w[j][e] = load_two<float>(p.conv_w + (int64_t)j * p.channels + hd.c0 + at[e]);
            if (2 * (lane + 32 * e) >= hd.n) w[j][e] = {0.f, 0.f};      // a lane beyond the head has zeros
        }
        if (p.bias) {
            const Pair bias = load_two<float>(p.bias + hd.c0 + at[e]);
#pragma unroll
            for (int i = 0; i < ROWS + TAPS - 1; i++) x[i][e] = {x[i][e].a + bias.a, x[i][e].b + bias.b};
        }
    }
    const int pos0 = CACHE || p.rot > 0 ? p.row_pos[r0] : 0;      // rows of a sequence are consecutive positions
    int64_t first_page = 0, last_page = 0;                        // eight rows lie in two pages at most
    if (CACHE && hd.kind != 0) {
        const int slot = p.seq_slot[seq0];
        first_page = page_at(p, slot, pos0);
        last_page = page_at(p, slot, pos0 + n - 1);
    }
#pragma unroll
    for (int i = 0; i < ROWS; i++) {
        if (i >= n) break;
        Pair y[NE];
#pragma unroll
        for (int e = 0; e < NE; e++) {
            y[e] = {0.f, 0.f};
#pragma unroll
            for (int j = 0; j < TAPS; j++) y[e] = {fmaf(w[j][e].a, x[i + j][e].a, y[e].a), fmaf(w[j][e].b, x[i + j][e].b, y[e].b)};
        }
        finish_head<T, NE, CACHE, false>(p, hd, r0 + i, pos0 + i, (pos0 + i) / GB_PAGE == pos0 / GB_PAGE ? first_page : last_page, y, nullptr, lane, true);
    }
}

// one row a warp, any number of taps; for single tokens it also moves the state on
template <typename T, int NE, bool CACHE>
__global__ void __launch_bounds__(32 * WARPS) short_conv_row_kernel(ShortConvParams p) {
    pdl_wait();
    pdl_trigger();
    __shared__ float sh[WARPS][MAX_HEAD];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int hh = blockIdx.y * WARPS + warp;
    if (hh >= p.q_heads + p.k_heads + p.v_heads) return;
    const Head hd = head_of(p, hh);
    const int64_t row = blockIdx.x;
    const int seq = p.row_seq[row];
    int slot = p.seq_slot[seq];
    if (!gb_check(slot, p.max_slots, GB_CHECK_SLOT)) slot = 0;
    Pair y[NE];
    convolve_row<T, NE>(p, hd, row, (int)(row - p.seq_q_start[seq]), slot, y, lane, p.vec);
    const int pos = CACHE || p.rot > 0 ? p.row_pos[row] : 0;
    finish_head<T, NE, CACHE, true>(p, hd, row, pos, CACHE && hd.kind != 0 ? page_at(p, slot, pos) : 0, y, sh[warp], lane, p.vec);
}

// the last taps - 1 rows u of every sequence's portion into its state; a portion shorter than that pushes the older rows on
template <typename T>
__global__ void short_conv_state_kernel(ShortConvParams p) {
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    const int seq = blockIdx.y;
    if (c >= p.channels) return;
    const int len = p.seq_q_len[seq];
    if (len <= 0) return;
    const int64_t start = p.seq_q_start[seq];
    int slot = p.seq_slot[seq];
    if (!gb_check(slot, p.max_slots, GB_CHECK_SLOT)) slot = 0;
    float* st = p.state + (int64_t)slot * p.state_slot_stride;
    const T* base = (const T*)p.src;
    const float bias = p.bias ? p.bias[c] : 0.f;
    for (int s = 0; s + 1 < p.taps; s++) {      // ascending: a place is read before it is written
        const int at = len - (p.taps - 1) + s;
        st[(int64_t)s * p.channels + c] = at >= 0 ? to_f32<T>(base[(start + at) * p.row_stride + c]) + bias : st[(int64_t)(s + len) * p.channels + c];
    }
}

constexpr int WINDOW_ROWS = 8;
constexpr int WINDOW_MIN_ROWS = 96;    // packed rows from which a warp takes eight of them

template <typename T, int NE, bool CACHE>
int launch_ne(const ShortConvParams& p, cudaStream_t stream) {
    const int heads = p.q_heads + p.k_heads + p.v_heads;
    const int hy = ceil_div(heads, WARPS);
    if (hy > 65535) GB_REFUSE("short_conv: %d heads exceed one launch", heads);
    if (p.max_q_len != 1 && p.taps <= 4 && p.rows >= WINDOW_MIN_ROWS && p.vec && (p.rot == 0 || p.pairs)) {
        const dim3 grid(ceil_div(p.rows, WINDOW_ROWS), hy), block(32 * WARPS);
        switch (p.taps) {
            case 1: launch_pdl(short_conv_window_kernel<T, WINDOW_ROWS, 1, NE, CACHE>, grid, block, 0, stream, p); break;
            case 2: launch_pdl(short_conv_window_kernel<T, WINDOW_ROWS, 2, NE, CACHE>, grid, block, 0, stream, p); break;
            case 3: launch_pdl(short_conv_window_kernel<T, WINDOW_ROWS, 3, NE, CACHE>, grid, block, 0, stream, p); break;
            default: launch_pdl(short_conv_window_kernel<T, WINDOW_ROWS, 4, NE, CACHE>, grid, block, 0, stream, p); break;
        }
    } else {
        launch_pdl(short_conv_row_kernel<T, NE, CACHE>, dim3(p.rows, hy), dim3(32 * WARPS), 0, stream, p);
    }
    GB_CHECK_LAUNCH("short_conv");
    if (p.taps > 1 && p.max_q_len != 1) {
        short_conv_state_kernel<T><<<dim3(ceil_div(p.channels, 128), p.nseq), 128, 0, stream>>>(p);
        GB_CHECK_LAUNCH("short_conv_state");
    }
    return 0;
}

template <typename T>
int launch(ShortConvParams p, cudaStream_t stream) {
    const uintptr_t pair = 2 * sizeof(T) - 1;
    p.vec = !(p.d & 1) && !(p.dv & 1) && !(p.row_stride & 1) && !((uintptr_t)p.src & pair) && !(p.out_stride & 1) &&
            !((uintptr_t)p.out & (p.to_cache ? pair : 7)) && !(((uintptr_t)p.k_plane | (uintptr_t)p.v_plane) & pair);
    p.vec = p.vec && !(((uintptr_t)p.conv_w | (uintptr_t)p.bias) & 7);
    const int most = p.d > p.dv ? p.d : p.dv;
    if (most <= 64) return p.to_cache ? launch_ne<T, 1, true>(p, stream) : launch_ne<T, 1, false>(p, stream);
    if (most <= 128) return p.to_cache ? launch_ne<T, 2, true>(p, stream) : launch_ne<T, 2, false>(p, stream);
    return p.to_cache ? launch_ne<T, 4, true>(p, stream) : launch_ne<T, 4, false>(p, stream);
}

}  // namespace

GB_API int gb_short_conv(const ShortConvParams* pp, int dtype, cudaStream_t stream) {
    ShortConvParams p = *pp;
    if (p.rows <= 0 || p.nseq <= 0) return 0;
    if (p.q_heads <= 0 || p.k_heads <= 0 || p.v_heads <= 0 || p.d <= 0 || p.d > MAX_HEAD || p.dv <= 0 || p.dv > MAX_HEAD)
        GB_REFUSE("short_conv: %d + %d heads of %d and %d of %d channels; a head has 1 to %d", p.q_heads, p.k_heads, p.d, p.v_heads, p.dv, MAX_HEAD);
    if (p.channels != (p.q_heads + p.k_heads) * p.d + p.v_heads * p.dv) GB_REFUSE("short_conv: %d channels do not fit the heads", p.channels);
    if (p.taps <= 0 || p.taps > MAX_TAPS) GB_REFUSE("short_conv: %d taps; 1 to %d", p.taps, MAX_TAPS);
    if (p.taps > 1 && (!p.conv_w || !p.state || p.state_slot_stride < (int64_t)(p.taps - 1) * p.channels))
        GB_REFUSE("short_conv: no weights for %d taps, or a state without room for %d rows of %d", p.taps, p.taps - 1, p.channels);
    if (p.rot < 0 || p.rot > p.d || (p.rot & 1) || (p.rot > 0 && (!p.cos_t || !p.sin_t))) GB_REFUSE("short_conv: %d rotated channels of %d", p.rot, p.d);
    if (!p.src || !p.out || (p.to_cache && (!p.k_plane || !p.v_plane || !p.block_table))) GB_REFUSE("short_conv: a tensor is missing");
    if (p.nseq > 65535) GB_REFUSE("short_conv: %d sequences exceed one launch", p.nseq);
    if (dtype == GB_F32) return launch<float>(p, stream);
    if (dtype == GB_BF16) return launch<__nv_bfloat16>(p, stream);
    GB_REFUSE("short_conv: unknown dtype %d", dtype);
}

// the checked build's record of the first index this file's kernels found out of bounds
GB_CHECK_READER(gb_checked_status_short_conv)
