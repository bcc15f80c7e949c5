// The gated delta rule: a matrix state per (sequence, head), d key channels x dv value channels, fp32, with a decay g (one
// number a head, or one a key channel) and a write strength b; for every token, in this order,
//
//     S <- diag(g) S,   u = b (v - S^T k),   S <- S + k u^T,   o = S^T q.
//
// q and k are unit vectors (q scaled) that several heads may share, made by short_conv together with v, all fp32.
// g = exp(-exp(A_h) softplus(z + bias)) and b = sigmoid(z_b) are formed here from fp32 pre-activations.
//
// Prompts.  Tokens are taken four at a time (counted from the portion's start).  With S the state ahead of the four, G_t the
// product of the decays up to token t and G_ts that of the decays behind s up to t,
//
//     u_t = b_t (v_t - S^T (G_t k_t) - sum_{s<t} A_ts u_s),     A_ts = k_t . (G_ts k_s)
//     o_t =            S^T (G_t q_t) + sum_{s<=t} B_ts u_s,     B_ts = q_t . (G_ts k_s)
//     S  <- G_4 S + sum_s (G_4s k_s) u_s^T
//
// which is the same recurrence: every factor is a product of decays (nothing is divided), and the sums over the key channels
// that a token's u waits for are taken once for four tokens instead of once a token.  A preparation kernel leaves g, b, A and B.
//
// Columns of S are independent of one another, so the work is spread over (sequence, head, block of value columns).  A warp
// owns CW columns, its 32 lanes the key channels (RC each); a thread keeps RC x CW state elements in registers across the
// step.  The four tokens' partial sums a lane are added over the lanes by halving the values and the lanes; the 4 x CW finished
// v - S^T (G k) then pass through shared memory to all lanes, and every lane solves the four small triangular systems itself.  A prompt of one sequence leaves
// every scheduler one such warp, so nothing but this chain is on it: four further warps of the CTA fetch the tokens' rows, form
// the products of decays and lay them out in shared memory a tile of eight tokens ahead, and add the outputs' remaining terms a
// tile behind.
//
// Single tokens: reading and writing the state once, 16 bytes a thread and load, everything else of the token formed in the
// same kernel.
#include "api.h"
#include "common.cuh"

#include <math.h>

namespace {

constexpr int TT = 8;        // tokens staged at a time
constexpr int C = 4;         // tokens taken together
constexpr int THREADS = 128;
constexpr int WARPS = THREADS / 32;

__device__ __forceinline__ float softplus_f(float z) { return z > 20.f ? z : log1pf(expf(z)); }
__device__ __forceinline__ float decay_factor(float z, float rate) { return expf(-rate * softplus_f(z)); }   // rate = exp(A_h)
__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }

// ------------------------------------------------------------------------------------------
// N values a lane added over the lanes: N / 2 exchanged with the lane O away, and so on; lane l is left with the value of
// number l * N / 32
template <int N, int O>
__device__ __forceinline__ float add_over_lanes(float* a, int lane) {
    if constexpr (O == 0) {
        return a[0];
    } else if constexpr (N == 1) {
        a[0] += __shfl_xor_sync(0xffffffffu, a[0], O);
        return add_over_lanes<1, O / 2>(a, lane);
    } else {
        const bool up = lane & O;
#pragma unroll
        for (int j = 0; j < N / 2; j++) {
            const float keep = up ? a[j + N / 2] : a[j], give = up ? a[j] : a[j + N / 2];
            a[j] = keep + __shfl_xor_sync(0xffffffffu, give, O);
        }
        return add_over_lanes<N / 2, O / 2>(a, lane);
    }
}

// ------------------------------------------------------------------------------------------
// preparation of a prompt's tokens, one warp per (four tokens of a sequence, head): the decay factors, and for token t
// (A_t0, A_t1, A_t2, b, B_t0 .. B_t3), with zeros where the other token is not earlier (for B: not later).
template <bool CHANNEL>
__global__ void __launch_bounds__(128) gated_delta_prep_kernel(GatedDeltaParams p) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int seq = blockIdx.z, h = blockIdx.y * 4 + warp, first = blockIdx.x * C;
    const int q_len = p.seq_q_len[seq];
    if (h >= p.heads || first >= q_len) return;
    const int n = q_len - first < C ? q_len - first : C;       // tokens that are there
    const int64_t row0 = p.seq_q_start[seq] + first;
    const int d = p.d, H = p.heads, kh = h / (H / p.kv_heads);
    const float rate = expf(p.a_log[h]);
    float g_head[C];
    if (!CHANNEL) {
#pragma unroll
        for (int t = 0; t < C; t++) {
            g_head[t] = t < n ? decay_factor(p.decay_in[(row0 + t) * p.decay_stride + h] + p.dt_bias[h], rate) : 1.f;
            if (lane == 0 && t < n) p.decay_out[(row0 + t) * H + h] = g_head[t];
        }
    }
    // sums[t * 4 + s], s < t: A_ts; sums[16 + t * 4 + s], s <= t: B_ts; the rest stays zero and costs nothing but its exchange
    float sums[32];
#pragma unroll
    for (int i = 0; i < 32; i++) sums[i] = 0.f;
    for (int c = lane; c < d; c += 32) {
        float q[C], k[C], g[C];
#pragma unroll
        for (int t = 0; t < C; t++) {
            const int64_t row = row0 + (t < n ? t : n - 1);
            const float* r = p.rows_in + row * p.row_stride + kh * d + c;
            q[t] = r[p.q_off];
            k[t] = t < n ? r[p.k_off] : 0.f;
            if (CHANNEL) {
                g[t] = decay_factor(p.decay_in[row * p.decay_stride + h * d + c] + p.dt_bias[h * d + c], rate);
                if (t < n) p.decay_out[(row * H + h) * d + c] = g[t];
            } else {
                g[t] = g_head[t];
            }
        }
#pragma unroll
        for (int t = 0; t < C; t++) {
            float between = 1.f;               // the decays behind s up to t
#pragma unroll
            for (int s = t; s >= 0; s--) {
                const float ks = between * k[s];
                if (s < t) sums[t * 4 + s] = fmaf(k[t], ks, sums[t * 4 + s]);
                sums[16 + t * 4 + s] = fmaf(q[t], ks, sums[16 + t * 4 + s]);
                between *= g[s];
            }
        }
    }
    const float total = add_over_lanes<32, 16>(sums, lane);    // lane l: sum number l
    const int t = (lane & 15) >> 2, s = lane & 3;
    if (t < n) {
        float v = total;
        int place = lane < 16 ? s : 4 + s;
        if (lane < 16 && s == 3) v = sigmoid_f(p.beta_in[(row0 + t) * p.beta_stride + h]);
        p.coef[((row0 + t) * H + h) * 8 + place] = v;
    }
}

// The same for 4 N values in an order of the lane's own over the first two steps: the values of the upper half are the ones the
// lane O away keeps, so nothing is chosen there.
template <int N>
__device__ __forceinline__ float fold_lanes(float* a, int lane) {
#pragma unroll
    for (int j = 0; j < 2 * N; j++) a[j] += __shfl_xor_sync(0xffffffffu, a[j + 2 * N], 16);
#pragma unroll
    for (int j = 0; j < N; j++) a[j] += __shfl_xor_sync(0xffffffffu, a[j + N], 8);
    return add_over_lanes<N, 4>(a, lane);
}

template <int V>
__device__ __forceinline__ void lds(const float* p, float* v) {
    if constexpr (V == 4) {
        const float4 t = *reinterpret_cast<const float4*>(p);
        v[0] = t.x, v[1] = t.y, v[2] = t.z, v[3] = t.w;
    } else if constexpr (V == 2) {
        const float2 t = *reinterpret_cast<const float2*>(p);
        v[0] = t.x, v[1] = t.y;
    } else {
        v[0] = *p;
    }
}
template <int V>
__device__ __forceinline__ void sts(float* p, const float* v) {
    if constexpr (V == 4)
        *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    else if constexpr (V == 2)
        *reinterpret_cast<float2*>(p) = make_float2(v[0], v[1]);
    else
        *p = v[0];
}

// RC: key channels a lane (32 RC >= d), CW: value columns a warp
template <int RC, int CW>
struct ScanShared {
    static constexpr int D = 32 * RC, COLS = WARPS * CW;
    struct __align__(16) Tile {
        float gk[TT][D], gq[TT][D], kp[TT][D], gc[TT / C][D];
        float v[TT][COLS];
    } tile[2];
    float u[2][TT][COLS], p2[2][TT][COLS];
    float coef[4][TT][8];
    float left[WARPS][2][C][CW];      // a warp's finished v - S^T (G k), for its lanes
    float st[D][COLS + 1];
};

template <int RC, int CW, bool CHANNEL>
__global__ void __launch_bounds__(2 * THREADS) gated_delta_scan_kernel(GatedDeltaParams p) {
    constexpr int D = 32 * RC, COLS = WARPS * CW;
    constexpr int V = RC < 4 ? RC : 4;           // neighbouring channels of a lane: lane l has l V .. l V + V - 1 of every 32 V
    constexpr int NV = C * CW;                   // sums of four tokens, token by token
    constexpr int PER = 32 / NV;                 // lanes that are left with the same sum
    constexpr int ITEMS = (TT / C * D + THREADS - 1) / THREADS;   // (four tokens, channel) pieces a staging thread makes
    extern __shared__ __align__(16) unsigned char smem_raw[];
    ScanShared<RC, CW>& sm = *reinterpret_cast<ScanShared<RC, CW>*>(smem_raw);

    const int tid = threadIdx.x & (THREADS - 1), warp = tid >> 5, lane = tid & 31;
    const bool stages = threadIdx.x >= THREADS;  // the second half of the CTA feeds the first
    const int d = p.d, dv = p.dv, H = p.heads;
    const int h = blockIdx.y, seq = blockIdx.z, kh = h / (H / p.kv_heads);
    const int j0 = blockIdx.x * COLS;
    const int q_len = p.seq_q_len[seq], q_start = p.seq_q_start[seq];
    int slot = p.seq_slot[seq];
    if (!gb_check(slot, p.max_slots, GB_CHECK_SLOT)) slot = 0;
    float* S = p.state + (int64_t)slot * p.slot_stride + (int64_t)h * p.head_stride;
    auto channel = [&](int i) { return i / V * (32 * V) + lane * V + i % V; };
    // A thread's slot j of the four tokens' sums is token j ^ mine_t; adding over the lanes (fold_lanes) leaves each lane the sum of
    // token mine_t and column mine_c
    const int mine_t = lane >> 3, mine_c = (lane / PER) % CW;
    const int tiles = (q_len + TT - 1) / TT;

    for (int idx = threadIdx.x; idx < D * COLS; idx += 2 * THREADS) {
        const int c = idx / COLS, jj = idx % COLS;
        sm.st[c][jj] = (c < d && j0 + jj < dv) ? S[(int64_t)c * dv + j0 + jj] : 0.f;
    }

    // ---- staging: a tile's rows are fetched into registers a tile ahead of their place in shared memory; every load is
    // unconditional (indices clamped); what is not there changes nothing (decay 1, key 0, strength 0)
    float rq[ITEMS][C], rk[ITEMS][C], rg[ITEMS][C], rv = 0.f, rcoef = 0.f;
    const int stride = (int)p.row_stride;
    auto fetch = [&](int tile) {
        const int t0 = tile * TT, nt = q_len - t0 < TT ? q_len - t0 : TT;
        const int row0 = q_start + t0;           // products of two 32-bit numbers, one instruction an address
#pragma unroll
        for (int e = 0; e < ITEMS; e++) {
            const int idx = tid + e * THREADS;
            int ch = idx / D, c = idx % D;
            ch = ch < TT / C ? ch : TT / C - 1;
            c = c < d ? c : d - 1;
#pragma unroll
            for (int j = 0; j < C; j++) {
                int t = ch * C + j;
                t = t < nt ? t : nt - 1;
                const float* r = p.rows_in + (int64_t)(row0 + t) * stride + kh * d + c;
                rq[e][j] = r[p.q_off];
                rk[e][j] = r[p.k_off];
                rg[e][j] = CHANNEL ? p.decay_out[(int64_t)((row0 + t) * H + h) * d + c] : p.decay_out[(row0 + t) * H + h];
            }
        }
        if (tid < TT * COLS) {
            int t = tid / COLS, jj = j0 + tid % COLS;
            t = t < nt ? t : nt - 1;
            jj = jj < dv ? jj : dv - 1;
            rv = p.rows_in[(int64_t)(row0 + t) * stride + p.v_off + h * dv + jj];
        }
        if (tid < TT * 8) {
            int t = tid >> 3;
            t = t < nt ? t : nt - 1;
            rcoef = p.coef[(int64_t)((row0 + t) * H + h) * 8 + (tid & 7)];
        }
    };
    auto place = [&](int tile) {
        const int t0 = tile * TT, nt = q_len - t0 < TT ? q_len - t0 : TT;
        auto& to = sm.tile[tile & 1];
#pragma unroll
        for (int e = 0; e < ITEMS; e++) {
            const int idx = tid + e * THREADS;
            const int ch = idx / D, c = idx % D;
            if (ch >= TT / C) continue;
            float up = 1.f;
#pragma unroll
            for (int j = 0; j < C; j++) {
                const int t = ch * C + j;
                const bool there = t < nt && c < d;
                rg[e][j] = there ? rg[e][j] : 1.f;
                rk[e][j] = there ? rk[e][j] : 0.f;
                up *= rg[e][j];
                to.gk[t][c] = rk[e][j] * up;
                to.gq[t][c] = there ? rq[e][j] * up : 0.f;
            }
            to.gc[ch][c] = up;
            float down = 1.f;
#pragma unroll
            for (int j = C - 1; j >= 0; j--) {
                to.kp[ch * C + j][c] = rk[e][j] * down;
                down *= rg[e][j];
            }
        }
        if (tid < TT * COLS) {
            const int t = tid / COLS, jj = tid % COLS;
            to.v[t][jj] = (t < nt && j0 + jj < dv) ? rv : 0.f;
        }
        if (tid < TT * 8) sm.coef[tile & 3][tid >> 3][tid & 7] = (tid >> 3) < nt ? rcoef : 0.f;
    };
    auto leave = [&](int tile) {
        const int t0 = tile * TT, nt = q_len - t0 < TT ? q_len - t0 : TT;
        for (int idx = tid; idx < nt * COLS; idx += THREADS) {
            const int t = idx / COLS, jj = idx % COLS;
            float o = sm.p2[tile & 1][t][jj];
#pragma unroll
            for (int s = 0; s < C; s++) o = fmaf(sm.coef[tile & 3][t][4 + s], sm.u[tile & 1][t / C * C + s][jj], o);     // B is zero for later tokens
            if (j0 + jj < dv) p.out[(int64_t)(q_start + t0 + t) * p.out_stride + h * dv + j0 + jj] = o;
        }
    };
    if (stages && tiles > 0) {
        fetch(0);
        place(0);
        if (tiles > 1) fetch(1);
    }
    __syncthreads();
    float st[RC][CW];
    if (!stages) {
#pragma unroll
        for (int i = 0; i < RC; i++)
#pragma unroll
            for (int c = 0; c < CW; c++) st[i][c] = sm.st[channel(i)][warp * CW + c];
    }
    for (int tile = 0; tile < tiles; tile++) {
        if (stages) {
            if (tile + 1 < tiles) place(tile + 1);
            if (tile + 2 < tiles) fetch(tile + 2);
            if (tile > 0) leave(tile - 1);
        } else {
            const auto& in = sm.tile[tile & 1];
#pragma unroll
            for (int ch = 0; ch < TT / C; ch++) {
                float a1[NV], a2[NV];
#pragma unroll
                for (int j = 0; j < C; j++) {
#pragma unroll
                    for (int c = 0; c < CW; c++) a1[j * CW + c] = a2[j * CW + c] = 0.f;
#pragma unroll
                    for (int i = 0; i < RC; i += V) {
                        float k4[V], q4[V];
                        lds<V>(&in.gk[ch * C + (j ^ mine_t)][channel(i)], k4);
                        lds<V>(&in.gq[ch * C + (j ^ mine_t)][channel(i)], q4);
#pragma unroll
                        for (int w = 0; w < V; w++)
#pragma unroll
                            for (int c = 0; c < CW; c++) {
                                a1[j * CW + c] = fmaf(k4[w], st[i + w][c], a1[j * CW + c]);
                                a2[j * CW + c] = fmaf(q4[w], st[i + w][c], a2[j * CW + c]);
                            }
                    }
                }
                // what a token writes but for its four's earlier writes: the lane that has the sum takes it off the value
                const float t1 = in.v[ch * C + mine_t][warp * CW + mine_c] - fold_lanes<CW>(a1, lane);
                if (lane % PER == 0) sm.left[warp][ch & 1][mine_t][mine_c] = t1;
                __syncwarp();
                float u[C][CW];
#pragma unroll
                for (int j = 0; j < C; j++) lds<CW>(sm.left[warp][ch & 1][j], u[j]);
                const float t2 = fold_lanes<CW>(a2, lane);
                if (lane % PER == 0) sm.p2[tile & 1][ch * C + mine_t][warp * CW + mine_c] = t2;
#pragma unroll
                for (int j = 0; j < C; j++) {
                    const float4 a4 = *reinterpret_cast<const float4*>(&sm.coef[tile & 3][ch * C + j][0]);
                    const float aa[C - 1] = {a4.x, a4.y, a4.z};
#pragma unroll
                    for (int c = 0; c < CW; c++) {
                        float t = u[j][c];
#pragma unroll
                        for (int s = 0; s < j; s++) t = fmaf(-aa[s], u[s][c], t);
                        u[j][c] = a4.w * t;
                    }
                }
#pragma unroll
                for (int i = 0; i < RC; i += V) {
                    float g4[V];
                    lds<V>(&in.gc[ch][channel(i)], g4);
#pragma unroll
                    for (int w = 0; w < V; w++)
#pragma unroll
                        for (int c = 0; c < CW; c++) st[i + w][c] *= g4[w];
#pragma unroll
                    for (int j = 0; j < C; j++) {
                        float k4[V];
                        lds<V>(&in.kp[ch * C + j][channel(i)], k4);
#pragma unroll
                        for (int w = 0; w < V; w++)
#pragma unroll
                            for (int c = 0; c < CW; c++) st[i + w][c] = fmaf(k4[w], u[j][c], st[i + w][c]);
                    }
                }
                if (lane == 0) {
#pragma unroll
                    for (int j = 0; j < C; j++) sts<CW>(&sm.u[tile & 1][ch * C + j][warp * CW], u[j]);
                }
            }
        }
        __syncthreads();
    }
    if (stages) {
        if (tiles > 0) leave(tiles - 1);
    } else {
#pragma unroll
        for (int i = 0; i < RC; i++)
#pragma unroll
            for (int c = 0; c < CW; c++) sm.st[channel(i)][warp * CW + c] = st[i][c];
    }
    __syncthreads();
    for (int idx = threadIdx.x; idx < D * COLS; idx += 2 * THREADS) {
        const int c = idx / COLS, jj = idx % COLS;
        if (c < d && j0 + jj < dv) S[(int64_t)c * dv + j0 + jj] = sm.st[c][jj];
    }
}

// ------------------------------------------------------------------------------------------
// One token for every sequence.  A CTA owns 8 V columns of one head's S; thread (group of 16, 8 places of V columns) takes the
// channels group, group + 16, ..., keeps them in registers from load to store; sums over the groups by shuffles and then over
// the four warps in shared memory.
template <int V, int R, bool CHANNEL>
__global__ void __launch_bounds__(THREADS) gated_delta_step_kernel(GatedDeltaParams p) {
    constexpr int GROUPS = THREADS / 8, COLS = 8 * V, D = GROUPS * R;
    __shared__ float gk_s[D], gq_s[D], k_s[D], g_s[D];
    __shared__ __align__(16) float red[2][WARPS][COLS];
    __shared__ float part[WARPS];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int g = tid >> 3, jt = tid & 7;
    const int d = p.d, dv = p.dv, H = p.heads;
    const int h = blockIdx.y, seq = blockIdx.z, kh = h / (H / p.kv_heads);
    const int j = blockIdx.x * COLS + jt * V;
    int slot = p.seq_slot[seq];
    if (!gb_check(slot, p.max_slots, GB_CHECK_SLOT)) slot = 0;
    float* S = p.state + (int64_t)slot * p.slot_stride + (int64_t)h * p.head_stride;
    const bool mine = j < dv;                  // V divides dv where V is 4
    float st[R][V];
#pragma unroll
    for (int i = 0; i < R; i++) {
        const int c = g + GROUPS * i;
#pragma unroll
        for (int u = 0; u < V; u++) st[i][u] = 0.f;
        if (mine && c < d) lds<V>(S + (int64_t)c * dv + j, st[i]);
    }
    pdl_wait();                                // the state is this kernel's own; the rows come from the kernels ahead
    pdl_trigger();
    const int64_t row = p.seq_q_start[seq];
    const float* in = p.rows_in + row * p.row_stride;
    const float rate = expf(p.a_log[h]);
    const float beta = sigmoid_f(p.beta_in[row * p.beta_stride + h]);
    float g_head = 1.f;
    if (!CHANNEL) g_head = decay_factor(p.decay_in[row * p.decay_stride + h] + p.dt_bias[h], rate);
    float kq = 0.f;
    for (int c = tid; c < D; c += THREADS) {
        float k = 0.f, q = 0.f, gg = 1.f;
        if (c < d) {
            k = in[p.k_off + kh * d + c];
            q = in[p.q_off + kh * d + c];
            gg = CHANNEL ? decay_factor(p.decay_in[row * p.decay_stride + h * d + c] + p.dt_bias[h * d + c], rate) : g_head;
        }
        gk_s[c] = gg * k, gq_s[c] = gg * q, k_s[c] = k, g_s[c] = gg;
        kq = fmaf(k, q, kq);
    }
    kq = warp_sum(kq);
    if (lane == 0) part[warp] = kq;
    __syncthreads();
    kq = (part[0] + part[1]) + (part[2] + part[3]);
    float p1[V], p2[V];
#pragma unroll
    for (int u = 0; u < V; u++) p1[u] = p2[u] = 0.f;
#pragma unroll
    for (int i = 0; i < R; i++) {
        const int c = g + GROUPS * i;
        const float k = gk_s[c], q = gq_s[c];
#pragma unroll
        for (int u = 0; u < V; u++) {
            p1[u] = fmaf(k, st[i][u], p1[u]);
            p2[u] = fmaf(q, st[i][u], p2[u]);
        }
    }
#pragma unroll
    for (int o = 8; o <= 16; o <<= 1)
#pragma unroll
        for (int u = 0; u < V; u++) {
            p1[u] += __shfl_xor_sync(0xffffffffu, p1[u], o);
            p2[u] += __shfl_xor_sync(0xffffffffu, p2[u], o);
        }
    if (lane < 8) {
        sts<V>(&red[0][warp][jt * V], p1);
        sts<V>(&red[1][warp][jt * V], p2);
    }
    __syncthreads();
    float uu[V], vj[V];
#pragma unroll
    for (int u = 0; u < V; u++) {
        p1[u] = p2[u] = 0.f;
        vj[u] = mine ? in[p.v_off + h * dv + j + u] : 0.f;
    }
#pragma unroll
    for (int w = 0; w < WARPS; w++) {
        float a[V], b[V];
        lds<V>(&red[0][w][jt * V], a);
        lds<V>(&red[1][w][jt * V], b);
#pragma unroll
        for (int u = 0; u < V; u++) p1[u] += a[u], p2[u] += b[u];
    }
#pragma unroll
    for (int u = 0; u < V; u++) uu[u] = beta * (vj[u] - p1[u]);
#pragma unroll
    for (int i = 0; i < R; i++) {
        const int c = g + GROUPS * i;
        const float gg = g_s[c], k = k_s[c];
#pragma unroll
        for (int u = 0; u < V; u++) st[i][u] = fmaf(gg, st[i][u], k * uu[u]);
        if (mine && c < d) sts<V>(S + (int64_t)c * dv + j, st[i]);
    }
    if (g == 0 && mine) {
#pragma unroll
        for (int u = 0; u < V; u++) p.out[row * p.out_stride + h * dv + j + u] = fmaf(kq, uu[u], p2[u]);
    }
}

template <int V, bool CHANNEL>
int launch_step(const GatedDeltaParams& p, cudaStream_t stream) {
    const dim3 grid(ceil_div(p.dv, 8 * V), p.heads, p.nseq), block(THREADS);
    if (p.d <= 64)
        launch_pdl(gated_delta_step_kernel<V, 4, CHANNEL>, grid, block, 0, stream, p);
    else if (p.d <= 128)
        launch_pdl(gated_delta_step_kernel<V, 8, CHANNEL>, grid, block, 0, stream, p);
    else
        launch_pdl(gated_delta_step_kernel<V, 16, CHANNEL>, grid, block, 0, stream, p);
    GB_CHECK_LAUNCH("gated_delta_step");
    return 0;
}

template <int RC, int CW, bool CHANNEL>
int launch_scan(const GatedDeltaParams& p, cudaStream_t stream) {
    constexpr int smem = (int)sizeof(ScanShared<RC, CW>);
    static bool configured = false;
    if (!configured && smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(gated_delta_scan_kernel<RC, CW, CHANNEL>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
        if (e != cudaSuccess) GB_REFUSE("gated_delta: cannot reserve %d bytes of shared memory: %s", smem, cudaGetErrorString(e));
        configured = true;
    }
    gated_delta_scan_kernel<RC, CW, CHANNEL><<<dim3(ceil_div(p.dv, WARPS * CW), p.heads, p.nseq), 2 * THREADS, smem, stream>>>(p);
    GB_CHECK_LAUNCH("gated_delta_scan");
    return 0;
}

template <bool CHANNEL>
int launch(const GatedDeltaParams& p, cudaStream_t stream) {
    if (p.heads > 65535 || p.nseq > 65535) GB_REFUSE("gated_delta: %d heads of %d sequences exceed one launch", p.heads, p.nseq);
    if (p.max_q_len == 1) {
        const bool vec = !(p.dv & 3) && !(p.head_stride & 3) && !(p.slot_stride & 3) && !((uintptr_t)p.state & 15);
        return vec ? launch_step<4, CHANNEL>(p, stream) : launch_step<1, CHANNEL>(p, stream);
    }
    if (!p.coef || !p.decay_out) GB_REFUSE("gated_delta: no room for the tokens' factors");
    gated_delta_prep_kernel<CHANNEL><<<dim3(ceil_div(p.max_q_len, C), ceil_div(p.heads, 4), p.nseq), 128, 0, stream>>>(p);
    GB_CHECK_LAUNCH("gated_delta_prep");
    // short heads and few (head, column block) pairs: two columns a warp leave more CTAs, and warps, to hide one another's chains
    const int rc = ceil_div(p.d, 32);
    const bool narrow = rc <= 2 && (int64_t)p.heads * p.nseq * ceil_div(p.dv, 16) < p.narrow_below;
    if (rc <= 1) return narrow ? launch_scan<1, 2, CHANNEL>(p, stream) : launch_scan<1, 4, CHANNEL>(p, stream);
    if (rc <= 2) return narrow ? launch_scan<2, 2, CHANNEL>(p, stream) : launch_scan<2, 4, CHANNEL>(p, stream);
    if (rc <= 4) return launch_scan<4, 4, CHANNEL>(p, stream);
    return launch_scan<8, 4, CHANNEL>(p, stream);
}

}  // namespace

GB_API int gb_gated_delta(const GatedDeltaParams* pp, cudaStream_t stream) {
    GatedDeltaParams p = *pp;
    if (p.nseq <= 0 || p.rows <= 0) return 0;
    if (p.heads <= 0 || p.kv_heads <= 0 || p.heads % p.kv_heads || p.d <= 0 || p.d > 256 || p.dv <= 0)
        GB_REFUSE("gated_delta: %d heads over %d of %d key and %d value channels; at most 256 key channels", p.heads, p.kv_heads, p.d, p.dv);
    if (!p.rows_in || !p.decay_in || !p.beta_in || !p.a_log || !p.dt_bias || !p.state || !p.out) GB_REFUSE("gated_delta: a tensor is missing");
    if (p.head_stride < (int64_t)p.d * p.dv || p.slot_stride < p.head_stride * p.heads) GB_REFUSE("gated_delta: the state is too small for its heads");
    if (p.row_stride > 0x7fffffff || (int64_t)p.rows * p.heads > 0x7fffffff) GB_REFUSE("gated_delta: %d rows of %d heads are too many for one launch", p.rows, p.heads);
    if (p.per_channel) return launch<true>(p, stream);
    return launch<false>(p, stream);
}

// the checked build's record of the first index this file's kernels found out of bounds
GB_CHECK_READER(gb_checked_status_gated_delta)
