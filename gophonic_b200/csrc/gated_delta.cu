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
// step.  The four tokens' 2 x 4 x CW partial sums a lane are added over the lanes by halving the values and the lanes, five
// steps; the 4 x CW finished S^T (G k) are then broadcast, every lane solves the four small triangular systems itself, and
// the outputs' remaining terms are added when a tile of eight tokens is written out, off the chain.
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
// preparation of a prompt's tokens, one warp per (row, head): the decay factors, and (A_t0, A_t1, A_t2, b, B_t0 .. B_t3), with
// the indices counting the tokens of the row's four and zeros where the other token is not earlier (for B: not later).
template <bool CHANNEL>
__global__ void __launch_bounds__(128) gated_delta_prep_kernel(GatedDeltaParams p) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int64_t row = blockIdx.x;
    const int h = blockIdx.y * 4 + warp;
    if (h >= p.heads) return;
    const int d = p.d, kh = h / (p.heads / p.kv_heads);
    const int local = (int)(row - p.seq_q_start[p.row_seq[row]]);
    const int n = local % C;                   // earlier tokens of the row's four
    const float rate = expf(p.a_log[h]);
    const float* q = p.rows_in + row * p.row_stride + p.q_off + kh * d;
    const float* k = p.rows_in + row * p.row_stride + p.k_off + kh * d;
    float a[C - 1], b[C];
#pragma unroll
    for (int s = 0; s < C; s++) {
        if (s < C - 1) a[s] = 0.f;
        b[s] = 0.f;
    }
    float g_head[C];       // one decay a head: of this row and of the earlier ones of its four, backwards
    if (!CHANNEL) {
#pragma unroll
        for (int s = 0; s < C; s++)
            g_head[s] = s <= n ? decay_factor(p.decay_in[(row - s) * p.decay_stride + h] + p.dt_bias[h], rate) : 1.f;
        if (lane == 0) p.decay_out[row * p.heads + h] = g_head[0];
    }
    for (int c = lane; c < d; c += 32) {
        const float qc = q[c], kc = k[c];
        float between = 1.f;                   // the decays behind the other token up to this one
#pragma unroll
        for (int s = 0; s < C; s++) {          // s tokens back
            if (s > n) break;
            const float ks = s == 0 ? kc : k[c - s * p.row_stride];
            if (s > 0) a[s - 1] = fmaf(kc, between * ks, a[s - 1]);
            b[s] = fmaf(qc, between * ks, b[s]);
            if (CHANNEL) {
                if (s < C - 1 && (s < n || s == 0)) {
                    const float g = decay_factor(p.decay_in[(row - s) * p.decay_stride + h * d + c] + p.dt_bias[h * d + c], rate);
                    if (s == 0) p.decay_out[row * (int64_t)p.heads * d + h * d + c] = g;
                    between *= g;
                }
            } else {
                between *= g_head[s];
            }
        }
    }
#pragma unroll
    for (int s = 0; s < C; s++) {
        if (s < C - 1) a[s] = warp_sum(a[s]);
        b[s] = warp_sum(b[s]);
    }
    if (lane == 0) {
        float out[8];
#pragma unroll
        for (int e = 0; e < 8; e++) out[e] = 0.f;
        out[3] = sigmoid_f(p.beta_in[row * p.beta_stride + h]);
#pragma unroll
        for (int e = 0; e < C; e++) {          // token e of the four is n - e tokens back
#pragma unroll
            for (int s = 0; s < C; s++) {
                if (n - e != s) continue;
                out[4 + e] = b[s];
                if (s > 0 && e < C - 1) out[e] = a[s - 1];
            }
        }
        float4* dst = reinterpret_cast<float4*>(p.coef + (row * p.heads + h) * 8);
        dst[0] = make_float4(out[0], out[1], out[2], out[3]);
        dst[1] = make_float4(out[4], out[5], out[6], out[7]);
    }
}

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
template <int RC, int CW, bool CHANNEL>
__global__ void __launch_bounds__(THREADS) gated_delta_scan_kernel(GatedDeltaParams p) {
    constexpr int D = 32 * RC, COLS = WARPS * CW;
    constexpr int V = RC < 4 ? RC : 4;           // neighbouring channels of a lane: lane l has l V .. l V + V - 1 of every 32 V
    constexpr int NV = 2 * C * CW;               // sums of four tokens: S^T (G k), then S^T (G q), token by token
    constexpr int ITEMS = (TT / C * D + THREADS - 1) / THREADS;   // (four tokens, channel) pieces a thread stages
    __shared__ __align__(16) float gk_s[TT][D], gq_s[TT][D], kp_s[TT][D], gc_s[TT / C][D];
    __shared__ __align__(16) float v_s[TT][COLS], u_s[TT][COLS], p2_s[TT][COLS], coef_s[TT][8];
    __shared__ float st_s[D][COLS + 1];

    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int d = p.d, dv = p.dv, H = p.heads;
    const int h = blockIdx.y, seq = blockIdx.z, kh = h / (H / p.kv_heads);
    const int j0 = blockIdx.x * COLS;
    const int q_len = p.seq_q_len[seq], q_start = p.seq_q_start[seq];
    int slot = p.seq_slot[seq];
    if (!gb_check(slot, p.max_slots, GB_CHECK_SLOT)) slot = 0;
    float* S = p.state + (int64_t)slot * p.slot_stride + (int64_t)h * p.head_stride;
    auto channel = [&](int i) { return i / V * (32 * V) + lane * V + i % V; };

    for (int idx = tid; idx < D * COLS; idx += THREADS) {
        const int c = idx / COLS, jj = idx % COLS;
        st_s[c][jj] = (c < d && j0 + jj < dv) ? S[(int64_t)c * dv + j0 + jj] : 0.f;
    }
    __syncthreads();
    float st[RC][CW];
#pragma unroll
    for (int i = 0; i < RC; i++)
#pragma unroll
        for (int c = 0; c < CW; c++) st[i][c] = st_s[channel(i)][warp * CW + c];

    // A tile's rows are fetched into registers while the tile before it is worked on: every load is unconditional (indices
    // clamped), so they are all in flight at once; what is not there changes nothing (decay 1, key 0, strength 0).
    float rq[ITEMS][C], rk[ITEMS][C], rg[ITEMS][C], rv = 0.f, rcoef = 0.f;
    auto fetch = [&](int t0) {
        const int nt = q_len - t0 < TT ? q_len - t0 : TT;
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
                const int64_t row = q_start + t0 + t;
                const float* r = p.rows_in + row * p.row_stride + kh * d + c;
                rq[e][j] = r[p.q_off];
                rk[e][j] = r[p.k_off];
                rg[e][j] = CHANNEL ? p.decay_out[(row * H + h) * d + c] : p.decay_out[row * H + h];
            }
        }
        if (tid < TT * COLS) {
            int t = tid / COLS, jj = j0 + tid % COLS;
            t = t < nt ? t : nt - 1;
            jj = jj < dv ? jj : dv - 1;
            rv = p.rows_in[(int64_t)(q_start + t0 + t) * p.row_stride + p.v_off + h * dv + jj];
        }
        if (tid < TT * 8) {
            int t = tid >> 3;
            t = t < nt ? t : nt - 1;
            rcoef = p.coef[((int64_t)(q_start + t0 + t) * H + h) * 8 + (tid & 7)];
        }
    };
    if (q_len > 0) fetch(0);
    for (int t0 = 0; t0 < q_len; t0 += TT) {
        const int nt = q_len - t0 < TT ? q_len - t0 : TT;
        __syncthreads();   // the tile before is done with
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
                gk_s[t][c] = rk[e][j] * up;
                gq_s[t][c] = there ? rq[e][j] * up : 0.f;
            }
            gc_s[ch][c] = up;
            float down = 1.f;
#pragma unroll
            for (int j = C - 1; j >= 0; j--) {
                kp_s[ch * C + j][c] = rk[e][j] * down;
                down *= rg[e][j];
            }
        }
        if (tid < TT * COLS) {
            const int t = tid / COLS, jj = tid % COLS;
            v_s[t][jj] = (t < nt && j0 + jj < dv) ? rv : 0.f;
        }
        if (tid < TT * 8) coef_s[tid >> 3][tid & 7] = (tid >> 3) < nt ? rcoef : 0.f;
        __syncthreads();
        if (t0 + TT < q_len) fetch(t0 + TT);
#pragma unroll
        for (int ch = 0; ch < TT / C; ch++) {
            float acc[NV];
#pragma unroll
            for (int j = 0; j < C; j++) {
                float s1[CW], s2[CW];
#pragma unroll
                for (int c = 0; c < CW; c++) s1[c] = s2[c] = 0.f;
#pragma unroll
                for (int i = 0; i < RC; i += V) {
                    float k4[V], q4[V];
                    lds<V>(&gk_s[ch * C + j][channel(i)], k4);
                    lds<V>(&gq_s[ch * C + j][channel(i)], q4);
#pragma unroll
                    for (int u = 0; u < V; u++)
#pragma unroll
                        for (int c = 0; c < CW; c++) {
                            s1[c] = fmaf(k4[u], st[i + u][c], s1[c]);
                            s2[c] = fmaf(q4[u], st[i + u][c], s2[c]);
                        }
                }
#pragma unroll
                for (int c = 0; c < CW; c++) {
                    acc[j * CW + c] = s1[c];
                    acc[C * CW + j * CW + c] = s2[c];
                }
            }
            const float total = add_over_lanes<NV, 16>(acc, lane);
            constexpr int PER = 32 / NV;              // lanes that hold the same sum
            float u[C][CW];
#pragma unroll
            for (int j = 0; j < C; j++)
#pragma unroll
                for (int c = 0; c < CW; c++) u[j][c] = __shfl_sync(0xffffffffu, total, (j * CW + c) * PER);
            if (lane >= 16 && lane % PER == 0) {
                const int at = (lane - 16) / PER;
                p2_s[ch * C + at / CW][warp * CW + at % CW] = total;
            }
#pragma unroll
            for (int j = 0; j < C; j++) {
                const float4 a4 = *reinterpret_cast<const float4*>(&coef_s[ch * C + j][0]);
                const float aa[C - 1] = {a4.x, a4.y, a4.z};
                float vj[CW];
                lds<CW>(&v_s[ch * C + j][warp * CW], vj);
#pragma unroll
                for (int c = 0; c < CW; c++) {
                    float t = vj[c] - u[j][c];
#pragma unroll
                    for (int s = 0; s < j; s++) t = fmaf(-aa[s], u[s][c], t);
                    u[j][c] = a4.w * t;
                }
            }
            if (lane == 0) {
#pragma unroll
                for (int j = 0; j < C; j++) sts<CW>(&u_s[ch * C + j][warp * CW], u[j]);
            }
#pragma unroll
            for (int i = 0; i < RC; i += V) {
                float g4[V];
                lds<V>(&gc_s[ch][channel(i)], g4);
#pragma unroll
                for (int w = 0; w < V; w++)
#pragma unroll
                    for (int c = 0; c < CW; c++) st[i + w][c] *= g4[w];
#pragma unroll
                for (int j = 0; j < C; j++) {
                    float k4[V];
                    lds<V>(&kp_s[ch * C + j][channel(i)], k4);
#pragma unroll
                    for (int w = 0; w < V; w++)
#pragma unroll
                        for (int c = 0; c < CW; c++) st[i + w][c] = fmaf(k4[w], u[j][c], st[i + w][c]);
                }
            }
        }
        __syncthreads();
        for (int idx = tid; idx < nt * COLS; idx += THREADS) {
            const int t = idx / COLS, jj = idx % COLS;
            float o = p2_s[t][jj];
#pragma unroll
            for (int s = 0; s < C; s++) o = fmaf(coef_s[t][4 + s], u_s[t / C * C + s][jj], o);     // B is zero for later tokens
            if (j0 + jj < dv) p.out[(int64_t)(q_start + t0 + t) * p.out_stride + h * dv + j0 + jj] = o;
        }
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < RC; i++)
#pragma unroll
        for (int c = 0; c < CW; c++) st_s[channel(i)][warp * CW + c] = st[i][c];
    __syncthreads();
    for (int idx = tid; idx < D * COLS; idx += THREADS) {
        const int c = idx / COLS, jj = idx % COLS;
        if (c < d && j0 + jj < dv) S[(int64_t)c * dv + j0 + jj] = st_s[c][jj];
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
    gated_delta_scan_kernel<RC, CW, CHANNEL><<<dim3(ceil_div(p.dv, WARPS * CW), p.heads, p.nseq), THREADS, 0, stream>>>(p);
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
    if (!p.coef || !p.decay_out || !p.row_seq) GB_REFUSE("gated_delta: no room for the tokens' factors");
    gated_delta_prep_kernel<CHANNEL><<<dim3(p.rows, ceil_div(p.heads, 4)), 128, 0, stream>>>(p);
    GB_CHECK_LAUNCH("gated_delta_prep");
    // few (head, column block) pairs: two columns a warp leave more CTAs, and warps, to hide one another's chains
    const bool narrow = (int64_t)p.heads * p.nseq * ceil_div(p.dv, 16) < p.narrow_below;
    const int rc = ceil_div(p.d, 32);
    if (rc <= 1) return narrow ? launch_scan<1, 2, CHANNEL>(p, stream) : launch_scan<1, 4, CHANNEL>(p, stream);
    if (rc <= 2) return narrow ? launch_scan<2, 2, CHANNEL>(p, stream) : launch_scan<2, 4, CHANNEL>(p, stream);
    if (rc <= 4) return narrow ? launch_scan<4, 2, CHANNEL>(p, stream) : launch_scan<4, 4, CHANNEL>(p, stream);
    return narrow ? launch_scan<8, 2, CHANNEL>(p, stream) : launch_scan<8, 4, CHANNEL>(p, stream);
}

}  // namespace

GB_API int gb_gated_delta(const GatedDeltaParams* pp, cudaStream_t stream) {
    GatedDeltaParams p = *pp;
    if (p.nseq <= 0 || p.rows <= 0) return 0;
    if (p.heads <= 0 || p.kv_heads <= 0 || p.heads % p.kv_heads || p.d <= 0 || p.d > 256 || p.dv <= 0)
        GB_REFUSE("gated_delta: %d heads over %d of %d key and %d value channels; at most 256 key channels", p.heads, p.kv_heads, p.d, p.dv);
    if (!p.rows_in || !p.decay_in || !p.beta_in || !p.a_log || !p.dt_bias || !p.state || !p.out) GB_REFUSE("gated_delta: a tensor is missing");
    if (p.head_stride < (int64_t)p.d * p.dv || p.slot_stride < p.head_stride * p.heads) GB_REFUSE("gated_delta: the state is too small for its heads");
    if (p.per_channel) return launch<true>(p, stream);
    return launch<false>(p, stream);
}

// the checked build's record of the first index this file's kernels found out of bounds
GB_CHECK_READER(gb_checked_status_gated_delta)
