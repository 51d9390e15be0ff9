// The kernels of a delta-rule mixer that are neither matrix products nor the chunked form (delta_chunk.cu): what happens to
// the projections in front of the recurrence, the recurrence token by token, and the gated norm behind it.
//
// Per head h (key head g = h / (H / G)), with q_t, k_t [D] unit vectors (q times q_scale), v_t [DV], a step size beta_t and a
// decay a_t per key channel, or one for all of them:
//     S <- diag(a_t) S;   u = beta_t (v_t - S^T k_t);   S <- S + k_t u^T;   o_t = S^T q_t
// S is float32 [D, DV], lives in the request's state slot as [H][DV][D] and is carried from token to token; the last K - 1
// inputs of the short convolution stand behind it ([K - 1][channels], oldest first), and the recurrence's kernels move those on
// when they are done with a request's rows.
//
//   delta_prepare    a warp per (token, head of q, k or v): the causal convolution per channel over the last K inputs (kept ones
//                    where a portion starts, zeros before a request's start), silu, and for q and k the division by
//                    sqrt(sum of squares + 1e-6).  Split-K partial sums of the projections are added up on the way in.  More
//                    warps per token finish what else the projections' rows hold: beta = sigmoid, the decay's logarithm where
//                    there is one per head, the rows of the low-rank products, the gate's logits when they came in parts.
//   delta_scan       token by token: a group of lanes holds four columns of S, the channels spread over the lanes.  With R the
//                    decayed state, u = beta (v - R^T k) and o = R^T q + (k . q) u, so a token costs one round of butterflies.
//                    Decoding, short portions, float32.
//   head_norm_gate   o / sqrt(mean over the head of o^2 + eps) * weight * silu or sigmoid of the gate.
// Everything here is float32 arithmetic; the rows may be stored in bfloat16.
#include "delta_rule.cuh"

#include <math.h>

namespace {

using namespace ph;

constexpr int PREP_WARPS = 8;
constexpr int TAIL = 128;               // elements of a tail unit
constexpr int RUN = 8;                  // tokens that a warp walks where there are many rows (RUN_FROM of them)
constexpr int RUN_FROM = 256;
constexpr float UNIT_EPS = 1e-6f;

struct PrepParams {
    const void* rows; int splits; long long split_stride, width;
    const float* taps;                                          // [K][channels]
    const float* state; long long state_stride, conv_at;
    const int32_t* row_seg; const int32_t* seg_start; const int32_t* seg_slot;
    int H, G, D, DV, K;
    int qk_v, qk_n, v_v, v_n;                                   // elements per access and accesses per lane of a q / k and of a v head
    float q_scale;
    float* qkv;                                                 // [T, channels]
    int b_col; float* beta;                                     // [T, H]
    int a_col; const float* rate; const float* a_bias; float* log_decay;        // [H], [H], [T, H]; a_col < 0: no decay per head
    int low_col, low_n; void* low;                              // [T, low_n], 0: none
    int gate_col, gate_n; void* gate;                           // [T, gate_n], 0: stays in the rows
};

template <int V, typename T> __device__ __forceinline__ void get_v(const T* p, float* v) {
    if constexpr (V == 4) { const float4 u = load4(p); v[0] = u.x; v[1] = u.y; v[2] = u.z; v[3] = u.w; }
    else v[0] = to_float<T>(*p);
}

// One head of q (kind 0), k (1) or v (2) for token t: channels c0 .. c0 + n - 1, lane l takes (i * 32 + l) * V .. + V - 1.
template <typename TI, int V, int NI>
__device__ __forceinline__ void conv_head(const PrepParams& p, int t, int kind, int c0, int n) {
    const int lane = threadIdx.x & 31, CH = 2 * p.G * p.D + p.H * p.DV;
    const int s = p.row_seg[t], first = p.seg_start[s], i0 = t - first;
    const float* past = p.state + (size_t)p.seg_slot[s] * p.state_stride + p.conv_at;
    const TI* rows = static_cast<const TI*>(p.rows);
    float y[NI * V];
#pragma unroll
    for (int i = 0; i < NI * V; ++i) y[i] = 0.0f;
#pragma unroll 4
    for (int j = 0; j < p.K; ++j) {
        const int src = i0 - (p.K - 1) + j;
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const int d = (i * 32 + lane) * V;
            if (d >= n) continue;
            float x[V], w[V];
            if (src >= 0) {
                const TI* at = rows + (size_t)(first + src) * p.width + c0 + d;
                get_v<V>(at, x);
                for (int sp = 1; sp < p.splits; ++sp) {
                    float more[V];
                    get_v<V>(at + (size_t)sp * p.split_stride, more);
#pragma unroll
                    for (int e = 0; e < V; ++e) x[e] += more[e];
                }
            } else {
                get_v<V>(past + (size_t)(src + p.K - 1) * CH + c0 + d, x);
            }
            get_v<V>(p.taps + (size_t)j * CH + c0 + d, w);
#pragma unroll
            for (int e = 0; e < V; ++e) y[i * V + e] = fmaf(w[e], x[e], y[i * V + e]);
        }
    }
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < NI * V; ++i) {
        y[i] = y[i] / (1.0f + expf(-y[i]));
        ss += y[i] * y[i];
    }
    float f = 1.0f;
    if (kind < 2) f = rsqrtf(warp_sum(ss) + UNIT_EPS) * (kind == 0 ? p.q_scale : 1.0f);
    float* out = p.qkv + (size_t)t * CH + c0;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const int d = (i * 32 + lane) * V;
        if (d >= n) continue;
        if constexpr (V == 4) *reinterpret_cast<float4*>(out + d) = make_float4(y[4 * i] * f, y[4 * i + 1] * f, y[4 * i + 2] * f, y[4 * i + 3] * f);
        else out[d] = y[i] * f;
    }
}

template <typename TI>
__device__ __forceinline__ void conv_any(const PrepParams& p, int t, int kind, int c0, int n, int v, int ni) {
    if (v == 4) {
        if (ni <= 1) conv_head<TI, 4, 1>(p, t, kind, c0, n);
        else if (ni <= 2) conv_head<TI, 4, 2>(p, t, kind, c0, n);
        else conv_head<TI, 4, 4>(p, t, kind, c0, n);
    } else {
        if (ni <= 1) conv_head<TI, 1, 1>(p, t, kind, c0, n);
        else if (ni <= 4) conv_head<TI, 1, 4>(p, t, kind, c0, n);
        else conv_head<TI, 1, 16>(p, t, kind, c0, n);
    }
}

// silu; in a bfloat16 model from the hardware's exponential and reciprocal, still float32 (relative error about 1e-6)
template <bool FAST> __device__ __forceinline__ float silu(float v) { return FAST ? __fdividef(v, 1.0f + __expf(-v)) : v / (1.0f + expf(-v)); }

// The same for the tokens t .. t_end - 1 with the last KT inputs in registers, so that a row is read once, R rows on their
// way at a time: heads of up to 128 channels, four per lane.  The order of each sum is the one above.
template <typename TI, int KT, bool FAST, int R>
__device__ __forceinline__ void conv_run(const PrepParams& p, int t, int t_end, int kind, int c0, int n) {
    const int lane = threadIdx.x & 31, d = lane * 4, CH = 2 * p.G * p.D + p.H * p.DV;
    const bool on = d < n;
    const float4 none = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    const TI* rows = static_cast<const TI*>(p.rows) + c0 + d;
    float4 w[KT], x[KT + R - 1];
#pragma unroll
    for (int j = 0; j < KT; ++j) w[j] = on ? load4(p.taps + (size_t)j * CH + c0 + d) : none;
    auto input = [&](int row) {
        if (!on) return none;
        float4 v = load4(rows + (size_t)row * p.width);
        for (int sp = 1; sp < p.splits; ++sp) {
            const float4 m = load4(rows + (size_t)row * p.width + (size_t)sp * p.split_stride);
            v.x += m.x; v.y += m.y; v.z += m.z; v.w += m.w;
        }
        return v;
    };
    while (t < t_end) {
        const int s = p.row_seg[t], first = p.seg_start[s], stop = min(t_end, p.seg_start[s + 1]);
        const float* past = p.state + (size_t)p.seg_slot[s] * p.state_stride + p.conv_at + c0 + d;
#pragma unroll
        for (int j = 0; j < KT - 1; ++j) {
            const int src = t - first - (KT - 1) + j;
            x[j] = src >= 0 ? input(first + src) : on ? load4(past + (size_t)(src + KT - 1) * CH) : none;
        }
        for (; t < stop; t += R) {
#pragma unroll
            for (int r = 0; r < R; ++r) x[KT - 1 + r] = t + r < stop ? input(t + r) : none;
#pragma unroll
            for (int r = 0; r < R; ++r) {
                float4 y = none;
#pragma unroll
                for (int j = 0; j < KT; ++j) {
                    y.x = fmaf(w[j].x, x[r + j].x, y.x); y.y = fmaf(w[j].y, x[r + j].y, y.y);
                    y.z = fmaf(w[j].z, x[r + j].z, y.z); y.w = fmaf(w[j].w, x[r + j].w, y.w);
                }
                y.x = silu<FAST>(y.x); y.y = silu<FAST>(y.y); y.z = silu<FAST>(y.z); y.w = silu<FAST>(y.w);
                float f = 1.0f;
                if (kind < 2) {
                    float ss = 0.0f;
                    ss += y.x * y.x; ss += y.y * y.y; ss += y.z * y.z; ss += y.w * y.w;
                    f = rsqrtf(warp_sum(ss) + UNIT_EPS) * (kind == 0 ? p.q_scale : 1.0f);
                }
                if (on && t + r < stop)
                    *reinterpret_cast<float4*>(p.qkv + (size_t)(t + r) * CH + c0 + d) = make_float4(y.x * f, y.y * f, y.z * f, y.w * f);
            }
#pragma unroll
            for (int j = 0; j < KT - 1; ++j) x[j] = x[j + R];
        }
        t = stop;
    }
}

// The tail of a token's row, [beta | decay | low rows | gate]: TAIL elements by a warp.  TO: the model's dtype.
template <typename TI, typename TO>
__device__ __forceinline__ void finish_tail(const PrepParams& p, int t, int part) {
    const TI* row = static_cast<const TI*>(p.rows) + (size_t)t * p.width;
    const int nb = p.H, na = p.a_col >= 0 ? p.H : 0, all = nb + na + p.low_n + p.gate_n;
#pragma unroll
    for (int k = 0; k < TAIL / 32; ++k) {
        int i = part * TAIL + k * 32 + (threadIdx.x & 31);
        if (i >= all) break;
        const int which = i < nb ? 0 : i < nb + na ? 1 : i < nb + na + p.low_n ? 2 : 3;
        i -= which == 0 ? 0 : which == 1 ? nb : which == 2 ? nb + na : nb + na + p.low_n;
        const TI* from = row + i + (which == 0 ? p.b_col : which == 1 ? p.a_col : which == 2 ? p.low_col : p.gate_col);
        float v = to_float<TI>(*from);
        for (int s = 1; s < p.splits; ++s) v += to_float<TI>(from[(size_t)s * p.split_stride]);
        if (which == 0) p.beta[(size_t)t * p.H + i] = 1.0f / (1.0f + expf(-v));
        else if (which == 1) p.log_decay[(size_t)t * p.H + i] = p.rate[i] * ph_delta::softplus(v + p.a_bias[i]);
        else if (which == 2) static_cast<TO*>(p.low)[(size_t)t * p.low_n + i] = from_float<TO>(v);
        else static_cast<TO*>(p.gate)[(size_t)t * p.gate_n + i] = from_float<TO>(v);
    }
}

// TI: the dtype of the rows (rows in parts are float32 in a bfloat16 model too)
template <typename TI, typename TO>
__global__ void __launch_bounds__(PREP_WARPS * 32, 2) delta_prepare_kernel(const PrepParams p) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    int unit = blockIdx.y * PREP_WARPS + (threadIdx.x >> 5);
    if (unit < 2 * p.G) {
        conv_any<TI>(p, t, unit < p.G ? 0 : 1, unit * p.D, p.D, p.qk_v, p.qk_n);
        return;
    }
    unit -= 2 * p.G;
    if (unit < p.H) {
        conv_any<TI>(p, t, 2, 2 * p.G * p.D + unit * p.DV, p.DV, p.v_v, p.v_n);
        return;
    }
    finish_tail<TI, TO>(p, t, unit - p.H);
}

// The form for the usual heads and taps: a warp per (`run` tokens, head), and per (token, part of the tail).
template <typename TI, typename TO, int KT, int R>
__global__ void __launch_bounds__(PREP_WARPS * 32, 3) delta_prepare_run_kernel(const PrepParams p, int T) {
    constexpr int run = R == 1 ? 1 : RUN;
    constexpr bool FAST = sizeof(TO) == 2;
    pdl_launch_dependents();
    pdl_wait();
    const int t0 = blockIdx.x * run;
    int unit = blockIdx.y * PREP_WARPS + (threadIdx.x >> 5);
    const int heads = 2 * p.G + p.H;
    if (unit < heads) {
        const int kind = unit < p.G ? 0 : unit < 2 * p.G ? 1 : 2;
        conv_run<TI, KT, FAST, R>(p, t0, min(T, t0 + run), kind, kind < 2 ? unit * p.D : 2 * p.G * p.D + (unit - 2 * p.G) * p.DV, kind < 2 ? p.D : p.DV);
        return;
    }
    unit -= heads;
    if (t0 + unit % run < T) finish_tail<TI, TO>(p, t0 + unit % run, unit / run);
}

constexpr int SCAN_THREADS = 128, SCAN_COLS = 4;

// L lanes per group of SCAN_COLS columns; lane l holds the channels (i * L + l) * V .. + V - 1 of each, i < NI.
template <typename TI, int NI, int V>
__global__ void __launch_bounds__(SCAN_THREADS) delta_scan_kernel(const ph_delta::ScanParams p, int L) {
    constexpr int N = NI * V;
    pdl_launch_dependents();
    const int seg = blockIdx.z, h = blockIdx.y;
    const int row0 = p.seg_start[seg], n_rows = p.seg_start[seg + 1] - row0;
    if (n_rows < p.rows_from || n_rows > p.rows_to) { pdl_wait(); return; }
    const int lane = threadIdx.x % L, group = threadIdx.x / L;
    const int D = p.D, DV = p.DV, CH = 2 * p.G * D + p.H * DV;
    const int c0 = (blockIdx.x * (SCAN_THREADS / L) + group) * SCAN_COLS;
    const int g = h / (p.H / p.G);
    float* st = p.state + (size_t)p.seg_slot[seg] * p.state_stride;
    float* S0 = st + (size_t)h * DV * D;
    const float rate = p.z ? p.rate[h] : 0.0f;
    float bias[N];
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const int d = (i * L + lane) * V;
#pragma unroll
        for (int j = 0; j < V; ++j) bias[i * V + j] = p.z && d + j < D ? p.z_bias[(size_t)h * D + d + j] : 0.0f;
    }
    pdl_wait();
    float S[SCAN_COLS][N];
#pragma unroll
    for (int c = 0; c < SCAN_COLS; ++c)
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const int d = (i * L + lane) * V;
#pragma unroll
            for (int j = 0; j < V; ++j) S[c][i * V + j] = 0.0f;
            if (c0 + c < DV && d < D) get_v<V>(S0 + (size_t)(c0 + c) * D + d, &S[c][i * V]);
        }
    struct Token { float q[N], k[N], z[N], v[SCAN_COLS], beta, log_decay; };
    auto fetch = [&](int t, Token& x) {
        const float* row = p.qkv + (size_t)(row0 + t) * CH;
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const int d = (i * L + lane) * V;
#pragma unroll
            for (int j = 0; j < V; ++j) x.q[i * V + j] = x.k[i * V + j] = x.z[i * V + j] = 0.0f;
            if (d < D) {
                get_v<V>(row + (size_t)g * D + d, &x.q[i * V]);
                get_v<V>(row + (size_t)(p.G + g) * D + d, &x.k[i * V]);
                if (p.z) get_v<V>(p.z + (size_t)(row0 + t) * p.z_stride + (size_t)h * D + d, &x.z[i * V]);
            }
        }
#pragma unroll
        for (int c = 0; c < SCAN_COLS; ++c) x.v[c] = c0 + c < DV ? row[2 * p.G * D + (size_t)h * DV + c0 + c] : 0.0f;
        x.beta = p.beta[(size_t)(row0 + t) * p.H + h];
        x.log_decay = p.log_decay ? p.log_decay[(size_t)(row0 + t) * p.H + h] : 0.0f;
    };
    Token next;
    fetch(0, next);
    for (int t = 0; t < n_rows; ++t) {
        const Token x = next;
        if (t + 1 < n_rows) fetch(t + 1, next);
        const float all = expf(x.log_decay);
        float sk[SCAN_COLS], sq[SCAN_COLS], kq = 0.0f;
#pragma unroll
        for (int c = 0; c < SCAN_COLS; ++c) sk[c] = sq[c] = 0.0f;
#pragma unroll
        for (int i = 0; i < N; ++i) {
            const float a = p.z ? expf(rate * ph_delta::softplus(x.z[i] + bias[i])) : all;
            kq = fmaf(x.k[i], x.q[i], kq);
#pragma unroll
            for (int c = 0; c < SCAN_COLS; ++c) {
                S[c][i] *= a;
                sk[c] = fmaf(S[c][i], x.k[i], sk[c]);
                sq[c] = fmaf(S[c][i], x.q[i], sq[c]);
            }
        }
        for (int o = L >> 1; o > 0; o >>= 1) {
            kq += __shfl_xor_sync(0xffffffffu, kq, o);
#pragma unroll
            for (int c = 0; c < SCAN_COLS; ++c) {
                sk[c] += __shfl_xor_sync(0xffffffffu, sk[c], o);
                sq[c] += __shfl_xor_sync(0xffffffffu, sq[c], o);
            }
        }
        float* y = p.o + (size_t)(row0 + t) * p.H * DV + (size_t)h * DV + c0;
#pragma unroll
        for (int c = 0; c < SCAN_COLS; ++c) {
            const float u = x.beta * (x.v[c] - sk[c]);
#pragma unroll
            for (int i = 0; i < N; ++i) S[c][i] = fmaf(x.k[i], u, S[c][i]);
            if (lane == 0 && c0 + c < DV) y[c] = fmaf(kq, u, sq[c]);
        }
    }
#pragma unroll
    for (int c = 0; c < SCAN_COLS; ++c)
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const int d = (i * L + lane) * V;
            if (c0 + c >= DV || d >= D) continue;
            if constexpr (V == 4) store4(S0 + (size_t)(c0 + c) * D + d, &S[c][i * V]);
            else S0[(size_t)(c0 + c) * D + d] = S[c][i];
        }
    ph_delta::move_conv_inputs<TI>(p, st, row0, n_rows, blockIdx.y * gridDim.x + blockIdx.x, gridDim.x * gridDim.y, threadIdx.x, SCAN_THREADS);
}

// A warp per (token, head).
template <typename TG, typename TO>
__global__ void __launch_bounds__(256) head_norm_gate_kernel(const float* __restrict__ o, const float* __restrict__ w, float eps,
                                                             const TG* __restrict__ gate, long long gate_stride, int act, TO* __restrict__ out,
                                                             long long items, int H, int DV, int vec) {
    pdl_launch_dependents();
    pdl_wait();
    const long long item = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (item >= items) return;
    const int lane = threadIdx.x & 31;
    const long long t = item / H;
    const int h = (int)(item % H);
    const float* src = o + item * DV;
    const TG* gr = gate + t * gate_stride + (size_t)h * DV;
    TO* dst = out + item * DV;
    auto open = [&](float g) { const float s = 1.0f / (1.0f + expf(-g)); return act ? s : g * s; };
    float ss = 0.0f;
    if (vec) {
        for (int c = lane * 4; c < DV; c += 128) {
            const float4 v = load4(src + c);
            ss += (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w);
        }
        const float inv = rsqrtf(warp_sum(ss) / (float)DV + eps);
        for (int c = lane * 4; c < DV; c += 128) {
            const float4 v = load4(src + c), ww = load4(w + c), g = load4(gr + c);
            const float r[4] = {v.x * inv * ww.x * open(g.x), v.y * inv * ww.y * open(g.y), v.z * inv * ww.z * open(g.z), v.w * inv * ww.w * open(g.w)};
            store4(dst + c, r);
        }
        return;
    }
    for (int c = lane; c < DV; c += 32) ss += src[c] * src[c];
    const float inv = rsqrtf(warp_sum(ss) / (float)DV + eps);
    for (int c = lane; c < DV; c += 32) dst[c] = from_float<TO>(src[c] * inv * w[c] * open(to_float<TG>(gr[c])));
}

// elements per access and accesses per lane for n channels at columns that are multiples of `align`
void lanes_for(int n, bool vec, int* v, int* ni) {
    *v = vec ? 4 : 1;
    *ni = (n + 32 * *v - 1) / (32 * *v);
}

}  // namespace

// rows [splits][T][width] in rows_dtype: [q (G D) | k (G D) | v (H DV) | ...]; taps [K][2 G D + H DV] float32, the current
// token's last.  state: the request's slots, the convolution's inputs conv_at floats into each.  b_col, a_col (< 0: none),
// low_col / low_n, gate_col / gate_n (0: none): where the rest of a row is.  low and gate are written in model_dtype.
PH_EXPORT int ph_delta_prepare(const void* rows, int rows_dtype, int splits, long long split_stride, long long width, const float* taps, int K,
                               const float* state, long long state_stride, long long conv_at, const int32_t* row_seg, const int32_t* seg_start,
                               const int32_t* seg_slot, int T, int H, int G, int D, int DV, float q_scale, float* qkv, int b_col, float* beta,
                               int a_col, const float* rate, const float* a_bias, float* log_decay, int low_col, int low_n, void* low,
                               int gate_col, int gate_n, void* gate, int model_dtype, cudaStream_t stream) {
    if (!rows || !taps || !state || !row_seg || !seg_start || !seg_slot || !qkv || !beta || splits < 1 || T < 0 || H < 1 || G < 1 || H % G ||
        D < 1 || DV < 1 || K < 1 || !valid_dtype(rows_dtype) || !valid_dtype(model_dtype) || b_col < 0 ||
        (a_col >= 0 && (!rate || !a_bias || !log_decay)) || low_n < 0 || (low_n && !low) || gate_n < 0 || (gate_n && !gate))
        return fail(PH_ERR_ARG, "delta_prepare: bad arguments (T %d, H %d, G %d, D %d, DV %d, K %d)", T, H, G, D, DV, K);
    const long long CH = 2LL * G * D + (long long)H * DV;
    const long long last[4] = {CH, (long long)b_col + H, a_col >= 0 ? (long long)a_col + H : 0, (long long)low_col + low_n};
    for (long long e : last)
        if (e > width) return fail(PH_ERR_ARG, "delta_prepare: rows of %lld elements hold no %lld", width, e);
    if (gate_n && (long long)gate_col + gate_n > width) return fail(PH_ERR_ARG, "delta_prepare: the gate is outside the rows");
    if (T == 0) return PH_OK;
    PrepParams p;
    p.rows = rows; p.splits = splits; p.split_stride = split_stride; p.width = width; p.taps = taps;
    p.state = state; p.state_stride = state_stride; p.conv_at = conv_at; p.row_seg = row_seg; p.seg_start = seg_start; p.seg_slot = seg_slot;
    p.H = H; p.G = G; p.D = D; p.DV = DV; p.K = K; p.q_scale = q_scale; p.qkv = qkv; p.b_col = b_col; p.beta = beta;
    p.a_col = a_col; p.rate = rate; p.a_bias = a_bias; p.log_decay = log_decay; p.low_col = low_col; p.low_n = low_n; p.low = low;
    p.gate_col = gate_col; p.gate_n = gate_n; p.gate = gate;
    const bool vec = CH % 4 == 0 && width % 4 == 0 && split_stride % 4 == 0 && state_stride % 4 == 0 && conv_at % 4 == 0 &&
                     (((uintptr_t)rows | (uintptr_t)taps | (uintptr_t)state | (uintptr_t)qkv) & 15) == 0;
    lanes_for(D, vec && D % 4 == 0, &p.qk_v, &p.qk_n);
    lanes_for(DV, vec && DV % 4 == 0 && (2LL * G * D) % 4 == 0, &p.v_v, &p.v_n);
    if (D > 512 || DV > 512) return fail(PH_ERR_UNSUPPORTED, "delta_prepare: heads of %d / %d exceed the supported 512", D, DV);
    const int tail = H + (a_col >= 0 ? H : 0) + low_n + gate_n, parts = (tail + TAIL - 1) / TAIL;
    if (p.qk_v == 4 && p.qk_n == 1 && p.v_v == 4 && p.v_n == 1 && K >= 2 && K <= 4) {
        const int run = T >= RUN_FROM ? RUN : 1;
        const dim3 grid((T + run - 1) / run, (2 * G + H + parts * run + PREP_WARPS - 1) / PREP_WARPS);
#define LAUNCH_RUN(TI, TO, KT)                                                                               \
    do {                                                                                                     \
        if (run == 1) launch_overlapped(delta_prepare_run_kernel<TI, TO, KT, 1>, grid, dim3(PREP_WARPS * 32), 0, stream, p, T); \
        else launch_overlapped(delta_prepare_run_kernel<TI, TO, KT, 4>, grid, dim3(PREP_WARPS * 32), 0, stream, p, T); \
    } while (0)
#define LAUNCH_K(TI, TO)                                                                                     \
    do {                                                                                                     \
        if (K == 2) LAUNCH_RUN(TI, TO, 2); else if (K == 3) LAUNCH_RUN(TI, TO, 3); else LAUNCH_RUN(TI, TO, 4); \
    } while (0)
        PH_DISPATCH(rows_dtype, TI, PH_DISPATCH(model_dtype, TO, LAUNCH_K(TI, TO)));
#undef LAUNCH_K
#undef LAUNCH_RUN
        return check_launch("delta_prepare");
    }
    const dim3 grid(T, (2 * G + H + parts + PREP_WARPS - 1) / PREP_WARPS);
    PH_DISPATCH(rows_dtype, TI, PH_DISPATCH(model_dtype, TO,
        launch_overlapped(delta_prepare_kernel<TI, TO>, grid, dim3(PREP_WARPS * 32), 0, stream, p)));
    return check_launch("delta_prepare");
}

// qkv, beta and log_decay (null: z, a decay per channel) as delta_prepare leaves them; o [T, H DV] float32.
PH_EXPORT int ph_delta_scan(const float* qkv, const float* beta, const float* log_decay, const float* z, long long z_stride, const float* z_bias,
                            const float* rate, const void* rows, int rows_dtype, int splits, long long split_stride, long long width,
                            float* state, long long state_stride, long long conv_at, const int32_t* seg_start, const int32_t* seg_slot, int S,
                            int H, int G, int D, int DV, int K, int rows_from, int rows_to, float* o, cudaStream_t stream) {
    if (!qkv || !beta || (!log_decay == !z) || (z && (!z_bias || !rate)) || !rows || !state || !seg_start || !seg_slot || !o || S < 0 || H < 1 ||
        G < 1 || H % G || D < 1 || DV < 1 || K < 1 || splits < 1 || !valid_dtype(rows_dtype))
        return fail(PH_ERR_ARG, "delta_scan: bad arguments (S %d, H %d, G %d, D %d, DV %d)", S, H, G, D, DV);
    if (D > 512) return fail(PH_ERR_UNSUPPORTED, "delta_scan: heads of %d channels exceed the supported 512", D);
    if (S == 0) return PH_OK;
    ph_delta::ScanParams p;
    p.qkv = qkv; p.beta = beta; p.log_decay = log_decay; p.z = z; p.z_stride = z_stride; p.z_bias = z_bias; p.rate = rate;
    p.rows = rows; p.splits = splits; p.split_stride = split_stride; p.width = width; p.state = state; p.state_stride = state_stride;
    p.conv_at = conv_at; p.seg_start = seg_start; p.seg_slot = seg_slot; p.o = o; p.H = H; p.G = G; p.D = D; p.DV = DV; p.K = K;
    p.rows_from = rows_from; p.rows_to = rows_to > 0 ? rows_to : 0x7fffffff;
    const bool vec = D % 4 == 0 && (2LL * G * D + (long long)H * DV) % 4 == 0 && state_stride % 4 == 0 && z_stride % 4 == 0 &&
                     (((uintptr_t)qkv | (uintptr_t)state | (uintptr_t)z) & 15) == 0;
    const int V = vec ? 4 : 1;
    int L = 1;
    while (L < 32 && L * V < D) L *= 2;
    const int ni = (D + L * V - 1) / (L * V), per_block = SCAN_THREADS / L * SCAN_COLS;
    const dim3 grid((DV + per_block - 1) / per_block, H, S);
#define SCAN(NI, V) PH_DISPATCH(rows_dtype, TI, launch_overlapped(delta_scan_kernel<TI, NI, V>, grid, dim3(SCAN_THREADS), 0, stream, p, L))
    if (V == 4) {
        if (ni <= 1) SCAN(1, 4); else if (ni <= 2) SCAN(2, 4); else SCAN(4, 4);
    } else {
        if (ni <= 1) SCAN(1, 1); else if (ni <= 2) SCAN(2, 1); else if (ni <= 4) SCAN(4, 1); else SCAN(16, 1);
    }
#undef SCAN
    return check_launch("delta_scan");
}

// o [T, H DV] float32 -> out in out_dtype.  gate: rows of H DV logits in gate_dtype, gate_stride elements apart; act 0: silu, 1:
// sigmoid.  w [DV].
PH_EXPORT int ph_head_norm_gate(const float* o, const float* w, float eps, const void* gate, int gate_dtype, long long gate_stride, int act,
                                void* out, int out_dtype, int T, int H, int DV, cudaStream_t stream) {
    if (!o || !w || !gate || !out || T < 0 || H < 1 || DV < 1 || act < 0 || act > 1 || !valid_dtype(gate_dtype) || !valid_dtype(out_dtype))
        return fail(PH_ERR_ARG, "head_norm_gate: bad arguments (T %d, H %d, DV %d)", T, H, DV);
    if (T == 0) return PH_OK;
    const long long items = (long long)T * H;
    const int vec = DV % 4 == 0 && gate_stride % 4 == 0 && (((uintptr_t)o | (uintptr_t)w | (uintptr_t)gate | (uintptr_t)out) & 15) == 0;
    PH_DISPATCH(gate_dtype, TG, PH_DISPATCH(out_dtype, TO,
        launch_overlapped(head_norm_gate_kernel<TG, TO>, dim3((unsigned)((items + 7) / 8)), dim3(256), 0, stream, o, w, eps, (const TG*)gate,
                          gate_stride, act, (TO*)out, items, H, DV, vec)));
    return check_launch("head_norm_gate");
}
