// Attention whose heads talk to each other before the softmax, over cache pages, and the kernel that prepares its
// queries, keys and values.
//
//   joint_norm_kv_write   from the rows [q | k | ...] of one product (partial sums added up): q and k are RMS-normed over
//                         their whole width (all heads as one row, one weight per element; a null weight: no norm), q
//                         goes out in the compute dtype, the normed k goes to the key rows of the token's cache slot, and
//                         the value rows receive k as it was projected, before the norm (values that are the keys), or
//                         the v part of the row when the product has one.
//   attention_talking     for the row at position z and every key p that it sees (first_seen(z) <= p <= z):
//                             s_g = (q_g . k_kv(g)) * scale
//                             s_g = cap * tanh(s_g / cap)                          (cap > 0)
//                             s_g = s_g - r1_g * ln(1 + r2_g * (z - p))            (r1, r2 given; r1 alone: r1_g * (z - p))
//                             s'_h = sum_g talk[h][g] * s_g                        (talk given: [HQ, HQ])
//                         then a softmax over the seen keys per head h (with exp(sink_h) in the denominator when a sink
//                         is given), o_h = sum_p w_hp v_kv(h)p, and o_h * sigmoid(gate_h) when a gate row is given.
//                         Because every head's score enters every head's softmax, one block handles all heads of a row:
//                         warp g scores head g for 32 keys at a time (a key per lane), the block exchanges the scores
//                         through shared memory, and warp h mixes, runs the online softmax and sums the values of head h
//                         (above 32 heads a warp takes two or four heads in turn).
// All arithmetic is float32 in an order that depends on (z, window) only, never on how a request was cut into steps or
// on what else is in the batch.  Cache addressing as in qk_norm_rope.cu.
#include "common.cuh"

#include <math.h>

namespace {

using namespace ph;

constexpr int MAX_DV = 512;      // widest value row
constexpr int MAX_HEADS = 64;    // a block per row: a warp per head up to 32 heads, two or four heads per warp above

// HPW: heads per warp.  A block has ceil(HQ / HPW) warps; warp w takes the heads w, w + warps, ... (at most HPW of them).
template <typename TQ, typename TKV, typename TG, typename TO, int HPW>
__global__ void attention_talking_kernel(const TQ* __restrict__ q, const TKV* __restrict__ k_base, const TKV* __restrict__ v_base,
                                         long long page_stride, int page_size, const int32_t* __restrict__ block_table, int table_stride,
                                         const int32_t* __restrict__ row_seg, const int32_t* __restrict__ positions,
                                         TO* __restrict__ out, int HQ, int HKV, int D, int DV, int window, int chunk, float scale,
                                         float cap, const float* __restrict__ r1, const float* __restrict__ r2,
                                         const float* __restrict__ talk, const float* __restrict__ sink, const TG* __restrict__ gate,
                                         long long gate_stride) {
    extern __shared__ float smem[];
    float* qs = smem;                          // [HQ][D]
    float* sc = qs + (size_t)HQ * D;           // [HQ][32]: the heads' own scores of the current 32 keys
    float* tk = sc + (size_t)HQ * 32;          // [HQ][HQ]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    const int t = blockIdx.x;
    const int group = HQ / HKV;
    const int z = positions[t];
    const int lo = first_seen(z, window, chunk);
    const int32_t* table = block_table + (size_t)row_seg[t] * table_stride;
    const TQ* qr = q + (size_t)t * HQ * D;
    for (int i = threadIdx.x; i < HQ * D; i += blockDim.x) qs[i] = to_float<TQ>(qr[i]);
    if (talk)
        for (int i = threadIdx.x; i < HQ * HQ; i += blockDim.x) tk[i] = talk[i];
    __syncthreads();

    float m[HPW], l[HPW];
    float acc[HPW][MAX_DV / 32];
#pragma unroll
    for (int u = 0; u < HPW; ++u) {
        m[u] = -INFINITY; l[u] = 0.0f;
#pragma unroll
        for (int i = 0; i < MAX_DV / 32; ++i) acc[u][i] = 0.0f;
    }

    for (int base = lo; base <= z; base += 32) {
        const int p = base + lane;
        const bool seen = p <= z;
        int page = 0, off = 0;
        if (seen) { page = table[p / page_size]; off = p % page_size; }
        float s[HPW];
#pragma unroll
        for (int u = 0; u < HPW; ++u) {
            const int h = warp + u * warps;
            s[u] = 0.0f;
            if (h < HQ && seen) {
                const TKV* krow = k_base + (size_t)page * page_stride + ((size_t)(h / group) * page_size + off) * D;
                const float* qh = qs + (size_t)h * D;
                float dot = 0.0f;
                for (int d = 0; d < D; ++d) dot += qh[d] * to_float<TKV>(krow[d]);
                float v = dot * scale;
                if (cap > 0.0f) v = cap * tanhf(v / cap);
                if (r1) v -= r1[h] * (r2 ? log1pf(r2[h] * (float)(z - p)) : (float)(z - p));
                s[u] = v;
            }
        }
        if (talk) {
#pragma unroll
            for (int u = 0; u < HPW; ++u) {
                const int h = warp + u * warps;
                if (h < HQ) sc[h * 32 + lane] = s[u];
            }
            __syncthreads();
#pragma unroll
            for (int u = 0; u < HPW; ++u) {
                const int h = warp + u * warps;
                if (h >= HQ) continue;
                float mixed = 0.0f;
                for (int j = 0; j < HQ; ++j) mixed += tk[h * HQ + j] * sc[j * 32 + lane];
                s[u] = mixed;
            }
        }
        const int n = (z - base + 1) < 32 ? (z - base + 1) : 32;
#pragma unroll
        for (int u = 0; u < HPW; ++u) {
            const int h = warp + u * warps;
            if (h >= HQ) continue;                         // the whole warp: h depends on the warp alone
            const float sv = seen ? s[u] : -INFINITY;
            const float m_new = fmaxf(m[u], warp_max(sv));
            const float pexp = seen ? expf(sv - m_new) : 0.0f;
            const float corr = expf(m[u] - m_new);         // m = -inf on the first block: corr = 0, l and acc are 0
            l[u] = l[u] * corr + warp_sum(pexp);
#pragma unroll
            for (int i = 0; i < MAX_DV / 32; ++i) acc[u][i] *= corr;
            const TKV* vrow = seen ? v_base + (size_t)page * page_stride + ((size_t)(h / group) * page_size + off) * DV : nullptr;
            for (int j = 0; j < n; ++j) {
                const float pj = __shfl_sync(0xffffffffu, pexp, j);
                const unsigned long long vp = __shfl_sync(0xffffffffu, (unsigned long long)vrow, j);
                const TKV* vj = (const TKV*)vp;
#pragma unroll
                for (int i = 0; i < MAX_DV / 32; ++i) {
                    const int d = lane + 32 * i;
                    if (d < DV) acc[u][i] += pj * to_float<TKV>(vj[d]);
                }
            }
            m[u] = m_new;
        }
        if (talk) __syncthreads();                     // the scores are read before the next block overwrites them
    }
#pragma unroll
    for (int u = 0; u < HPW; ++u) {
        const int h = warp + u * warps;
        if (h >= HQ) continue;
        if (sink) {
            const float sk = sink[h], top = fmaxf(m[u], sk), corr = expf(m[u] - top);
            l[u] = l[u] * corr + expf(sk - top);
#pragma unroll
            for (int i = 0; i < MAX_DV / 32; ++i) acc[u][i] *= corr;
        }
        TO* o = out + ((size_t)t * HQ + h) * DV;
        const TG* gr = gate ? gate + (size_t)t * gate_stride + (size_t)h * DV : nullptr;
        const float inv = 1.0f / l[u];
#pragma unroll
        for (int i = 0; i < MAX_DV / 32; ++i) {
            const int d = lane + 32 * i;
            if (d < DV) {
                float v = acc[u][i] * inv;
                if (gr) v *= 1.0f / (1.0f + expf(-to_float<TG>(gr[d])));
                o[d] = from_float<TO>(v);
            }
        }
    }
}

// What may happen to a row beside the norms: a factor per token that the norm in front left out (sumsq, see RowScale), a bias
// [QW + KW + VW] added behind it, a rotation of the first n_rot dimensions of every q and k head (table [max_pos, n_rot]:
// cosines, then sines, one per pair; halves or neighbours), and the gate's logits behind v, gate_width of them, added up and
// stored in q's dtype (gate_out).  All optional.
struct RowExtras {
    const float* bias = nullptr;
    const float* table = nullptr; int n_rot = 0, max_pos = 0, interleaved = 0;
    const int32_t* positions = nullptr;
    const float* sumsq = nullptr; int chunks = 0, width = 0; float eps = 0.0f;
    void* gate_out = nullptr; int gate_width = 0;
};
__device__ __forceinline__ float row_factor(const RowExtras& x, int t) {
    if (!x.sumsq) return 1.0f;
    float s = 0.0f;
    for (int k = 0; k < x.chunks; ++k) s += x.sumsq[(size_t)t * x.chunks + k];
    return rsqrtf(s / (float)x.width + x.eps);
}
// Element d of a head at `head` (raw values, with factor inv and the weights at w, or none), rotated.
__device__ __forceinline__ float rotated(const RowExtras& x, const float* turn, const float* head, const float* w, float inv, int d) {
    auto at = [&](int e) { return w ? head[e] * inv * w[e] : head[e]; };
    const float own = at(d);
    if (!turn || d >= x.n_rot) return own;
    const int half = x.n_rot / 2;
    int pair; bool second; float other;
    if (x.interleaved) { pair = d >> 1; second = d & 1; other = at(d ^ 1); }
    else { second = d >= half; pair = second ? d - half : d; other = at(second ? d - half : d + half); }
    const float c = turn[pair], s = turn[half + pair];
    return second ? __fmaf_rn(other, s, __fmul_rn(own, c)) : __fmaf_rn(own, c, -__fmul_rn(other, s));
}
__device__ __forceinline__ const float* turn_of(const RowExtras& x, int t) {
    if (!x.table) return nullptr;
    int pos = x.positions[t];
    pos = pos < 0 ? 0 : pos < x.max_pos ? pos : x.max_pos - 1;
    return x.table + (size_t)pos * x.n_rot;
}

// The gate's logits, at `first` in the row: added up, scaled and stored.
template <typename TI, typename TQ>
__device__ __forceinline__ void finish_gate(const RowExtras& x, const TI* src, int splits, long long split_stride, int first, float factor, int t) {
    if (!x.gate_out) return;
    TQ* to = static_cast<TQ*>(x.gate_out) + (size_t)t * x.gate_width;
    for (int i = threadIdx.x; i < x.gate_width; i += blockDim.x) {
        float v = 0.0f;
        for (int s = 0; s < splits; ++s) v += to_float<TI>(src[(size_t)s * split_stride + first + i]);
        to[i] = from_float<TQ>(v * factor);
    }
}

// One block per token.  The row holds [q (QW) | k (KW) | v (VW, or nothing when the keys are the values) | gate | ...].
template <typename TI, typename TQ, typename TKV>
__global__ void joint_norm_kv_write_kernel(const TI* __restrict__ rows, int splits, long long split_stride, long long row_width,
                                           const float* __restrict__ q_w, const float* __restrict__ k_w, float eps,
                                           const int32_t* __restrict__ slot_mapping, TQ* __restrict__ q_out, TKV* __restrict__ k_base,
                                           TKV* __restrict__ v_base, long long page_stride, int page_size, int HQ, int HKV, int D, int DV,
                                           int v_from_row, const RowExtras x) {
    extern __shared__ float buf[];             // [QW + KW]
    __shared__ float scratch[32];
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    const int QW = HQ * D, KW = HKV * D;
    const TI* src = rows + (size_t)t * row_width;
    const float factor = row_factor(x, t);
    const float* turn = turn_of(x, t);
    float sq = 0.0f, sk = 0.0f;
    for (int i = threadIdx.x; i < QW + KW; i += blockDim.x) {
        float v = 0.0f;
        for (int s = 0; s < splits; ++s) v += to_float<TI>(src[(size_t)s * split_stride + i]);
        v *= factor;
        if (x.bias) v += x.bias[i];
        buf[i] = v;
        if (i < QW) sq += v * v; else sk += v * v;
    }
    const float iq = q_w ? rsqrtf(block_sum_any(sq, scratch) / (float)QW + eps) : 1.0f;
    const float ik = k_w ? rsqrtf(block_sum_any(sk, scratch) / (float)KW + eps) : 1.0f;
    __syncthreads();
    TQ* qo = q_out + (size_t)t * QW;
    for (int i = threadIdx.x; i < QW; i += blockDim.x) {
        const int h0 = i / D * D;
        qo[i] = from_float<TQ>(rotated(x, turn, buf + h0, q_w ? q_w + h0 : nullptr, iq, i - h0));
    }
    finish_gate<TI, TQ>(x, src, splits, split_stride, QW + KW + (v_from_row ? HKV * DV : 0), factor, t);
    if (!slot_mapping) return;
    const int slot = slot_mapping[t];
    if (slot < 0) return;
    const size_t page_at = (size_t)(slot / page_size) * page_stride;
    const int off = slot % page_size;
    for (int i = threadIdx.x; i < KW; i += blockDim.x) {
        const int h = i / D, d = i % D;
        const float raw = buf[QW + i];
        k_base[page_at + ((size_t)h * page_size + off) * D + d] =
            from_float<TKV>(rotated(x, turn, buf + QW + h * D, k_w ? k_w + h * D : nullptr, ik, d));
        if (!v_from_row) v_base[page_at + ((size_t)h * page_size + off) * DV + d] = from_float<TKV>(raw);
    }
    if (v_from_row) {
        for (int i = threadIdx.x; i < HKV * DV; i += blockDim.x) {
            const int h = i / DV, d = i % DV;
            float v = 0.0f;
            for (int s = 0; s < splits; ++s) v += to_float<TI>(src[(size_t)s * split_stride + QW + KW + i]);
            v *= factor;
            if (x.bias) v += x.bias[QW + KW + i];
            v_base[page_at + ((size_t)h * page_size + off) * DV + d] = from_float<TKV>(v);
        }
    }
}

// The same with eight consecutive elements per access (every width a multiple of 8, rows 16-byte aligned): a thread's
// elements never straddle a head.  The sums of squares are taken per thread over its own elements, then over the block:
// their order depends on the widths alone.
template <typename TI, typename TQ, typename TKV>
__global__ void joint_norm_kv_write_vec_kernel(const TI* __restrict__ rows, int splits, long long split_stride, long long row_width,
                                               const float* __restrict__ q_w, const float* __restrict__ k_w, float eps,
                                               const int32_t* __restrict__ slot_mapping, TQ* __restrict__ q_out, TKV* __restrict__ k_base,
                                               TKV* __restrict__ v_base, long long page_stride, int page_size, int HQ, int HKV, int D, int DV,
                                               int v_from_row) {
    extern __shared__ float buf[];             // [QW + KW]
    __shared__ float scratch[32];
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    const int QW = HQ * D, KW = HKV * D;
    const TI* src = rows + (size_t)t * row_width;
    float sq = 0.0f, sk = 0.0f;
    for (int i = threadIdx.x * 8; i < QW + KW; i += blockDim.x * 8) {
        float v[8] = {0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f};
        for (int s = 0; s < splits; ++s) {
            float u[8];
            load8(src + (size_t)s * split_stride + i, u);
#pragma unroll
            for (int j = 0; j < 8; ++j) v[j] += u[j];
        }
        float ss = 0.0f;
#pragma unroll
        for (int j = 0; j < 8; ++j) { buf[i + j] = v[j]; ss += v[j] * v[j]; }
        if (i < QW) sq += ss; else sk += ss;
    }
    const float iq = q_w ? rsqrtf(block_sum_any(sq, scratch) / (float)QW + eps) : 1.0f;
    const float ik = k_w ? rsqrtf(block_sum_any(sk, scratch) / (float)KW + eps) : 1.0f;
    __syncthreads();
    TQ* qo = q_out + (size_t)t * QW;
    for (int i = threadIdx.x * 8; i < QW; i += blockDim.x * 8) {
        float v[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] = q_w ? buf[i + j] * iq * q_w[i + j] : buf[i + j];
        store8(qo + i, v);
    }
    if (!slot_mapping) return;
    const int slot = slot_mapping[t];
    if (slot < 0) return;
    const size_t page_at = (size_t)(slot / page_size) * page_stride;
    const int off = slot % page_size;
    for (int i = threadIdx.x * 8; i < KW; i += blockDim.x * 8) {
        const int h = i / D, d = i % D;
        float raw[8], v[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) { raw[j] = buf[QW + i + j]; v[j] = k_w ? raw[j] * ik * k_w[i + j] : raw[j]; }
        store8(k_base + page_at + ((size_t)h * page_size + off) * D + d, v);
        if (!v_from_row) store8(v_base + page_at + ((size_t)h * page_size + off) * DV + d, raw);
    }
    if (v_from_row) {
        for (int i = threadIdx.x * 8; i < HKV * DV; i += blockDim.x * 8) {
            const int h = i / DV, d = i % DV;
            float v[8] = {0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f};
            for (int s = 0; s < splits; ++s) {
                float u[8];
                load8(src + (size_t)s * split_stride + QW + KW + i, u);
#pragma unroll
                for (int j = 0; j < 8; ++j) v[j] += u[j];
            }
            store8(v_base + page_at + ((size_t)h * page_size + off) * DV + d, v);
        }
    }
}

// The form with extras, eight consecutive elements per access in registers.  Two blocks per token: one norms, rotates and
// stores q and k, the other stores v and the gate.  A thread has IT runs of eight elements; weights are on their way before the
// kernel in front is done.
template <typename TI>
__device__ __forceinline__ void sum8(const TI* src, int splits, long long split_stride, float factor, float* v) {
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = 0.0f;
#pragma unroll 4
    for (int s = 0; s < splits; ++s) {
        float u[8];
        load8(src + (size_t)s * split_stride, u);
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] += u[j];
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] *= factor;
}
template <typename TI, typename TQ, typename TKV, int IT>
__global__ void joint_norm_rope_vec_kernel(const TI* __restrict__ rows, int splits, long long split_stride, long long row_width,
                                           const float* __restrict__ q_w, const float* __restrict__ k_w, float eps,
                                           const int32_t* __restrict__ slot_mapping, TQ* __restrict__ q_out, TKV* __restrict__ k_base,
                                           TKV* __restrict__ v_base, long long page_stride, int page_size, int HQ, int HKV, int D, int DV,
                                           const RowExtras x) {
    extern __shared__ float buf[];             // [QW + KW] where pairs are halves of a head apart
    __shared__ float2 scratch[32];
    pdl_launch_dependents();
    const int t = blockIdx.x, QW = HQ * D, KW = HKV * D, VW = HKV * DV, step = blockDim.x * 8;
    const TI* src = rows + (size_t)t * row_width;
    if (blockIdx.y == 1) {
        pdl_wait();
        const float factor = row_factor(x, t);
        const int slot = slot_mapping ? slot_mapping[t] : -1;
        const size_t page_at = slot >= 0 ? (size_t)(slot / page_size) * page_stride : 0;
        const int off = slot >= 0 ? slot % page_size : 0, all = VW + (x.gate_out ? x.gate_width : 0);
        for (int i = threadIdx.x * 8; i < all; i += step) {
            float v[8];
            sum8(src + QW + KW + i, splits, split_stride, factor, v);
            if (i >= VW) { store8(static_cast<TQ*>(x.gate_out) + (size_t)t * x.gate_width + (i - VW), v); continue; }
            if (slot < 0) continue;
            if (x.bias) {
                float b[8];
                load8(x.bias + QW + KW + i, b);
#pragma unroll
                for (int j = 0; j < 8; ++j) v[j] += b[j];
            }
            const int h = i / DV, d = i - h * DV;
            store8(v_base + page_at + ((size_t)h * page_size + off) * DV + d, v);
        }
        return;
    }
    float v[IT][8], w[IT][8];
#pragma unroll
    for (int it = 0; it < IT; ++it) {
        const int i = threadIdx.x * 8 + it * step;
#pragma unroll
        for (int j = 0; j < 8; ++j) w[it][j] = 1.0f;
        const float* from = i < QW ? (q_w ? q_w + i : nullptr) : i < QW + KW ? (k_w ? k_w + (i - QW) : nullptr) : nullptr;
        if (from) load8(from, w[it]);
    }
    pdl_wait();
    const float factor = row_factor(x, t);
    const float* turn = turn_of(x, t);
    const int slot = slot_mapping ? slot_mapping[t] : -1;
    float2 ss = make_float2(0.0f, 0.0f);
#pragma unroll
    for (int it = 0; it < IT; ++it) {
        const int i = threadIdx.x * 8 + it * step;
        if (i >= QW + KW) continue;
        sum8(src + i, splits, split_stride, factor, v[it]);
        if (x.bias) {
            float b[8];
            load8(x.bias + i, b);
#pragma unroll
            for (int j = 0; j < 8; ++j) v[it][j] += b[j];
        }
        float s8 = 0.0f;
#pragma unroll
        for (int j = 0; j < 8; ++j) s8 += v[it][j] * v[it][j];
        if (i < QW) ss.x += s8; else ss.y += s8;
    }
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    ss.x = warp_sum(ss.x); ss.y = warp_sum(ss.y);
    if (lane == 0) scratch[warp] = ss;
    __syncthreads();
    ss = lane < warps ? scratch[lane] : make_float2(0.0f, 0.0f);
    const float iq = q_w ? rsqrtf(warp_sum(ss.x) / (float)QW + eps) : 1.0f, ik = k_w ? rsqrtf(warp_sum(ss.y) / (float)KW + eps) : 1.0f;
    const int half = x.n_rot / 2;
    const bool apart = turn && !x.interleaved;
#pragma unroll
    for (int it = 0; it < IT; ++it) {
        const int i = threadIdx.x * 8 + it * step;
        if (i >= QW + KW) continue;
        const float inv = i < QW ? iq : ik;
#pragma unroll
        for (int j = 0; j < 8; ++j) v[it][j] = v[it][j] * inv * w[it][j];
        if (apart) store8(buf + i, v[it]);
    }
    if (apart) __syncthreads();
    const size_t page_at = slot >= 0 ? (size_t)(slot / page_size) * page_stride : 0;
    const int off = slot >= 0 ? slot % page_size : 0;
#pragma unroll
    for (int it = 0; it < IT; ++it) {
        const int i = threadIdx.x * 8 + it * step;
        if (i >= QW + KW) continue;
        const int head = i / D, d = i - head * D;
        if (turn && d < x.n_rot) {
            if (x.interleaved) {
                const float4 c = load4(turn + d / 2), s = load4(turn + half + d / 2);
                const float cc[4] = {c.x, c.y, c.z, c.w}, sn[4] = {s.x, s.y, s.z, s.w};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const float a = v[it][2 * e], b = v[it][2 * e + 1];
                    v[it][2 * e] = __fmaf_rn(a, cc[e], -__fmul_rn(b, sn[e]));
                    v[it][2 * e + 1] = __fmaf_rn(a, sn[e], __fmul_rn(b, cc[e]));
                }
            } else {
                const bool second = d >= half;
                float c[8], s[8], other[8];
                load8(turn + (second ? d - half : d), c);
                load8(turn + half + (second ? d - half : d), s);
                load8(buf + (second ? i - half : i + half), other);
#pragma unroll
                for (int j = 0; j < 8; ++j)
                    v[it][j] = second ? __fmaf_rn(other[j], s[j], __fmul_rn(v[it][j], c[j])) : __fmaf_rn(v[it][j], c[j], -__fmul_rn(other[j], s[j]));
            }
        }
        if (i < QW) store8(q_out + (size_t)t * QW + i, v[it]);
        else if (slot >= 0) store8(k_base + page_at + ((size_t)(head - HQ) * page_size + off) * D + d, v[it]);
    }
}

}  // namespace

// gate: rows of HQ * DV logits, gate_stride elements apart, in gate_dtype (null: no gate).  cap 0: no cap.  r1 without r2: a
// bias linear in the distance.  r1, r2, talk, sink: float32 per head ([HQ], [HQ], [HQ, HQ], [HQ]) or null.
PH_EXPORT int ph_attention_talking(const void* q, int q_dtype, const void* k_base, const void* v_base, int kv_dtype, long long page_stride,
                                   int page_size, const int32_t* block_table, int table_stride, const int32_t* row_seg,
                                   const int32_t* positions, void* out, int out_dtype, int T, int HQ, int HKV, int D, int DV, int window,
                                   int chunk, float scale, float cap, const float* r1, const float* r2, const float* talk,
                                   const float* sink, const void* gate, int gate_dtype, long long gate_stride, cudaStream_t stream) {
    if (!q || !k_base || !v_base || !block_table || !row_seg || !positions || !out || T < 0 || HQ < 1 || HKV < 1 || D < 1 || DV < 1 ||
        page_size < 1 || window < 0 || chunk < 0 || !valid_dtype(q_dtype) || !valid_dtype(kv_dtype) || !valid_dtype(out_dtype) ||
        (gate && !valid_dtype(gate_dtype)) || (r2 && !r1) || cap < 0.0f)
        return fail(PH_ERR_ARG, "attention_talking: bad arguments (T %d, HQ %d, HKV %d, D %d, DV %d)", T, HQ, HKV, D, DV);
    if (HQ % HKV) return fail(PH_ERR_ARG, "attention_talking: %d query heads are not a multiple of %d kv heads", HQ, HKV);
    if (HQ > MAX_HEADS) return fail(PH_ERR_UNSUPPORTED, "attention_talking: %d heads exceed the supported %d", HQ, MAX_HEADS);
    if (DV > MAX_DV) return fail(PH_ERR_UNSUPPORTED, "attention_talking: value rows of %d exceed the supported %d", DV, MAX_DV);
    const size_t smem = ((size_t)HQ * D + (size_t)HQ * 32 + (size_t)HQ * HQ) * sizeof(float);
    if (smem > 200 * 1024) return fail(PH_ERR_UNSUPPORTED, "attention_talking: %d heads of %d do not fit shared memory", HQ, D);
    if (T == 0) return PH_OK;
    if (!gate) gate_dtype = q_dtype;
    // (two heads per warp take 94 registers a thread and four take 127: 20 and 16 warps are what an SM's registers hold)
    const int hpw = HQ <= 32 ? 1 : HQ <= 40 ? 2 : 4, warps = (HQ + hpw - 1) / hpw;
#define LAUNCH_N(TQ, TKV, TG, TO, N)                                                                                              \
    do {                                                                                                                          \
        auto kern = attention_talking_kernel<TQ, TKV, TG, TO, N>;                                                                 \
        if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                 \
        kern<<<T, warps * 32, smem, stream>>>((const TQ*)q, (const TKV*)k_base, (const TKV*)v_base, page_stride, page_size, block_table, \
                                              table_stride, row_seg, positions, (TO*)out, HQ, HKV, D, DV, window, chunk, scale, cap, \
                                              r1, r2, talk, sink, (const TG*)gate, gate_stride);                                  \
    } while (0)
#define LAUNCH(TQ, TKV, TG, TO)                                                                                                   \
    do {                                                                                                                          \
        if (hpw == 1) LAUNCH_N(TQ, TKV, TG, TO, 1); else if (hpw == 2) LAUNCH_N(TQ, TKV, TG, TO, 2); else LAUNCH_N(TQ, TKV, TG, TO, 4); \
    } while (0)
    PH_DISPATCH(q_dtype, TQ, PH_DISPATCH(kv_dtype, TKV, PH_DISPATCH(gate_dtype, TG, PH_DISPATCH(out_dtype, TO, LAUNCH(TQ, TKV, TG, TO)))));
#undef LAUNCH
#undef LAUNCH_N
    return check_launch("attention_talking");
}

// rows: [splits][T][row_width] in rows_dtype.  q_w [HQ * D] and k_w [HKV * D] float32 or null.  slot_mapping null: no
// cache write (q only).  v_from_row 0: the values are the keys as projected; 1: the row's third part [HKV * DV].
static int joint_norm(const void* rows, int rows_dtype, int splits, long long split_stride, long long row_width,
                                     const float* q_w, const float* k_w, float eps, const int32_t* slot_mapping, void* q_out, int q_dtype,
                                     void* k_base, void* v_base, int kv_dtype, long long page_stride, int page_size, int T, int HQ,
                                     int HKV, int D, int DV, int v_from_row, const RowExtras& x, cudaStream_t stream) {
    if (!rows || !q_out || T < 0 || HQ < 1 || HKV < 1 || D < 1 || DV < 1 || splits < 1 || page_size < 1 || !valid_dtype(rows_dtype) ||
        !valid_dtype(q_dtype) || !valid_dtype(kv_dtype) || (slot_mapping && (!k_base || !v_base)))
        return fail(PH_ERR_ARG, "joint_norm_kv_write: bad arguments (T %d, HQ %d, HKV %d, D %d)", T, HQ, HKV, D);
    if (!v_from_row && DV != D) return fail(PH_ERR_ARG, "joint_norm_kv_write: values that are the keys are as wide as the keys (%d, not %d)", D, DV);
    const long long need = (long long)(HQ + HKV) * D + (v_from_row ? (long long)HKV * DV : 0) + (x.gate_out ? x.gate_width : 0);
    if (row_width < need) return fail(PH_ERR_ARG, "joint_norm_kv_write: rows of %lld elements hold no %lld", row_width, need);
    const size_t smem = (size_t)(HQ + HKV) * D * sizeof(float);
    if (smem > 200 * 1024) return fail(PH_ERR_UNSUPPORTED, "joint_norm_kv_write: rows of %d elements do not fit shared memory", (HQ + HKV) * D);
    if (T == 0) return PH_OK;
    const int threads = (HQ + HKV) * D >= 2048 ? 512 : 256;
    const bool vec = D % 8 == 0 && DV % 8 == 0 && row_width % 8 == 0 && split_stride % 8 == 0 && page_stride % 8 == 0 &&
                     (((uintptr_t)rows | (uintptr_t)q_out | (uintptr_t)k_base | (uintptr_t)v_base) % 32) == 0;
    const bool plain = !x.bias && !x.table && !x.sumsq && !x.gate_out;
    const bool turns_ok = !x.table || (((uintptr_t)x.table & 15) == 0 && (x.interleaved ? x.n_rot % 8 == 0 : x.n_rot % 16 == 0));
    const int runs = (HQ + HKV) * D / 8;
    if (vec && !plain && v_from_row && turns_ok && runs <= 4 * 512 && (!x.gate_out || (x.gate_width % 8 == 0 && ((uintptr_t)x.gate_out & 15) == 0)) &&
        (((uintptr_t)q_w | (uintptr_t)k_w | (uintptr_t)x.bias) & 15) == 0) {
        const int it = runs <= 512 ? 1 : runs <= 1024 ? 2 : 4, threads_x = ((runs + it - 1) / it + 31) / 32 * 32;
        const size_t bytes = x.table && !x.interleaved ? smem : 0;
#define LAUNCH_X(TI, TQ, TKV, N)                                                                                                   \
    do {                                                                                                                           \
        auto kern = joint_norm_rope_vec_kernel<TI, TQ, TKV, N>;                                                                    \
        if (bytes > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);                \
        launch_overlapped(kern, dim3(T, 2), dim3(threads_x), bytes, stream, (const TI*)rows, splits, split_stride, row_width, q_w, k_w, eps, \
                          slot_mapping, (TQ*)q_out, (TKV*)k_base, (TKV*)v_base, page_stride, page_size, HQ, HKV, D, DV, x);         \
    } while (0)
#define LAUNCH_X_ALL(TI, TQ, TKV)                                                                                                  \
    do {                                                                                                                           \
        if (it == 1) LAUNCH_X(TI, TQ, TKV, 1); else if (it == 2) LAUNCH_X(TI, TQ, TKV, 2); else LAUNCH_X(TI, TQ, TKV, 4);           \
    } while (0)
        PH_DISPATCH(rows_dtype, TI, PH_DISPATCH(q_dtype, TQ, PH_DISPATCH(kv_dtype, TKV, LAUNCH_X_ALL(TI, TQ, TKV))));
#undef LAUNCH_X_ALL
#undef LAUNCH_X
        return check_launch("joint_norm_rope_kv_write");
    }
    if (vec && plain) {
        const int vthreads = (HQ + HKV) * D / 8 >= 256 ? 256 : 128;
#define LAUNCH_VEC(TI, TQ, TKV)                                                                                                    \
    do {                                                                                                                           \
        auto kern = joint_norm_kv_write_vec_kernel<TI, TQ, TKV>;                                                                   \
        if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                  \
        launch_overlapped(kern, dim3(T), dim3(vthreads), smem, stream, (const TI*)rows, splits, split_stride, row_width, q_w, k_w, eps, slot_mapping, (TQ*)q_out, \
                                            (TKV*)k_base, (TKV*)v_base, page_stride, page_size, HQ, HKV, D, DV, v_from_row);       \
    } while (0)
        PH_DISPATCH(rows_dtype, TI, PH_DISPATCH(q_dtype, TQ, PH_DISPATCH(kv_dtype, TKV, LAUNCH_VEC(TI, TQ, TKV))));
#undef LAUNCH_VEC
        return check_launch("joint_norm_kv_write");
    }
#define LAUNCH(TI, TQ, TKV)                                                                                                        \
    do {                                                                                                                           \
        auto kern = joint_norm_kv_write_kernel<TI, TQ, TKV>;                                                                       \
        if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                  \
        launch_overlapped(kern, dim3(T), dim3(threads), smem, stream, (const TI*)rows, splits, split_stride, row_width, q_w, k_w, eps, slot_mapping, (TQ*)q_out, \
                                           (TKV*)k_base, (TKV*)v_base, page_stride, page_size, HQ, HKV, D, DV, v_from_row, x);        \
    } while (0)
    PH_DISPATCH(rows_dtype, TI, PH_DISPATCH(q_dtype, TQ, PH_DISPATCH(kv_dtype, TKV, LAUNCH(TI, TQ, TKV))));
#undef LAUNCH
    return check_launch("joint_norm_kv_write");
}

PH_EXPORT int ph_joint_norm_kv_write(const void* rows, int rows_dtype, int splits, long long split_stride, long long row_width,
                                     const float* q_w, const float* k_w, float eps, const int32_t* slot_mapping, void* q_out, int q_dtype,
                                     void* k_base, void* v_base, int kv_dtype, long long page_stride, int page_size, int T, int HQ,
                                     int HKV, int D, int DV, int v_from_row, cudaStream_t stream) {
    return joint_norm(rows, rows_dtype, splits, split_stride, row_width, q_w, k_w, eps, slot_mapping, q_out, q_dtype, k_base, v_base, kv_dtype,
                      page_stride, page_size, T, HQ, HKV, D, DV, v_from_row, RowExtras(), stream);
}

// The same for rows [q | k | v | (gate)] with a bias, a rotation, a row's missing factor and the gate's logits (RowExtras says
// what each is; null: without it).
PH_EXPORT int ph_joint_norm_rope_kv_write(const void* rows, int rows_dtype, int splits, long long split_stride, long long row_width,
                                          const float* q_w, const float* k_w, float eps, const int32_t* slot_mapping, void* q_out, int q_dtype,
                                          void* k_base, void* v_base, int kv_dtype, long long page_stride, int page_size, int T, int HQ,
                                          int HKV, int D, int DV, const float* bias, const float* cos_sin, int n_rot, int max_pos,
                                          const int32_t* positions, int interleaved, const float* row_sumsq, int row_chunks, int row_dim,
                                          float row_eps, void* gate_out, int gate_width, cudaStream_t stream) {
    if (cos_sin && (n_rot < 2 || n_rot % 2 || n_rot > D || max_pos < 1 || !positions))
        return fail(PH_ERR_ARG, "joint_norm_rope_kv_write: %d of %d dimensions cannot be rotated", n_rot, D);
    if ((row_sumsq && (row_chunks < 1 || row_dim < 1)) || (gate_out && gate_width < 1))
        return fail(PH_ERR_ARG, "joint_norm_rope_kv_write: bad arguments");
    RowExtras x;
    x.bias = bias; x.table = cos_sin; x.n_rot = n_rot; x.max_pos = max_pos; x.interleaved = interleaved; x.positions = positions;
    x.sumsq = row_sumsq; x.chunks = row_chunks; x.width = row_dim; x.eps = row_eps; x.gate_out = gate_out; x.gate_width = gate_width;
    return joint_norm(rows, rows_dtype, splits, split_stride, row_width, q_w, k_w, eps, slot_mapping, q_out, q_dtype, k_base, v_base, kv_dtype,
                      page_stride, page_size, T, HQ, HKV, D, DV, 1, x, stream);
}
