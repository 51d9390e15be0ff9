// The kernels of a state-space mixer of Mamba's second form that are neither matrix products nor the short convolution
// (causal_conv_silu in mamba.cu): the recurrence, two ways, and the gated norm behind it.
//
// Per head h (group g = h / (H / G)), with x_t [P], B_t and C_t [N] of the convolution's output and dt_t =
// softplus(logit_t + bias_h):
//     S_t = exp(a_h dt_t) S_(t-1) + dt_t B_t x_t^T          (a_h < 0; S is N x P)
//     y_t = S_t^T C_t + d_h x_t
// S is float32, lives in the request's state slot as [H][P][N] and is carried from token to token; the last K - 1 inputs of
// the convolution stand behind it, and the recurrence's kernels move those on when they are done with a request's rows.
//
//   ssd_scan    token by token: a group of lanes holds four rows (p) of S, N spread over the lanes; a token costs a
//               multiply-add per state element and a butterfly per row.  Decoding, short portions, float32.
//   ssd_chunk   chunks of 64 tokens on the tensor cores (bfloat16 in, float32 sums), a block per (request, head, 32 of its P
//               columns) that walks the request's chunks in order.  Four of its warps make the chunk's outputs while the four
//               others fetch the next chunk, work out its step sizes and carry S, which they hold in registers, over the
//               current one.  With cum_i the sum of a dt over the
//               chunk's tokens up to i:
//                   y_i = sum_(j <= i) (C_i . B_j) exp(cum_i - cum_j) dt_j x_j + exp(cum_i) C_i^T S + d x_i
//                   S   = exp(cum_last) S + sum_j exp(cum_last - cum_j) dt_j B_j x_j^T
//               B, C and x are exact in bfloat16; every float32 factor that meets them in a product (the weights of the
//               first sum with the decays in them, S, the weighted x) is split into a bfloat16 and the bfloat16 of what is
//               left, two products, so that decays, step sizes and the state keep 16 bits through the tensor cores and
//               float32 everywhere else.  Rows beyond a request's last token have a step size of zero.
//   gate_rms    y * silu(z), then an RMS norm in equal parts, each by its own root mean square, times a weight.
#include "attention_mma.cuh"

#include <math.h>

namespace {

using namespace ph;
using namespace ph_attn;

__device__ __forceinline__ float softplus(float v) { return log1pf(expf(-fabsf(v))) + fmaxf(v, 0.0f); }
__device__ __forceinline__ float silu(float v) { return v / (1.0f + expf(-v)); }

struct SsdParams {
    const void* xbc;                                  // [T, H * P + 2 * G * N]: x | B | C behind convolution and silu
    const void* in; long long in_stride;              // [T, in_stride]: the in-projection's rows
    int dt_col, conv_col;                             // where the step's logits and the convolution's inputs start there
    const float* dt_bias; const float* a; const float* d;      // [H]
    float* state; long long state_stride;
    const int32_t* seg_start; const int32_t* seg_slot;
    float* y;                                         // [T, H * P]
    int H, P, N, G, K;
    int rows_from, rows_to;                           // this launch takes the requests whose portion has rows_from .. rows_to rows
};

// The last K - 1 inputs of the convolution, oldest first: from this step's rows, or moved up from what was kept.  The
// channels are spread over the `blocks` groups of `threads` threads that work on a request.
template <typename TX>
__device__ __forceinline__ void move_conv_inputs(const SsdParams& p, float* st, int row0, int n, int block, int blocks, int thread, int threads) {
    const int CH = p.H * p.P + 2 * p.G * p.N;
    float* past = st + (size_t)p.H * p.P * p.N;
    const TX* src = static_cast<const TX*>(p.in) + p.conv_col;
    for (int c = block * threads + thread; c < CH; c += blocks * threads)
        for (int k = 0; k < p.K - 1; ++k) {
            const int i = n - (p.K - 1) + k;
            past[(size_t)k * CH + c] = i >= 0 ? to_float<TX>(src[(size_t)(row0 + i) * p.in_stride + c]) : past[(size_t)(k + n) * CH + c];
        }
}

// V consecutive elements of a row as floats
template <int V, typename T> __device__ __forceinline__ void load_v(const T* p, float* v) {
    if constexpr (V == 4) { const float4 u = load4(p); v[0] = u.x; v[1] = u.y; v[2] = u.z; v[3] = u.w; }
    else v[0] = to_float<T>(*p);
}

constexpr int SCAN_THREADS = 128, SCAN_ROWS = 4;

// L lanes per group of SCAN_ROWS rows; lane l holds the states n = (i * L + l) * V .. + V - 1 of each, i < NI.
template <typename TX, int NI, int V>
__global__ void __launch_bounds__(SCAN_THREADS) ssd_scan_kernel(const SsdParams p, int L) {
    pdl_launch_dependents();
    const int seg = blockIdx.z, h = blockIdx.y;
    const int row0 = p.seg_start[seg], n_rows = p.seg_start[seg + 1] - row0;
    const float bias = p.dt_bias[h], a = p.a[h], skip = p.d[h];
    if (n_rows < p.rows_from || n_rows > p.rows_to) { pdl_wait(); return; }
    const int lane = threadIdx.x % L, group = threadIdx.x / L;
    const int P = p.P, N = p.N, inner = p.H * P, CH = inner + 2 * p.G * N;
    const int p0 = (blockIdx.x * (SCAN_THREADS / L) + group) * SCAN_ROWS;
    const int g = h / (p.H / p.G);
    float* st = p.state + (size_t)p.seg_slot[seg] * p.state_stride;
    float* S0 = st + (size_t)h * P * N;
    pdl_wait();
    float S[SCAN_ROWS][NI * V];
#pragma unroll
    for (int r = 0; r < SCAN_ROWS; ++r)
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const int n = (i * L + lane) * V;
#pragma unroll
            for (int j = 0; j < V; ++j) S[r][i * V + j] = 0.0f;
            if (p0 + r < P && n < N) load_v<V>(S0 + (size_t)(p0 + r) * N + n, &S[r][i * V]);
        }
    const TX* xbc = static_cast<const TX*>(p.xbc) + (size_t)row0 * CH;
    const TX* dt_in = static_cast<const TX*>(p.in) + (size_t)row0 * p.in_stride + p.dt_col + h;
    for (int t = 0; t < n_rows; ++t, xbc += CH, dt_in += p.in_stride) {
        float Bv[NI * V], Cv[NI * V], x[SCAN_ROWS];
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const int n = (i * L + lane) * V;
#pragma unroll
            for (int j = 0; j < V; ++j) Bv[i * V + j] = Cv[i * V + j] = 0.0f;
            if (n < N) {
                load_v<V>(xbc + inner + (size_t)g * N + n, &Bv[i * V]);
                load_v<V>(xbc + inner + (size_t)(p.G + g) * N + n, &Cv[i * V]);
            }
        }
#pragma unroll
        for (int r = 0; r < SCAN_ROWS; ++r) x[r] = p0 + r < P ? to_float<TX>(xbc[(size_t)h * P + p0 + r]) : 0.0f;
        const float dt = softplus(to_float<TX>(*dt_in) + bias), decay = expf(a * dt);
        float acc[SCAN_ROWS];
#pragma unroll
        for (int r = 0; r < SCAN_ROWS; ++r) {
            const float dx = dt * x[r];
            acc[r] = 0.0f;
#pragma unroll
            for (int i = 0; i < NI * V; ++i) {
                S[r][i] = fmaf(decay, S[r][i], dx * Bv[i]);
                acc[r] = fmaf(S[r][i], Cv[i], acc[r]);
            }
        }
#pragma unroll
        for (int r = 0; r < SCAN_ROWS; ++r)
            for (int o = L >> 1; o > 0; o >>= 1) acc[r] += __shfl_xor_sync(0xffffffffu, acc[r], o);
        if (lane == 0) {
            float* y = p.y + (size_t)(row0 + t) * inner + (size_t)h * P;
#pragma unroll
            for (int r = 0; r < SCAN_ROWS; ++r)
                if (p0 + r < P) y[p0 + r] = acc[r] + skip * x[r];
        }
    }
#pragma unroll
    for (int r = 0; r < SCAN_ROWS; ++r)
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const int n = (i * L + lane) * V;
            if (p0 + r >= P || n >= N) continue;
            if constexpr (V == 4) store4(S0 + (size_t)(p0 + r) * N + n, &S[r][i * V]);
            else S0[(size_t)(p0 + r) * N + n] = S[r][i];
        }
    move_conv_inputs<TX>(p, st, row0, n_rows, blockIdx.y * gridDim.x + blockIdx.x, gridDim.x * gridDim.y, threadIdx.x, SCAN_THREADS);
}

// ---- chunks on the tensor cores ------------------------------------------------------------------------------------
constexpr int CQ = 64;                 // tokens of a chunk
constexpr int CP = 32;                 // columns (p) of a block
constexpr int CWARPS = 4;              // warps 0 .. 3: outputs, 16 rows of the chunk each; warps 4 .. 7: the next chunk and S
constexpr int CTHREADS = 2 * CWARPS * 32;
constexpr int XPITCH = CP * 2 + 16;    // bytes of a row of the x tile

__host__ __device__ constexpr int ssd_pitch(int NP) { return NP * 2 + 16; }
// B, C and x of two chunks, S as two bfloat16 tiles, and (cum, dt, w) of two chunks
__host__ __device__ constexpr int ssd_smem(int NP) { return 4 * CQ * ssd_pitch(NP) + 2 * CQ * XPITCH + 2 * CP * ssd_pitch(NP) + 2 * 3 * CQ * 4; }

// v = hi + lo with both in bfloat16 (hi the rounded value, lo the rounded rest), two values at a time
__device__ __forceinline__ void split2(float u, float v, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16(u, v);
    lo = pack_bf16(u - __uint_as_float(hi << 16), v - __uint_as_float(hi & 0xffff0000u));
}

// NP: N rounded up to 16.  NTW: tiles of 16 states that a warp holds of S (tile w + 4 k).
template <int NTW>
__global__ void __launch_bounds__(CTHREADS, NTW <= 2 ? 2 : 1) ssd_chunk_kernel(const SsdParams p, int NP) {
    extern __shared__ __align__(128) uint8_t smem[];
    pdl_launch_dependents();
    const int seg = blockIdx.z, h = blockIdx.y, pt0 = blockIdx.x * CP;
    const int row0 = p.seg_start[seg], n_rows = p.seg_start[seg + 1] - row0;
    if (n_rows < p.rows_from || n_rows > p.rows_to) { pdl_wait(); return; }
    const int warp = (threadIdx.x >> 5) & (CWARPS - 1), lane = threadIdx.x & 31;
    const bool outputs = threadIdx.x < CWARPS * 32;
    const int P = p.P, N = p.N, inner = p.H * P, CH = inner + 2 * p.G * N;
    const int g = h / (p.H / p.G), pitch = ssd_pitch(NP), ntiles = NP / 16;
    const uint32_t b_tiles = smem_u32(smem), c_tiles = b_tiles + 2 * CQ * pitch, x_tiles = c_tiles + 2 * CQ * pitch;
    const uint32_t s_hi = x_tiles + 2 * CQ * XPITCH, s_lo = s_hi + CP * pitch;
    float* sums = reinterpret_cast<float*>(smem + (s_lo - b_tiles) + CP * pitch);      // [2][cum | dt | w][CQ]
    const int chunks = (n_rows + CQ - 1) / CQ;
    const int nc = (lane & 3) * 2;
    pdl_wait();

    if (outputs) {
        // ---- y of the rows 16 warp .. 16 warp + 15 of every chunk
        const float skip = p.d[h];
        const int r0 = warp * 16 + (lane >> 2), r1 = r0 + 8;
        float* y_out = p.y + (size_t)row0 * inner + (size_t)h * P;
        for (int c = 0; c < chunks; ++c) {
            const int buf = c & 1;
            const uint32_t bt = b_tiles + buf * CQ * pitch, ct = c_tiles + buf * CQ * pitch, xt = x_tiles + buf * CQ * XPITCH;
            const float* cum = sums + buf * 3 * CQ;
            const float* dts = cum + CQ;
            asm volatile("bar.sync 2, %0;" ::"n"(CTHREADS) : "memory");                             // the chunk, its sums and the S it starts from are there
            // C_i . B_j for this warp's rows and the keys up to their last, and C_i^T S
            float s[CQ / 8][4], y[CP / 8][4], rest[CP / 8][4];
#pragma unroll
            for (int nt = 0; nt < CQ / 8; ++nt)
#pragma unroll
                for (int i = 0; i < 4; ++i) s[nt][i] = 0.0f;
#pragma unroll
            for (int nt = 0; nt < CP / 8; ++nt)
#pragma unroll
                for (int i = 0; i < 4; ++i) y[nt][i] = rest[nt][i] = 0.0f;
            for (int ks = 0; ks < ntiles; ++ks) {
                uint32_t a0, a1, a2, a3;
                ldmatrix_x4(ct + (warp * 16 + (lane & 15)) * pitch + (ks * 2 + (lane >> 4)) * 16, a0, a1, a2, a3);
                const int col = (ks * 2 + ((lane >> 3) & 1)) * 16, row = (lane & 7) + ((lane >> 4) << 3);
#pragma unroll
                for (int nt = 0; nt < CP / 8; nt += 2) {
                    uint32_t b0, b1, b2, b3;
                    const int at = (nt * 8 + row) * pitch + col;
                    ldmatrix_x4(s_hi + at, b0, b1, b2, b3);
                    mma_bf16(y[nt], a0, a1, a2, a3, b0, b1);
                    mma_bf16(y[nt + 1], a0, a1, a2, a3, b2, b3);
                    ldmatrix_x4(s_lo + at, b0, b1, b2, b3);
                    mma_bf16(rest[nt], a0, a1, a2, a3, b0, b1);
                    mma_bf16(rest[nt + 1], a0, a1, a2, a3, b2, b3);
                }
#pragma unroll
                for (int nt = 0; nt < CQ / 8; nt += 2) {
                    if (nt > 2 * warp) continue;         // keys behind every row of this warp
                    uint32_t b0, b1, b2, b3;
                    ldmatrix_x4(bt + (nt * 8 + row) * pitch + col, b0, b1, b2, b3);
                    mma_bf16(s[nt], a0, a1, a2, a3, b0, b1);
                    mma_bf16(s[nt + 1], a0, a1, a2, a3, b2, b3);
                }
            }
            asm volatile("bar.arrive 1, %0;" ::"n"(CTHREADS) : "memory");      // S is read: it may be written for the next chunk
            const float cum0 = cum[r0], cum1 = cum[r1];
            const float e0 = __expf(cum0), e1 = __expf(cum1);
#pragma unroll
            for (int nt = 0; nt < CP / 8; ++nt) {
                y[nt][0] = (y[nt][0] + rest[nt][0]) * e0; y[nt][1] = (y[nt][1] + rest[nt][1]) * e0;
                y[nt][2] = (y[nt][2] + rest[nt][2]) * e1; y[nt][3] = (y[nt][3] + rest[nt][3]) * e1;
            }
            // the weights of the chunk's own tokens (the skip sits on the diagonal), times x
#pragma unroll
            for (int kt = 0; kt < CQ / 16; ++kt) {
                if (kt > warp) continue;
                uint32_t hi[4], lo[4];
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    const int nt = 2 * kt + half, j = nt * 8 + nc;
                    const float2 cj = *reinterpret_cast<const float2*>(cum + j), dj = *reinterpret_cast<const float2*>(dts + j);
                    float w[4] = {s[nt][0] * (__expf(cum0 - cj.x) * dj.x), s[nt][1] * (__expf(cum0 - cj.y) * dj.y),
                                  s[nt][2] * (__expf(cum1 - cj.x) * dj.x), s[nt][3] * (__expf(cum1 - cj.y) * dj.y)};
                    if (kt == warp) {                    // the tile on the diagonal
#pragma unroll
                        for (int i = 0; i < 4; ++i) {
                            const int row = i < 2 ? r0 : r1, key = j + (i & 1);
                            w[i] = key > row ? 0.0f : key == row ? w[i] + skip : w[i];
                        }
                    }
                    split2(w[0], w[1], hi[2 * half], lo[2 * half]);
                    split2(w[2], w[3], hi[2 * half + 1], lo[2 * half + 1]);
                }
                const int row = kt * 16 + (lane & 7) + (((lane >> 3) & 1) << 3);
#pragma unroll
                for (int nt = 0; nt < CP / 8; nt += 2) {
                    uint32_t b0, b1, b2, b3;
                    ldmatrix_x4_trans(xt + row * XPITCH + (nt + (lane >> 4)) * 16, b0, b1, b2, b3);
                    mma_bf16(y[nt], hi[0], hi[1], hi[2], hi[3], b0, b1);
                    mma_bf16(y[nt + 1], hi[0], hi[1], hi[2], hi[3], b2, b3);
                    mma_bf16(y[nt], lo[0], lo[1], lo[2], lo[3], b0, b1);
                    mma_bf16(y[nt + 1], lo[0], lo[1], lo[2], lo[3], b2, b3);
                }
            }
#pragma unroll
            for (int nt = 0; nt < CP / 8; ++nt) {
                const int col = pt0 + nt * 8 + nc;
                if (col >= P) continue;                  // P is even: a pair is inside or outside
                const int t0 = c * CQ + r0, t1 = c * CQ + r1;
                if (t0 < n_rows) *reinterpret_cast<float2*>(y_out + (size_t)t0 * inner + col) = make_float2(y[nt][0], y[nt][1]);
                if (t1 < n_rows) *reinterpret_cast<float2*>(y_out + (size_t)t1 * inner + col) = make_float2(y[nt][2], y[nt][3]);
            }
        }
        return;
    }

    // ---- the chunks' rows, their step sizes, and S
    const float bias = p.dt_bias[h], a = p.a[h];
    float* st = p.state + (size_t)p.seg_slot[seg] * p.state_stride;
    float* S0 = st + (size_t)h * P * N;
    uint8_t* s_hi_ptr = smem + (s_hi - b_tiles);
    uint8_t* s_lo_ptr = smem + (s_lo - b_tiles);
    const __nv_bfloat16* xbc = static_cast<const __nv_bfloat16*>(p.xbc) + (size_t)row0 * CH;
    const __nv_bfloat16* dt_in = static_cast<const __nv_bfloat16*>(p.in) + (size_t)row0 * p.in_stride + p.dt_col + h;
    const int pieces = NP / 8;                               // 16-byte pieces of a row of B or C
    auto load_chunk = [&](int c) {
        const int buf = c & 1, first = c * CQ;
        for (int r = warp; r < CQ; r += CWARPS) {            // a row of B and of C by a warp
            const bool there = first + r < n_rows;
            const __nv_bfloat16* src = xbc + (there ? (size_t)(first + r) * CH : 0) + inner + (size_t)g * N;
            for (int q = lane; q < 2 * pieces; q += 32) {
                const bool is_c = q >= pieces;
                const int piece = is_c ? q - pieces : q;
                cp_async16((is_c ? c_tiles : b_tiles) + (buf * CQ + r) * pitch + piece * 16,
                           src + (is_c ? (size_t)p.G * N : 0) + (piece * 8 < N ? piece * 8 : 0), there && piece * 8 < N);
            }
        }
#pragma unroll
        for (int i = 0; i < CQ * (CP / 8) / (CWARPS * 32); ++i) {
            const int at = i * CWARPS * 32 + warp * 32 + lane, r = at / (CP / 8), piece = at % (CP / 8), col = pt0 + piece * 8;
            const bool there = first + r < n_rows && col < P;
            cp_async16(x_tiles + (buf * CQ + r) * XPITCH + piece * 16, xbc + (there ? (size_t)(first + r) * CH + (size_t)h * P + col : 0), there);
        }
        cp_async_commit();
    };
    // step sizes, the running sums of a dt, and what each token's outer product is worth at the chunk's end (by one warp; a
    // lane has two neighbouring tokens)
    auto make_sums = [&](int c, float u, float v) {
        const int t = c * CQ + 2 * lane;
        const float d0 = t < n_rows ? softplus(u + bias) : 0.0f, d1 = t + 1 < n_rows ? softplus(v + bias) : 0.0f;
        const float l0 = a * d0, l1 = a * d1;
        float run = l0 + l1;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, run, o);
            if (lane >= o) run += up;
        }
        const float last = __shfl_sync(0xffffffffu, run, 31), before = __shfl_up_sync(0xffffffffu, run, 1);
        const float c0 = (lane ? before : 0.0f) + l0;
        float* to = sums + (c & 1) * 3 * CQ + 2 * lane;
        *reinterpret_cast<float2*>(to) = make_float2(c0, run);
        *reinterpret_cast<float2*>(to + CQ) = make_float2(d0, d1);
        *reinterpret_cast<float2*>(to + 2 * CQ) = make_float2(__expf(last - c0) * d0, __expf(last - run) * d1);
    };
    auto load_dt = [&](int c, float& u, float& v) {
        const int t = c * CQ + 2 * lane;
        u = t < n_rows ? __bfloat162float(dt_in[(size_t)t * p.in_stride]) : 0.0f;
        v = t + 1 < n_rows ? __bfloat162float(dt_in[(size_t)(t + 1) * p.in_stride]) : 0.0f;
    };

    load_chunk(0);
    float u, v;
    if (warp == 0) load_dt(0, u, v);
    // S: rows p = mt * 16 + lane / 4 (+ 8), columns n = 16 tile + nt * 8 + 2 (lane % 4) (+ 1)
    float S[NTW][2][2][4];
    const int pr = lane >> 2;
#pragma unroll
    for (int k = 0; k < NTW; ++k)
#pragma unroll
        for (int mt = 0; mt < 2; ++mt)
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    const int pp = pt0 + mt * 16 + pr + half * 8, n = (warp + 4 * k) * 16 + nt * 8 + nc;      // N is even
                    const float2 v2 = pp < P && n < N ? *reinterpret_cast<const float2*>(S0 + (size_t)pp * N + n) : make_float2(0.0f, 0.0f);
                    S[k][mt][nt][2 * half] = v2.x;
                    S[k][mt][nt][2 * half + 1] = v2.y;
                }
    auto put_state = [&]() {
#pragma unroll
        for (int k = 0; k < NTW; ++k) {
            if (warp + 4 * k >= ntiles) continue;
#pragma unroll
            for (int mt = 0; mt < 2; ++mt)
#pragma unroll
                for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                    for (int half = 0; half < 2; ++half) {
                        uint32_t hi, lo;
                        split2(S[k][mt][nt][2 * half], S[k][mt][nt][2 * half + 1], hi, lo);
                        const int at = (mt * 16 + pr + half * 8) * pitch + ((warp + 4 * k) * 16 + nt * 8 + nc) * 2;
                        *reinterpret_cast<uint32_t*>(s_hi_ptr + at) = hi;
                        *reinterpret_cast<uint32_t*>(s_lo_ptr + at) = lo;
                    }
        }
    };
    put_state();
    if (warp == 0) make_sums(0, u, v);
    cp_async_wait<0>();
    for (int c = 0; c < chunks; ++c) {
        const int buf = c & 1;
        const uint32_t bt = b_tiles + buf * CQ * pitch, xt = x_tiles + buf * CQ * XPITCH;
        const float* cum = sums + buf * 3 * CQ;
        const float* wts = cum + 2 * CQ;
        asm volatile("bar.sync 2, %0;" ::"n"(CTHREADS) : "memory");                                 // everyone is done with the other buffer
        const bool more = c + 1 < chunks;
        if (more) {
            load_chunk(c + 1);
            if (warp == 0) load_dt(c + 1, u, v);
        }
        // S <- exp(cum_last) S + sum_j w_j x_j B_j^T: rows p, contraction over the tokens
        const float keep = __expf(cum[CQ - 1]);
#pragma unroll
        for (int k = 0; k < NTW; ++k)
#pragma unroll
            for (int mt = 0; mt < 2; ++mt)
#pragma unroll
                for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                    for (int i = 0; i < 4; ++i) S[k][mt][nt][i] *= keep;
#pragma unroll
        for (int kt = 0; kt < CQ / 16; ++kt) {
            const float2 w0 = *reinterpret_cast<const float2*>(wts + kt * 16 + nc), w1 = *reinterpret_cast<const float2*>(wts + kt * 16 + 8 + nc);
            uint32_t hi[2][4], lo[2][4];
#pragma unroll
            for (int mt = 0; mt < 2; ++mt) {
                // x^T as the left operand: stored by token, read transposed; matrices (p low, j low), (p high, j low), (p low, j
                // high), (p high, j high)
                uint32_t x[4];
                ldmatrix_x4_trans(xt + (kt * 16 + (lane & 7) + ((lane >> 4) << 3)) * XPITCH + (mt * 2 + ((lane >> 3) & 1)) * 16, x[0], x[1], x[2], x[3]);
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const float2 w = i < 2 ? w0 : w1;
                    split2(__uint_as_float(x[i] << 16) * w.x, __uint_as_float(x[i] & 0xffff0000u) * w.y, hi[mt][i], lo[mt][i]);
                }
            }
#pragma unroll
            for (int k = 0; k < NTW; ++k) {
                if (warp + 4 * k >= ntiles) continue;
                uint32_t b0, b1, b2, b3;
                const int row = kt * 16 + (lane & 7) + (((lane >> 3) & 1) << 3);
                ldmatrix_x4_trans(bt + row * pitch + ((warp + 4 * k) * 2 + (lane >> 4)) * 16, b0, b1, b2, b3);
#pragma unroll
                for (int mt = 0; mt < 2; ++mt) {
                    mma_bf16(S[k][mt][0], hi[mt][0], hi[mt][1], hi[mt][2], hi[mt][3], b0, b1);
                    mma_bf16(S[k][mt][1], hi[mt][0], hi[mt][1], hi[mt][2], hi[mt][3], b2, b3);
                    mma_bf16(S[k][mt][0], lo[mt][0], lo[mt][1], lo[mt][2], lo[mt][3], b0, b1);
                    mma_bf16(S[k][mt][1], lo[mt][0], lo[mt][1], lo[mt][2], lo[mt][3], b2, b3);
                }
            }
        }
        if (more && warp == 0) make_sums(c + 1, u, v);
        asm volatile("bar.sync 1, %0;" ::"n"(CTHREADS) : "memory");      // the outputs' warps have read the S of this chunk
        if (more) {
            put_state();
            cp_async_wait<0>();
        }
    }
#pragma unroll
    for (int k = 0; k < NTW; ++k)
#pragma unroll
        for (int mt = 0; mt < 2; ++mt)
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    const int pp = pt0 + mt * 16 + pr + half * 8, n = (warp + 4 * k) * 16 + nt * 8 + nc;
                    if (pp < P && n < N) *reinterpret_cast<float2*>(S0 + (size_t)pp * N + n) = make_float2(S[k][mt][nt][2 * half], S[k][mt][nt][2 * half + 1]);
                }
    move_conv_inputs<__nv_bfloat16>(p, st, row0, n_rows, (blockIdx.y * gridDim.x + blockIdx.x) * CWARPS + warp, gridDim.x * gridDim.y * CWARPS, lane, 32);
}

// One block per (token, part).
template <typename TZ, typename TO>
__global__ void gate_rms_kernel(const float* __restrict__ y, const TZ* __restrict__ z, long long z_stride, const float* __restrict__ w,
                                float eps, TO* __restrict__ out, int inner, int width) {
    extern __shared__ float row[];
    __shared__ float scratch[32];
    pdl_launch_dependents();
    pdl_wait();
    const size_t t = blockIdx.x;
    const int c0 = blockIdx.y * width;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < width; i += blockDim.x) {
        const float v = y[t * inner + c0 + i] * silu(to_float<TZ>(z[t * z_stride + c0 + i]));
        row[i] = v;
        ss += v * v;
    }
    const float inv = rsqrtf(block_sum_any(ss, scratch) / (float)width + eps);
    for (int i = threadIdx.x; i < width; i += blockDim.x) out[t * inner + c0 + i] = from_float<TO>(row[i] * inv * w[c0 + i]);
}

// The same with four elements per access and the part's products kept in registers (IT quads a thread).
template <typename TZ, typename TO, int IT>
__global__ void __launch_bounds__(1024) gate_rms_vec_kernel(const float* __restrict__ y, const TZ* __restrict__ z, long long z_stride,
                                                            const float* __restrict__ w, float eps, TO* __restrict__ out, int inner, int width) {
    __shared__ float scratch[32];
    pdl_launch_dependents();
    pdl_wait();
    const size_t t = blockIdx.x;
    const int c0 = blockIdx.y * width;
    float v[IT][4];
    float ss = 0.0f;
#pragma unroll
    for (int it = 0; it < IT; ++it) {
        const int i = (it * blockDim.x + threadIdx.x) * 4;
        v[it][0] = v[it][1] = v[it][2] = v[it][3] = 0.0f;
        if (i >= width) continue;
        const float4 a = load4(y + t * inner + c0 + i), b = load4(z + t * z_stride + c0 + i);
        v[it][0] = a.x * silu(b.x); v[it][1] = a.y * silu(b.y); v[it][2] = a.z * silu(b.z); v[it][3] = a.w * silu(b.w);
        ss += (v[it][0] * v[it][0] + v[it][1] * v[it][1]) + (v[it][2] * v[it][2] + v[it][3] * v[it][3]);
    }
    const float inv = rsqrtf(block_sum_any(ss, scratch) / (float)width + eps);
#pragma unroll
    for (int it = 0; it < IT; ++it) {
        const int i = (it * blockDim.x + threadIdx.x) * 4;
        if (i >= width) continue;
        const float4 g = load4(w + c0 + i);
        const float o[4] = {v[it][0] * inv * g.x, v[it][1] * inv * g.y, v[it][2] * inv * g.z, v[it][3] * inv * g.w};
        store4(out + t * inner + c0 + i, o);
    }
}

int check_ssd(const char* what, const SsdParams& p, int S, int dtype) {
    if (!p.xbc || !p.in || !p.dt_bias || !p.a || !p.d || !p.state || !p.seg_start || !p.seg_slot || !p.y || S < 0 || p.H < 1 || p.P < 1 ||
        p.N < 1 || p.G < 1 || p.K < 1 || p.H % p.G || p.dt_col < 0 || p.conv_col < 0 || p.in_stride < p.dt_col + p.H ||
        p.in_stride < p.conv_col + (long long)p.H * p.P + 2LL * p.G * p.N || !valid_dtype(dtype) || p.rows_from < 0)
        return fail(PH_ERR_ARG, "%s: bad arguments (S %d, H %d, P %d, N %d, G %d)", what, S, p.H, p.P, p.N, p.G);
    if (p.state_stride < (long long)p.H * p.P * p.N + (long long)(p.K - 1) * ((long long)p.H * p.P + 2LL * p.G * p.N))
        return fail(PH_ERR_ARG, "%s: a state of %lld floats is too small", what, p.state_stride);
    if (S > 65535 || p.H > 65535) return fail(PH_ERR_UNSUPPORTED, "%s: %d requests of %d heads exceed the grid", what, S, p.H);
    return PH_OK;
}

SsdParams make_params(const void* xbc, const void* in, long long in_stride, int dt_col, int conv_col, const float* dt_bias, const float* a,
                      const float* d, float* state, long long state_stride, const int32_t* seg_start, const int32_t* seg_slot, int H, int P,
                      int N, int G, int K, int rows_from, int rows_to, float* y) {
    SsdParams p;
    p.xbc = xbc; p.in = in; p.in_stride = in_stride; p.dt_col = dt_col; p.conv_col = conv_col; p.dt_bias = dt_bias; p.a = a; p.d = d;
    p.state = state; p.state_stride = state_stride; p.seg_start = seg_start; p.seg_slot = seg_slot; p.y = y; p.H = H; p.P = P; p.N = N;
    p.G = G; p.K = K; p.rows_from = rows_from; p.rows_to = rows_to > 0 ? rows_to : 0x7fffffff;
    return p;
}

}  // namespace

// xbc [T, H * P + 2 * G * N] and in [T, in_stride] in `dtype`; dt_bias, a (negative), d [H] float32; state [slots,
// state_stride] as laid out above; y [T, H * P] float32.  Requests whose portion has rows_from .. rows_to rows (rows_to 0: no
// bound) are taken, the others left alone.
PH_EXPORT int ph_ssd_scan(const void* xbc, const void* in, int dtype, long long in_stride, int dt_col, int conv_col, const float* dt_bias,
                          const float* a, const float* d, float* state, long long state_stride, const int32_t* seg_start,
                          const int32_t* seg_slot, int S, int H, int P, int N, int G, int K, int rows_from, int rows_to, float* y,
                          cudaStream_t stream) {
    const SsdParams p = make_params(xbc, in, in_stride, dt_col, conv_col, dt_bias, a, d, state, state_stride, seg_start, seg_slot, H, P, N, G,
                                    K, rows_from, rows_to, y);
    if (const int bad = check_ssd("ssd_scan", p, S, dtype)) return bad;
    if (S == 0) return PH_OK;
    const bool quads = N % 4 == 0 && ((long long)H * P) % 4 == 0 && state_stride % 4 == 0 && (((uintptr_t)state | (uintptr_t)xbc) & 15) == 0;
    const int units = quads ? N / 4 : N;
    if (units > 32 * 8) return fail(PH_ERR_UNSUPPORTED, "ssd_scan: %d states exceed the supported %d", N, quads ? 1024 : 256);
    int L = 1;
    while (L < 32 && L < units) L *= 2;
    const int ni = (units + L - 1) / L;
    const int per_block = SCAN_THREADS / L * SCAN_ROWS;
    const dim3 grid((P + per_block - 1) / per_block, H, S);
#define SCAN(TX, NI, V) launch_overlapped(ssd_scan_kernel<TX, NI, V>, grid, dim3(SCAN_THREADS), 0, stream, p, L)
#define SCAN_NI(TX, V) do { if (ni == 1) SCAN(TX, 1, V); else if (ni == 2) SCAN(TX, 2, V); else if (ni <= 4) SCAN(TX, 4, V); else SCAN(TX, 8, V); } while (0)
    PH_DISPATCH(dtype, TX, { if (quads) SCAN_NI(TX, 4); else SCAN_NI(TX, 1); });
#undef SCAN_NI
#undef SCAN
    return check_launch("ssd_scan");
}

// 1 when the chunked kernel takes these sizes: 16-byte pieces of x, B and C rows, and at most 256 states.
PH_EXPORT int ph_ssd_chunk_supports(int P, int N, int G) { return P % 8 == 0 && N % 8 == 0 && N >= 8 && N <= 256 && G >= 1; }

// As ph_ssd_scan over bfloat16 rows, in chunks of 64 tokens on the tensor cores.
PH_EXPORT int ph_ssd_chunk(const void* xbc, const void* in, long long in_stride, int dt_col, int conv_col, const float* dt_bias,
                           const float* a, const float* d, float* state, long long state_stride, const int32_t* seg_start,
                           const int32_t* seg_slot, int S, int H, int P, int N, int G, int K, int rows_from, int rows_to, float* y,
                           cudaStream_t stream) {
    const SsdParams p = make_params(xbc, in, in_stride, dt_col, conv_col, dt_bias, a, d, state, state_stride, seg_start, seg_slot, H, P, N, G,
                                    K, rows_from, rows_to, y);
    if (const int bad = check_ssd("ssd_chunk", p, S, PH_BF16)) return bad;
    if (!ph_ssd_chunk_supports(P, N, G)) return fail(PH_ERR_UNSUPPORTED, "ssd_chunk: heads of %d with %d states are not taken", P, N);
    if (((uintptr_t)xbc & 15) || ((uintptr_t)state & 7) || state_stride % 2 || ((uintptr_t)y & 7))
        return fail(PH_ERR_ARG, "ssd_chunk: rows must be 16-byte aligned");
    if (S == 0) return PH_OK;
    const int NP = (N + 15) / 16 * 16, smem = ssd_smem(NP);
    const dim3 grid((P + CP - 1) / CP, H, S);
#define CHUNK(NTW)                                                                                                                \
    do {                                                                                                                          \
        if (cudaFuncSetAttribute(ssd_chunk_kernel<NTW>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess)        \
            return fail(PH_ERR_LAUNCH, "ssd_chunk: %d bytes of shared memory were refused", smem);                                \
        launch_overlapped(ssd_chunk_kernel<NTW>, grid, dim3(CTHREADS), (size_t)smem, stream, p, NP);                              \
    } while (0)
    if (NP <= 64) CHUNK(1); else if (NP <= 128) CHUNK(2); else CHUNK(4);
#undef CHUNK
    return check_launch("ssd_chunk");
}

// y [T, inner] float32, z [T, z_stride] (its first `inner` columns), w [inner] -> out [T, inner]; parts equal parts of a row.
PH_EXPORT int ph_gate_rms(const float* y, const void* z, int z_dtype, long long z_stride, const float* w, float eps, void* out, int out_dtype,
                          int T, int inner, int parts, cudaStream_t stream) {
    if (!y || !z || !w || !out || T < 0 || inner < 1 || parts < 1 || inner % parts || z_stride < inner || !valid_dtype(z_dtype) || !valid_dtype(out_dtype))
        return fail(PH_ERR_ARG, "gate_rms: bad arguments (T %d, width %d in %d parts)", T, inner, parts);
    if (parts > 65535) return fail(PH_ERR_UNSUPPORTED, "gate_rms: %d parts exceed the grid", parts);
    if (T == 0) return PH_OK;
    const int width = inner / parts;
    if (width % 4 == 0 && width <= 16384 && z_stride % 4 == 0 && (((uintptr_t)y | (uintptr_t)z | (uintptr_t)w | (uintptr_t)out) & 15) == 0) {
        const int quads = width / 4;
        int it = 1;
        while (it < 4 && (quads > 1024 * it || (T >= 256 && quads > 256 * it))) it *= 2;
        const int threads = ((quads + it - 1) / it + 31) / 32 * 32;
#define RMS(IT) launch_overlapped(gate_rms_vec_kernel<TZ, TO, IT>, dim3(T, parts), dim3(threads), 0, stream, y, (const TZ*)z, z_stride, w, eps, (TO*)out, inner, width)
        PH_DISPATCH(z_dtype, TZ, PH_DISPATCH(out_dtype, TO, { if (it == 1) RMS(1); else if (it == 2) RMS(2); else RMS(4); }));
#undef RMS
        return check_launch("gate_rms");
    }
    const size_t smem = (size_t)width * sizeof(float);
    if (smem > 200 * 1024) return fail(PH_ERR_UNSUPPORTED, "gate_rms: a part of %d numbers does not fit shared memory", width);
    const int threads = width >= 1024 ? 256 : width >= 128 ? 128 : 32;
#define RMS(TZ, TO)                                                                                                              \
    do {                                                                                                                         \
        auto kern = gate_rms_kernel<TZ, TO>;                                                                                     \
        if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                \
        launch_overlapped(kern, dim3(T, parts), dim3(threads), smem, stream, y, (const TZ*)z, z_stride, w, eps, (TO*)out, inner, width); \
    } while (0)
    PH_DISPATCH(z_dtype, TZ, PH_DISPATCH(out_dtype, TO, RMS(TZ, TO)));
#undef RMS
    return check_launch("gate_rms");
}
