// The delta rule's recurrence in chunks of 64 tokens, for long portions of a bfloat16 model (delta_rule.cu states the
// recurrence and what stands around it).
//
// Within a chunk let G_i be the running sum of the decays' logarithms per key channel up to and with token i, S the state at
// the chunk's start, and
//     A_ij = sum_d k_i k_j exp(G_i - G_j)  (j < i),     P_ij = sum_d q_i k_j exp(G_i - G_j)  (j <= i).
// Then, over all the chunk's tokens,
//     (1 + diag(beta) A) U = diag(beta) (V - (k exp(G)) S),      O = (q exp(G)) S + P U,
//     S <- diag(exp(G_last)) S + (k exp(G_last - G))^T U.
// The triangular system is solved for its two right-hand sides before S is known: U = U0 - W S with
// (1 + diag(beta) A) [W | U0] = diag(beta) [k exp(G) | V].
//
//   delta_chunk_make   a block per (chunk, head), all chunks side by side: A and P in float32 on packed multiply-adds, row block
//                      by row block of 16 with the decays taken from the block's first token, so that every exponential of an
//                      earlier block is at most 1; inside a block the inverse factor may grow, and where it would grow beyond
//                      2^60 the block takes every pair's exponential itself.  The system is solved by forward
//                      substitution in float32, two columns per thread.  W, q exp(G), k exp(G_last - G) and P leave as two
//                      bfloat16 each, the rounded value and the rounded rest.
//   delta_chunk_walk   a block per (request, head, 32 columns of S) that walks the request's chunks in order with S in registers
//                      (float32, spread over its eight warps) and, split the same way, in shared memory.  Every product is three
//                      tensor-core products of the split operands, so 16 bits of every factor count, and the sums are float32.
//                      Four warps make U while four others make (q exp(G)) S, then all add their part to S while the
//                      second four add P U and store O; the next chunk's operands are on their way meanwhile.
// Tokens beyond a request's last have k = q = v = beta = 0 and a decay of 1.
#include "attention_mma.cuh"
#include "delta_rule.cuh"

#include <math.h>

namespace {

using namespace ph;
using namespace ph_attn;

constexpr int C = 64;                  // tokens of a chunk
constexpr int RB = 16;                 // tokens of a row block
constexpr int NC = 32;                 // columns of S per block of the walk
constexpr int MAX_DIM = 128;
constexpr int MAKE_THREADS = 256, WALK_THREADS = 256;
constexpr float GROW_LIMIT = 60.0f;    // log2 of the largest inverse factor inside a row block

struct ChunkParams {
    ph_delta::ScanParams s;
    const int32_t* chunks;             // [n][2]: first row, rows
    const int32_t* seg_chunks;         // [S + 1]
    __nv_bfloat16* ops;                // per (chunk, head): [W hi | W lo | Q hi | Q lo | K hi | K lo] of 64 x D, then [P hi | P lo] of 64 x 64
    float* u0;                         // per (chunk, head): [64][DV]
    float* last;                       // per (chunk, head): [D] exp(G_last)
    int rows_bf16;                     // the projections' rows are bfloat16
};

__host__ __device__ constexpr long long ops_elems(int D) { return 6LL * C * D + 2LL * C * C; }

__device__ __forceinline__ float ex2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
    float2 d;
    asm("{\n.reg .b64 ra, rb, rc, rd;\n"
        "mov.b64 ra, {%2, %3};\nmov.b64 rb, {%4, %5};\nmov.b64 rc, {%6, %7};\n"
        "fma.rn.f32x2 rd, ra, rb, rc;\n"
        "mov.b64 {%0, %1}, rd;\n}"
        : "=f"(d.x), "=f"(d.y) : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y), "f"(c.x), "f"(c.y));
    return d;
}
// v = hi + lo with both in bfloat16 (hi the rounded value, lo the rounded rest), two values at a time
__device__ __forceinline__ void split2(float u, float v, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16(u, v);
    lo = pack_bf16(u - __uint_as_float(hi << 16), v - __uint_as_float(hi & 0xffff0000u));
}

// floats of shared memory of delta_chunk_make: k, q, G, the scaled keys [64][D + 4], the scaled rows of k and q [16][D + 4],
// the system [64][64 + 4] and P [64][64 + 4], beta [64]
__host__ __device__ constexpr int make_floats(int D) { return 4 * C * (D + 4) + 2 * RB * (D + 4) + 2 * C * (C + 4) + C; }

__global__ void __launch_bounds__(MAKE_THREADS, 1) delta_chunk_make_kernel(const ChunkParams p) {
    extern __shared__ __align__(16) float sm[];
    __shared__ int slow;
    const int D = p.s.D, DV = p.s.DV, DP = D + 4, H = p.s.H, CH = 2 * p.s.G * D + H * DV;
    constexpr int NP = C + 4;
    float* ks = sm;                    // [64][DP]
    float* qs = ks + C * DP;
    float* Gs = qs + C * DP;           // in units of log2
    float* kj = Gs + C * DP;
    float* ki = kj + C * DP;           // [16][DP]
    float* qi = ki + RB * DP;
    float* N = qi + RB * DP;           // [64][NP]
    float* P = N + C * NP;
    float* beta = P + C * NP;
    const int tid = threadIdx.x, item = blockIdx.x, h = blockIdx.y, g = h / (H / p.s.G);
    pdl_launch_dependents();
    pdl_wait();
    const int row0 = p.chunks[2 * item], n = p.chunks[2 * item + 1];
    const float* rows = p.s.qkv + (size_t)row0 * CH;

    // ---- the chunk's rows
    const int per_row = D / 4;
    for (int i = tid; i < C * per_row; i += MAKE_THREADS) {
        const int r = i / per_row, d = (i % per_row) * 4;
        float4 q4 = make_float4(0.0f, 0.0f, 0.0f, 0.0f), k4 = q4;
        if (r < n) {
            q4 = *reinterpret_cast<const float4*>(rows + (size_t)r * CH + g * D + d);
            k4 = *reinterpret_cast<const float4*>(rows + (size_t)r * CH + (p.s.G + g) * D + d);
        }
        *reinterpret_cast<float4*>(qs + r * DP + d) = q4;
        *reinterpret_cast<float4*>(ks + r * DP + d) = k4;
    }
    if (tid < C) beta[tid] = tid < n ? p.s.beta[(size_t)(row0 + tid) * H + h] : 0.0f;
    // ---- G: each half of the tokens summed by a thread of its own per channel, then the first half's sum added to the second
    if (tid < 2 * D) {
        const int d = tid % D, part = tid / D, first = part * (C / 2);
        float run = 0.0f;
        if (p.s.z) {
            const float rate = p.s.rate[h] * LOG2E, bias = p.s.z_bias[(size_t)h * D + d];
            const float* z = p.s.z + (size_t)row0 * p.s.z_stride + (size_t)h * D + d;
#pragma unroll 8
            for (int t = 0; t < C / 2; ++t) {
                const int i = first + t;
                run += i < n ? rate * ph_delta::softplus(z[(size_t)i * p.s.z_stride] + bias) : 0.0f;
                Gs[i * DP + d] = run;
            }
        } else {
            const float* ld = p.s.log_decay + (size_t)row0 * H + h;
#pragma unroll 8
            for (int t = 0; t < C / 2; ++t) {
                const int i = first + t;
                run += i < n ? ld[(size_t)i * H] * LOG2E : 0.0f;
                Gs[i * DP + d] = run;
            }
        }
    }
    __syncthreads();
    for (int i = tid; i < C / 2 * D; i += MAKE_THREADS) {
        const int r = C / 2 + i / D, d = i % D;
        Gs[r * DP + d] += Gs[(C / 2 - 1) * DP + d];
    }
    for (int i = tid; i < C * NP; i += MAKE_THREADS) { N[i] = 0.0f; P[i] = 0.0f; }

    // ---- A and P, 16 rows at a time
    for (int I = 0; I < C / RB; ++I) {
        __syncthreads();
        if (tid == 0) slow = 0;
        __syncthreads();
        for (int d = tid; d < D; d += MAKE_THREADS) {
            const float ref = I ? Gs[(I * RB - 1) * DP + d] : 0.0f;
            if (ref - Gs[(I * RB + RB - 1) * DP + d] > GROW_LIMIT) slow = 1;       // every writer writes the same
        }
        for (int i = tid; i < (I + 1) * RB * D; i += MAKE_THREADS) {
            const int r = i / D, d = i % D;
            const float ref = I ? Gs[(I * RB - 1) * DP + d] : 0.0f;
            kj[r * DP + d] = ks[r * DP + d] * ex2(fminf(ref - Gs[r * DP + d], GROW_LIMIT));
            if (r >= I * RB) {
                const float f = ex2(Gs[r * DP + d] - ref);
                ki[(r - I * RB) * DP + d] = ks[r * DP + d] * f;
                qi[(r - I * RB) * DP + d] = qs[r * DP + d] * f;
            }
        }
        __syncthreads();
        const bool every_pair = slow != 0;
        const int i = tid / RB, j0 = tid % RB;             // this thread's row of the block, and its column of each block of columns
        const float bi = beta[I * RB + i];
        const int blocks = every_pair ? I : I + 1;
        float2 a[C / RB], b[C / RB];
#pragma unroll
        for (int m = 0; m < C / RB; ++m) a[m] = b[m] = make_float2(0.0f, 0.0f);
        const float* kr = ki + i * DP;
        const float* qr = qi + i * DP;
        for (int d = 0; d < D; d += 4) {
            const float4 k4 = *reinterpret_cast<const float4*>(kr + d), q4 = *reinterpret_cast<const float4*>(qr + d);
#pragma unroll
            for (int m = 0; m < C / RB; ++m) {
                if (m >= blocks) break;
                const float4 x = *reinterpret_cast<const float4*>(kj + (m * RB + j0) * DP + d);
                a[m] = fma2(make_float2(k4.x, k4.y), make_float2(x.x, x.y), a[m]);
                a[m] = fma2(make_float2(k4.z, k4.w), make_float2(x.z, x.w), a[m]);
                b[m] = fma2(make_float2(q4.x, q4.y), make_float2(x.x, x.y), b[m]);
                b[m] = fma2(make_float2(q4.z, q4.w), make_float2(x.z, x.w), b[m]);
            }
        }
#pragma unroll
        for (int m = 0; m < C / RB; ++m) {
            if (m >= blocks) break;
            const int r = I * RB + i, j = m * RB + j0;
            if (j < r) N[r * NP + j] = bi * (a[m].x + a[m].y);
            if (j <= r) P[r * NP + j] = b[m].x + b[m].y;
        }
        if (every_pair && j0 <= i) {
            const int r = I * RB + i, j = I * RB + j0;
            float sa = 0.0f, sb = 0.0f;
            for (int d = 0; d < D; ++d) {
                const float x = ks[j * DP + d] * ex2(Gs[r * DP + d] - Gs[j * DP + d]);
                sa = fmaf(ks[r * DP + d], x, sa);
                sb = fmaf(qs[r * DP + d], x, sb);
            }
            if (j < r) N[r * NP + j] = bi * sa;
            P[r * NP + j] = sb;
        }
    }
    __syncthreads();

    const size_t at = (size_t)item * H + h;
    uint32_t* ops = reinterpret_cast<uint32_t*>(p.ops + at * ops_elems(D));
    const int tile = C * D / 2;        // pairs of a 64 x D operand
    if (tid < MAKE_THREADS / 2) {
        // ---- the system, two columns of [W | U0] per thread
        float* u0 = p.u0 + at * C * DV;
        for (int c = 2 * tid; c < D + DV; c += MAKE_THREADS) {
            const bool is_w = c < D;
            float2 x[C];
            const float* v = rows + 2 * p.s.G * D + (size_t)h * DV + (c - D);
#pragma unroll
            for (int i = 0; i < C; ++i) {
                float2 r = make_float2(0.0f, 0.0f);
                if (is_w) {
                    const float2 k2 = *reinterpret_cast<const float2*>(ks + i * DP + c), g2 = *reinterpret_cast<const float2*>(Gs + i * DP + c);
                    r = make_float2(k2.x * ex2(g2.x), k2.y * ex2(g2.y));
                } else if (i < n) {
                    r = *reinterpret_cast<const float2*>(v + (size_t)i * CH);
                }
                x[i] = make_float2(r.x * beta[i], r.y * beta[i]);
            }
#pragma unroll
            for (int i = 1; i < C; ++i) {
                float2 even = x[i], odd = make_float2(0.0f, 0.0f);
#pragma unroll
                for (int j = 0; j < i; j += 4) {
                    const float4 m = *reinterpret_cast<const float4*>(N + i * NP + j);     // (zero from j = i on)
                    even = fma2(make_float2(-m.x, -m.x), x[j], even);
                    if (j + 1 < i) odd = fma2(make_float2(-m.y, -m.y), x[j + 1], odd);
                    if (j + 2 < i) even = fma2(make_float2(-m.z, -m.z), x[j + 2], even);
                    if (j + 3 < i) odd = fma2(make_float2(-m.w, -m.w), x[j + 3], odd);
                }
                x[i] = make_float2(even.x + odd.x, even.y + odd.y);
            }
#pragma unroll
            for (int i = 0; i < C; ++i) {
                if (is_w) {
                    uint32_t hi, lo;
                    split2(x[i].x, x[i].y, hi, lo);
                    ops[(i * D + c) / 2] = hi;
                    ops[tile + (i * D + c) / 2] = lo;
                } else {
                    *reinterpret_cast<float2*>(u0 + (size_t)i * DV + (c - D)) = x[i];
                }
            }
        }
    } else {
        // ---- the other operands
        const int w = tid - MAKE_THREADS / 2;
        const float* gl = Gs + (C - 1) * DP;
        for (int e = w; e < tile; e += MAKE_THREADS / 2) {
            const int i = 2 * e / D, d = 2 * e % D;
            const float2 q2 = *reinterpret_cast<const float2*>(qs + i * DP + d), k2 = *reinterpret_cast<const float2*>(ks + i * DP + d),
                         g2 = *reinterpret_cast<const float2*>(Gs + i * DP + d), l2 = *reinterpret_cast<const float2*>(gl + d);
            uint32_t hi, lo;
            split2(q2.x * ex2(g2.x), q2.y * ex2(g2.y), hi, lo);
            ops[2 * tile + e] = hi; ops[3 * tile + e] = lo;
            split2(k2.x * ex2(l2.x - g2.x), k2.y * ex2(l2.y - g2.y), hi, lo);
            ops[4 * tile + e] = hi; ops[5 * tile + e] = lo;
        }
        for (int e = w; e < C * C / 2; e += MAKE_THREADS / 2) {
            const int i = 2 * e / C, j = 2 * e % C;
            uint32_t hi, lo;
            split2(P[i * NP + j], P[i * NP + j + 1], hi, lo);
            ops[6 * tile + e] = hi; ops[6 * tile + C * C / 2 + e] = lo;
        }
        for (int d = w; d < D; d += MAKE_THREADS / 2) p.last[at * D + d] = ex2(gl[d]);
    }
}

constexpr int S_PITCH = NC * 2 + 16;   // bytes of a row of the S and U tiles
constexpr int P_PITCH = C * 2 + 16;
__host__ __device__ constexpr int op_pitch(int D) { return D * 2 + 16; }
// W and Q of two chunks, K and P of one, S, U: each as two bfloat16 tiles
__host__ __device__ constexpr int walk_smem(int D) {
    return 2 * 4 * C * op_pitch(D) + 2 * C * op_pitch(D) + 2 * C * P_PITCH + 2 * D * S_PITCH + 2 * C * S_PITCH;
}

// acc[16 x 32] += (a_hi + a_lo)[16 x 16 KS] (b_hi + b_lo)[16 KS x 32] without the product of the two rests.  a: row-major rows
// of the warp's 16 (a_t: stored transposed), b: [k][32 columns].
template <bool A_T>
__device__ __forceinline__ void split_product(float (&acc)[NC / 8][4], float (&rest)[NC / 8][4], uint32_t a_hi, uint32_t a_lo, int a_pitch,
                                              uint32_t b_hi, uint32_t b_lo, int steps) {
    const int lane = threadIdx.x & 31;
#pragma unroll 4
    for (int ks = 0; ks < steps; ++ks) {
        uint32_t h[4], l[4];
        if constexpr (A_T) {
            // stored [k][row]: matrices (rows low, k low), (rows high, k low), (rows low, k high), (rows high, k high)
            const int at = (ks * 16 + (lane & 7) + ((lane >> 4) << 3)) * a_pitch + ((lane >> 3) & 1) * 16;
            ldmatrix_x4_trans(a_hi + at, h[0], h[1], h[2], h[3]);
            ldmatrix_x4_trans(a_lo + at, l[0], l[1], l[2], l[3]);
        } else {
            const int at = (lane & 15) * a_pitch + (ks * 2 + (lane >> 4)) * 16;
            ldmatrix_x4(a_hi + at, h[0], h[1], h[2], h[3]);
            ldmatrix_x4(a_lo + at, l[0], l[1], l[2], l[3]);
        }
        const int row = ks * 16 + (lane & 7) + (((lane >> 3) & 1) << 3);
#pragma unroll
        for (int nt = 0; nt < NC / 8; nt += 2) {
            uint32_t b0, b1, b2, b3, c0, c1, c2, c3;
            const int at = row * S_PITCH + (nt + (lane >> 4)) * 16;
            ldmatrix_x4_trans(b_hi + at, b0, b1, b2, b3);
            ldmatrix_x4_trans(b_lo + at, c0, c1, c2, c3);
            mma_bf16(acc[nt], h[0], h[1], h[2], h[3], b0, b1);
            mma_bf16(acc[nt + 1], h[0], h[1], h[2], h[3], b2, b3);
            mma_bf16(rest[nt], l[0], l[1], l[2], l[3], b0, b1);
            mma_bf16(rest[nt + 1], l[0], l[1], l[2], l[3], b2, b3);
            mma_bf16(rest[nt], h[0], h[1], h[2], h[3], c0, c1);
            mma_bf16(rest[nt + 1], h[0], h[1], h[2], h[3], c2, c3);
        }
    }
}

__global__ void __launch_bounds__(WALK_THREADS, 1) delta_chunk_walk_kernel(const ChunkParams p) {
    extern __shared__ __align__(128) uint8_t smem[];
    pdl_launch_dependents();
    pdl_wait();
    const int seg = blockIdx.z, h = blockIdx.y, col0 = blockIdx.x * NC;
    const int first = p.seg_chunks[seg], chunks = p.seg_chunks[seg + 1] - first;
    if (chunks <= 0) return;
    const int D = p.s.D, DV = p.s.DV, H = p.s.H, pitch = op_pitch(D), tiles = D / 16;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const bool outputs = warp >= 4;
    const int rows = warp & 3;                                 // this warp's 16 tokens of the chunk
    const uint32_t base = smem_u32(smem);
    const int op = C * pitch;                                  // bytes of a 64 x D tile
    const uint32_t k_tiles = base + 8 * op, p_tiles = k_tiles + 2 * op, s_tiles = p_tiles + 2 * C * P_PITCH, u_tiles = s_tiles + 2 * D * S_PITCH;
    const uint32_t s_lo = (uint32_t)(D * S_PITCH), u_lo = (uint32_t)(C * S_PITCH);
    const int pieces = D / 8;                                  // 16-byte pieces of a row

    // tiles [from, from + count) of the operands of a chunk (64 x D each) to `to`
    auto load_ops = [&](int c, int from, int count, uint32_t to) {
        const __nv_bfloat16* src = p.ops + ((size_t)(first + c) * H + h) * ops_elems(D) + (size_t)from * C * D;
        for (int i = threadIdx.x; i < count * C * pieces; i += WALK_THREADS) {
            const int row = i / pieces, piece = i % pieces;
            cp_async16(to + row * pitch + piece * 16, src + (size_t)row * D + piece * 8, true);
        }
    };
    auto load_p = [&](int c) {
        const __nv_bfloat16* src = p.ops + ((size_t)(first + c) * H + h) * ops_elems(D) + 6LL * C * D;
        for (int i = threadIdx.x; i < 2 * C * (C / 8); i += WALK_THREADS) {
            const int row = i / (C / 8), piece = i % (C / 8);
            cp_async16(p_tiles + row * P_PITCH + piece * 16, src + (size_t)row * C + piece * 8, true);
        }
    };

    load_ops(0, 0, 4, base);
    cp_async_commit();
    // S: warp w holds the channels 16 w .. 16 w + 15 (rows lane / 4 and + 8), columns nt * 8 + 2 (lane % 4) (+ 1)
    const int nc = (lane & 3) * 2, ch = warp * 16 + (lane >> 2);
    const bool holds = warp < tiles;
    float* S0 = p.s.state + (size_t)p.s.seg_slot[seg] * p.s.state_stride + (size_t)h * DV * D;
    float S[NC / 8][4];
#pragma unroll
    for (int nt = 0; nt < NC / 8; ++nt)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int col = col0 + nt * 8 + nc + (i & 1), d = ch + (i >> 1) * 8;
            S[nt][i] = holds && col < DV ? S0[(size_t)col * D + d] : 0.0f;
        }
    auto put_state = [&]() {
        if (!holds) return;
#pragma unroll
        for (int nt = 0; nt < NC / 8; ++nt)
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                uint32_t hi, lo;
                split2(S[nt][2 * half], S[nt][2 * half + 1], hi, lo);
                uint8_t* to = smem + (s_tiles - base) + (ch + half * 8) * S_PITCH + (nt * 8 + nc) * 2;
                *reinterpret_cast<uint32_t*>(to) = hi;
                *reinterpret_cast<uint32_t*>(to + s_lo) = lo;
            }
    };
    put_state();
    const int r0 = rows * 16 + (lane >> 2);
    for (int c = 0; c < chunks; ++c) {
        const size_t at = (size_t)(first + c) * H + h;
        const uint32_t w_tiles = base + (c & 1) * 4 * op, q_tiles = w_tiles + 2 * op;
        float acc[NC / 8][4], rest[NC / 8][4];
#pragma unroll
        for (int nt = 0; nt < NC / 8; ++nt)
#pragma unroll
            for (int i = 0; i < 4; ++i) acc[nt][i] = rest[nt][i] = 0.0f;
        float keep[2] = {1.0f, 1.0f};
        float2 u0[NC / 8][2];
        if (holds) { keep[0] = p.last[at * D + ch]; keep[1] = p.last[at * D + ch + 8]; }
        if (!outputs) {
#pragma unroll
            for (int nt = 0; nt < NC / 8; ++nt)
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    const int col = col0 + nt * 8 + nc;        // DV is even: a pair is inside or outside
                    u0[nt][half] = col < DV ? *reinterpret_cast<const float2*>(p.u0 + (at * C + r0 + half * 8) * DV + col) : make_float2(0.0f, 0.0f);
                }
        }
        cp_async_wait<0>();
        __syncthreads();                                       // W, Q and S are there; everyone is done with the last chunk's K, P and U
        load_ops(c, 4, 2, k_tiles);
        load_p(c);
        cp_async_commit();
        if (c + 1 < chunks) load_ops(c + 1, 0, 4, base + ((c + 1) & 1) * 4 * op);
        cp_async_commit();
        // W S for the tokens of warps 0 .. 3, Q S for those of warps 4 .. 7
        const uint32_t a = (outputs ? q_tiles : w_tiles) + rows * 16 * pitch;
        split_product<false>(acc, rest, a, a + op, pitch, s_tiles, s_tiles + s_lo, tiles);
        if (!outputs) {
#pragma unroll
            for (int nt = 0; nt < NC / 8; ++nt)
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    uint32_t hi, lo;
                    split2(u0[nt][half].x - (acc[nt][2 * half] + rest[nt][2 * half]), u0[nt][half].y - (acc[nt][2 * half + 1] + rest[nt][2 * half + 1]), hi, lo);
                    uint8_t* to = smem + (u_tiles - base) + (r0 + half * 8) * S_PITCH + (nt * 8 + nc) * 2;
                    *reinterpret_cast<uint32_t*>(to) = hi;
                    *reinterpret_cast<uint32_t*>(to + u_lo) = lo;
                }
        }
        cp_async_wait<1>();
        __syncthreads();                                       // U, K and P are there; everyone is done with S
        if (holds) {
            float sr[NC / 8][4];
#pragma unroll
            for (int nt = 0; nt < NC / 8; ++nt)
#pragma unroll
                for (int i = 0; i < 4; ++i) { S[nt][i] *= keep[i >> 1]; sr[nt][i] = 0.0f; }
            split_product<true>(S, sr, k_tiles + warp * 32, k_tiles + op + warp * 32, pitch, u_tiles, u_tiles + u_lo, C / 16);
#pragma unroll
            for (int nt = 0; nt < NC / 8; ++nt)
#pragma unroll
                for (int i = 0; i < 4; ++i) S[nt][i] += sr[nt][i];
            put_state();
        }
        if (outputs) {
            const uint32_t pa = p_tiles + rows * 16 * P_PITCH;
            split_product<false>(acc, rest, pa, pa + C * P_PITCH, P_PITCH, u_tiles, u_tiles + u_lo, rows + 1);      // later tokens weigh nothing
            const int row0 = p.chunks[2 * (first + c)], n = p.chunks[2 * (first + c) + 1];
            float* y = p.s.o + (size_t)row0 * H * DV + (size_t)h * DV;
#pragma unroll
            for (int nt = 0; nt < NC / 8; ++nt)
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    const int col = col0 + nt * 8 + nc, r = r0 + half * 8;
                    if (col < DV && r < n)
                        *reinterpret_cast<float2*>(y + (size_t)r * H * DV + col) =
                            make_float2(acc[nt][2 * half] + rest[nt][2 * half], acc[nt][2 * half + 1] + rest[nt][2 * half + 1]);
                }
        }
    }
    if (holds)
#pragma unroll
        for (int nt = 0; nt < NC / 8; ++nt)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int col = col0 + nt * 8 + nc + (i & 1), d = ch + (i >> 1) * 8;
                if (col < DV) S0[(size_t)col * D + d] = S[nt][i];
            }
    const int row0 = p.s.seg_start[seg], n_rows = p.s.seg_start[seg + 1] - row0;
    float* st = p.s.state + (size_t)p.s.seg_slot[seg] * p.s.state_stride;
    const int block = blockIdx.y * gridDim.x + blockIdx.x, blocks = gridDim.x * gridDim.y;
    if (p.rows_bf16) ph_delta::move_conv_inputs<__nv_bfloat16>(p.s, st, row0, n_rows, block, blocks, threadIdx.x, WALK_THREADS);
    else ph_delta::move_conv_inputs<float>(p.s, st, row0, n_rows, block, blocks, threadIdx.x, WALK_THREADS);
}

}  // namespace

// 1 when the chunked form takes heads of D channels and DV columns.
PH_EXPORT int ph_delta_chunk_supports(int D, int DV) { return D >= 16 && D % 16 == 0 && D <= MAX_DIM && DV >= 2 && DV % 2 == 0; }
PH_EXPORT int ph_delta_chunk_tokens(void) { return C; }
// bytes of scratch per (chunk, head): the operands, U0, and the chunk's decay
PH_EXPORT long long ph_delta_chunk_scratch_bytes(int D, int DV) { return (ops_elems(D) * 2 + 4LL * C * DV + 4LL * D + 255) / 256 * 256; }

namespace {
int fill(ChunkParams& p, const int32_t* chunks, int n_chunks, const int32_t* seg_chunks, void* scratch, int H, int G, int D, int DV) {
    if (!chunks || !scratch || n_chunks < 1 || H < 1 || G < 1 || H % G)
        return fail(PH_ERR_ARG, "delta_chunk: bad arguments (chunks %d, H %d, G %d, D %d, DV %d)", n_chunks, H, G, D, DV);
    if (!ph_delta_chunk_supports(D, DV)) return fail(PH_ERR_UNSUPPORTED, "delta_chunk: heads of %d / %d are not taken", D, DV);
    if ((2LL * G * D + (long long)H * DV) % 4 || ((uintptr_t)scratch & 255))
        return fail(PH_ERR_UNSUPPORTED, "delta_chunk: rows must be 16-byte aligned");
    const long long units = (long long)n_chunks * H;
    p.s.H = H; p.s.G = G; p.s.D = D; p.s.DV = DV;
    p.chunks = chunks; p.seg_chunks = seg_chunks;
    p.ops = static_cast<__nv_bfloat16*>(scratch);
    p.u0 = reinterpret_cast<float*>(p.ops + units * ops_elems(D));
    p.last = p.u0 + units * C * DV;
    return PH_OK;
}
}  // namespace

// The operands of every chunk and head.  chunks [n_chunks][2]: first row of the step and rows, at most 64; scratch: n_chunks * H *
// ph_delta_chunk_scratch_bytes, 256-byte aligned.  qkv, beta, log_decay / z as in ph_delta_scan.
PH_EXPORT int ph_delta_chunk_make(const float* qkv, const float* beta, const float* log_decay, const float* z, long long z_stride,
                                  const float* z_bias, const float* rate, const int32_t* chunks, int n_chunks, void* scratch, int H, int G, int D,
                                  int DV, cudaStream_t stream) {
    if (!qkv || !beta || (!log_decay == !z) || (z && (!z_bias || !rate)) || ((uintptr_t)qkv & 15))
        return fail(PH_ERR_ARG, "delta_chunk_make: bad arguments");
    ChunkParams p = {};
    if (int rc = fill(p, chunks, n_chunks, nullptr, scratch, H, G, D, DV)) return rc;
    p.s.qkv = qkv; p.s.beta = beta; p.s.log_decay = log_decay; p.s.z = z; p.s.z_stride = z_stride; p.s.z_bias = z_bias; p.s.rate = rate;
    const size_t smem = (size_t)make_floats(D) * sizeof(float);
    static size_t set = 0;
    if (smem > set) {
        if (cudaFuncSetAttribute(delta_chunk_make_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
            return fail(PH_ERR_LAUNCH, "delta_chunk_make: cannot reserve %zu bytes of shared memory", smem);
        set = smem;
    }
    launch_overlapped(delta_chunk_make_kernel, dim3(n_chunks, H), dim3(MAKE_THREADS), smem, stream, p);
    return check_launch("delta_chunk_make");
}

// The recurrence over the chunks of each request (seg_chunks [S + 1]; a request without chunks is left alone); what is left of
// its rows in the state as in ph_delta_scan.
PH_EXPORT int ph_delta_chunk_walk(const void* rows, int rows_dtype, int splits, long long split_stride, long long width, float* state,
                                  long long state_stride, long long conv_at, const int32_t* seg_start, const int32_t* seg_slot, int S,
                                  const int32_t* chunks, int n_chunks, const int32_t* seg_chunks, const void* scratch, int H, int G, int D,
                                  int DV, int K, float* o, cudaStream_t stream) {
    if (!rows || !state || !seg_start || !seg_slot || !seg_chunks || !o || S < 1 || K < 1 || splits < 1 || !valid_dtype(rows_dtype) || ((uintptr_t)o & 7))
        return fail(PH_ERR_ARG, "delta_chunk_walk: bad arguments (S %d)", S);
    ChunkParams p = {};
    if (int rc = fill(p, chunks, n_chunks, seg_chunks, const_cast<void*>(scratch), H, G, D, DV)) return rc;
    p.s.rows = rows; p.s.splits = splits; p.s.split_stride = split_stride; p.s.width = width; p.s.state = state; p.s.state_stride = state_stride;
    p.s.conv_at = conv_at; p.s.seg_start = seg_start; p.s.seg_slot = seg_slot; p.s.o = o; p.s.K = K;
    p.rows_bf16 = rows_dtype == PH_BF16;
    const size_t smem = (size_t)walk_smem(D);
    static size_t set = 0;
    if (smem > set) {
        if (cudaFuncSetAttribute(delta_chunk_walk_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
            return fail(PH_ERR_LAUNCH, "delta_chunk_walk: cannot reserve %zu bytes of shared memory", smem);
        set = smem;
    }
    launch_overlapped(delta_chunk_walk_kernel, dim3((DV + NC - 1) / NC, H, S), dim3(WALK_THREADS), smem, stream, p);
    return check_launch("delta_chunk_walk");
}
