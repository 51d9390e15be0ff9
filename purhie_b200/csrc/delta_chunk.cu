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
//   delta_chunk_make   a block per (chunk, head), all chunks side by side.  The chunk is cut into blocks of 16 tokens: with g_i
//                      the running sum inside token i's block and t_J block J's total, A and P of block rows I and block
//                      columns J come from k exp(g), q exp(g), k exp(t_J - g) (never above 1) and one factor per channel and
//                      pair of blocks, the decay between them; on the diagonal that factor is exp(-t_I), and where it would
//                      exceed 2^60 the block takes every pair's exponential itself.  Float32 on packed multiply-adds, 2 x 2
//                      pairs per thread.  M = (1 + diag(beta) A)^-1 in float32, block by block: the diagonal blocks by forward
//                      substitution, M_IJ = -M_II sum_K (diag(beta) A)_IK M_KJ below them, one distance from the diagonal
//                      after the other.  W and U0 are M diag(beta) times k exp(G) and V on the tensor cores, split operands as
//                      in the walk.  W, q exp(G), k exp(G_last - G) and P leave as two bfloat16 each, the rounded value and the
//                      rounded rest, in the layout of the walk's shared memory.
//   delta_chunk_walk   a block per (request, head, 32 columns of S) that walks the request's chunks in order with S in registers
//                      (float32, spread over its eight warps) and, split the same way, in shared memory.  Every product is three
//                      tensor-core products of the split operands, so 16 bits of every factor count, and the sums are float32.
//                      Four warps make U while four others make (q exp(G)) S, then all add their part to S while the
//                      second four add P U and store O; the next chunk's operands are on their way meanwhile, as bulk copies of
//                      whole regions that complete on mbarriers (bounded waits, an error word).
// Tokens beyond a request's last have k = q = v = beta = 0 and a decay of 1.
#include "attention_mma.cuh"
#include "delta_rule.cuh"
#include "mbarrier.cuh"

#include <math.h>

namespace {

using namespace ph;
using namespace ph_attn;

constexpr int C = 64;                  // tokens of a chunk
constexpr int RB = 16;                 // tokens of a row block
constexpr int NC = 32;                 // columns of S per block of the walk
constexpr int MAX_DIM = 128;
constexpr int MAKE_THREADS = 512, WALK_THREADS = 256;
constexpr int PH_ERR_WAIT_DELTA = 131;
constexpr float GROW_LIMIT = 60.0f;    // log2 of the largest inverse factor inside a row block

struct ChunkParams {
    ph_delta::ScanParams s;
    const int32_t* chunks;             // [n][2]: first row, rows
    const int32_t* seg_chunks;         // [S + 1]
    uint8_t* ops;                      // per (chunk, head): [W hi | W lo | Q hi | Q lo | K hi | K lo] of 64 rows of D, then [P hi | P lo] of 64 rows of 64
    float* u0;                         // per (chunk, head): [64][DV]
    float* last;                       // per (chunk, head): [D] exp(G_last)
    int rows_bf16;                     // the projections' rows are bfloat16
    int* error_flag;
};

// bytes between two rows of an operand of D (64) columns: 16 more than the row, so that eight rows miss each other's banks
__host__ __device__ constexpr int op_pitch(int D) { return D * 2 + 16; }
constexpr int P_PITCH = C * 2 + 16;
__host__ __device__ constexpr int first_bytes(int D) { return 4 * C * op_pitch(D); }               // W and Q
__host__ __device__ constexpr int second_bytes(int D) { return 2 * C * op_pitch(D) + 2 * C * P_PITCH; }    // K and P
__host__ __device__ constexpr long long ops_bytes(int D) { return first_bytes(D) + second_bytes(D); }

// log(1 + exp(v)) from the hardware's exponential and logarithm; where exp(-|v|) is small its series, so that slow decays keep
// their relative precision
__device__ __forceinline__ float fast_softplus(float v) {
    const float e = __expf(-fabsf(v));
    const float l = e < 0.01f ? e * (1.0f - e * (0.5f - e * (1.0f / 3.0f))) : __logf(1.0f + e);
    return l + fmaxf(v, 0.0f);
}
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
__device__ __forceinline__ float2 mul2(float2 a, float2 b) {
    float2 d;
    asm("{\n.reg .b64 ra, rb, rd;\n"
        "mov.b64 ra, {%2, %3};\nmov.b64 rb, {%4, %5};\n"
        "mul.rn.f32x2 rd, ra, rb;\n"
        "mov.b64 {%0, %1}, rd;\n}"
        : "=f"(d.x), "=f"(d.y) : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y));
    return d;
}
// v = hi + lo with both in bfloat16 (hi the rounded value, lo the rounded rest), two values at a time
__device__ __forceinline__ void split2(float u, float v, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16(u, v);
    lo = pack_bf16(u - __uint_as_float(hi << 16), v - __uint_as_float(hi & 0xffff0000u));
}

constexpr int BLOCKS = C / RB;
constexpr int YP = RB + 1;
// floats of shared memory of delta_chunk_make: k exp(g), q exp(g), k exp(t - g) and g [64][D + 4], the system, P and the inverse
// [64][64 + 4], the running sums at the blocks' starts [5][D], the factors between blocks [10][D], beta [64], three blocks of
// 16 x 16.  Once the operands are written, the tensor cores' tiles of k exp(G) and V take the place of the second to fourth,
// and the inverse's that of the system and P.
__host__ __device__ constexpr int make_floats(int D) { return 4 * C * (D + 4) + 3 * C * (C + 4) + 15 * D + C + 3 * RB * YP; }
// columns of V that fit there at a time
__host__ __device__ constexpr int v_group(int D) { return (2 * D - 4) / 16 * 16; }

__global__ void __launch_bounds__(MAKE_THREADS, 1) delta_chunk_make_kernel(const ChunkParams p) {
    extern __shared__ __align__(16) float sm[];
    __shared__ int slow[BLOCKS];
    const int D = p.s.D, DV = p.s.DV, DP = D + 4, H = p.s.H, CH = 2 * p.s.G * D + H * DV;
    constexpr int NP = C + 4;
    float* kd = sm;                    // [64][DP]: k exp(g)
    float* qd = kd + C * DP;           // q exp(g)
    float* ke = qd + C * DP;           // k exp(t - g)
    float* gs = ke + C * DP;           // g, in units of log2 (as every logarithm here)
    float* N = gs + C * DP;            // [64][NP]: diag(beta) A
    float* P = N + C * NP;
    float* M = P + C * NP;             // (1 + N)^-1
    float* base = M + C * NP;          // [5][D]: G at the start of each block, and at the chunk's end
    float* F = base + 5 * D;           // [10][D]
    float* beta = F + 10 * D;
    float* Y = beta + C;               // [3][16][YP]
    const int tid = threadIdx.x, item = blockIdx.x, h = blockIdx.y, g = h / (H / p.s.G);
    pdl_launch_dependents();
    pdl_wait();
    const int row0 = p.chunks[2 * item], n = p.chunks[2 * item + 1];
    const float* rows = p.s.qkv + (size_t)row0 * CH;
    const float* q_rows = rows + g * D;
    const float* k_rows = rows + (p.s.G + g) * D;

    // ---- the running sums inside the blocks: a thread per (channel, block)
    if (tid < BLOCKS) slow[tid] = 0;
    if (tid < C) beta[tid] = tid < n ? p.s.beta[(size_t)(row0 + tid) * H + h] : 0.0f;
    for (int i = tid; i < C * NP; i += MAKE_THREADS) { N[i] = 0.0f; P[i] = 0.0f; M[i] = 0.0f; }
    if (tid < BLOCKS * D) {
        const int d = tid % D, J = tid / D;
        float run = 0.0f, x[RB];
        if (p.s.z) {
            const float rate = p.s.rate[h] * LOG2E, bias = p.s.z_bias[(size_t)h * D + d];
            const float* z = p.s.z + (size_t)row0 * p.s.z_stride + (size_t)h * D + d;
#pragma unroll
            for (int t = 0; t < RB; ++t) x[t] = J * RB + t < n ? z[(size_t)(J * RB + t) * p.s.z_stride] : 0.0f;
#pragma unroll
            for (int t = 0; t < RB; ++t) x[t] = J * RB + t < n ? rate * fast_softplus(x[t] + bias) : 0.0f;
        } else {
            const float* ld = p.s.log_decay + (size_t)row0 * H + h;
#pragma unroll
            for (int t = 0; t < RB; ++t) x[t] = J * RB + t < n ? ld[(size_t)(J * RB + t) * H] * LOG2E : 0.0f;
        }
#pragma unroll
        for (int t = 0; t < RB; ++t) { run += x[t]; gs[(J * RB + t) * DP + d] = run; }
    }
    __syncthreads();
    if (tid < D) {
        float run = 0.0f;
        base[tid] = 0.0f;
#pragma unroll
        for (int J = 0; J < BLOCKS; ++J) {
            const float total = gs[(J * RB + RB - 1) * DP + tid];
            if (-total > GROW_LIMIT) slow[J] = 1;                       // every writer writes the same
            run += total;
            base[(J + 1) * D + tid] = run;
        }
    }
    __syncthreads();
    for (int i = tid; i < 10 * D; i += MAKE_THREADS) {
        const int pair = i / D, d = i - pair * D;
        const int I = pair >= 6 ? 3 : pair >= 3 ? 2 : pair >= 1 ? 1 : 0, J = pair - I * (I + 1) / 2;
        F[i] = ex2(fminf(base[I * D + d] - base[(J + 1) * D + d], GROW_LIMIT));
    }
    const int per_row = D / 4;
    for (int i = tid; i < C * per_row; i += MAKE_THREADS) {
        const int r = i / per_row, d = (i - r * per_row) * 4;
        float4 q4 = make_float4(0.0f, 0.0f, 0.0f, 0.0f), k4 = q4;
        if (r < n) { q4 = load4(q_rows + (size_t)r * CH + d); k4 = load4(k_rows + (size_t)r * CH + d); }
        const float4 g4 = load4(gs + r * DP + d), t4 = load4(gs + (r / RB * RB + RB - 1) * DP + d);
        const float4 f = make_float4(ex2(g4.x), ex2(g4.y), ex2(g4.z), ex2(g4.w));
        *reinterpret_cast<float4*>(kd + r * DP + d) = make_float4(k4.x * f.x, k4.y * f.y, k4.z * f.z, k4.w * f.w);
        *reinterpret_cast<float4*>(qd + r * DP + d) = make_float4(q4.x * f.x, q4.y * f.y, q4.z * f.z, q4.w * f.w);
        *reinterpret_cast<float4*>(ke + r * DP + d) =
            make_float4(k4.x * ex2(t4.x - g4.x), k4.y * ex2(t4.y - g4.y), k4.z * ex2(t4.z - g4.z), k4.w * ex2(t4.w - g4.w));
    }
    __syncthreads();

    // ---- A and P: two warps per pair of blocks, a thread has rows i, i + 8 and columns j, j + 8 of it
    const int warp = tid >> 5, lane = tid & 31;
    for (int job = warp; job < 20; job += MAKE_THREADS / 32) {
        const int pair = job >> 1;
        const int I = pair >= 6 ? 3 : pair >= 3 ? 2 : pair >= 1 ? 1 : 0, J = pair - I * (I + 1) / 2;
        const int i0 = I * RB + (lane >> 2), j0 = J * RB + (job & 1) * 4 + (lane & 3);
        float a[2][2], b[2][2];
        if (I == J && slow[I]) {
            for (int u = 0; u < 2; ++u)
                for (int v = 0; v < 2; ++v) {
                    const int r = i0 + 8 * u, c = j0 + 8 * v;
                    float sa = 0.0f, sb = 0.0f;
                    if (c <= r && r < n)
                        for (int d = 0; d < D; ++d) {
                            const float x = k_rows[(size_t)c * CH + d] * ex2(gs[r * DP + d] - gs[c * DP + d]);
                            sa = fmaf(k_rows[(size_t)r * CH + d], x, sa);
                            sb = fmaf(q_rows[(size_t)r * CH + d], x, sb);
                        }
                    a[u][v] = sa; b[u][v] = sb;
                }
        } else {
            float2 sa[2][2], sb[2][2];
#pragma unroll
            for (int u = 0; u < 2; ++u)
#pragma unroll
                for (int v = 0; v < 2; ++v) sa[u][v] = sb[u][v] = make_float2(0.0f, 0.0f);
            const float* f = F + pair * D;
#pragma unroll 2
            for (int d = 0; d < D; d += 4) {
                const float4 f4 = load4(f + d);
                float2 x[2][2];                                   // the two columns' keys with the factor between the blocks
#pragma unroll
                for (int v = 0; v < 2; ++v) {
                    const float4 e = load4(ke + (j0 + 8 * v) * DP + d);
                    x[v][0] = mul2(make_float2(e.x, e.y), make_float2(f4.x, f4.y));
                    x[v][1] = mul2(make_float2(e.z, e.w), make_float2(f4.z, f4.w));
                }
#pragma unroll
                for (int u = 0; u < 2; ++u) {
                    const float4 k4 = load4(kd + (i0 + 8 * u) * DP + d), q4 = load4(qd + (i0 + 8 * u) * DP + d);
#pragma unroll
                    for (int v = 0; v < 2; ++v) {
                        sa[u][v] = fma2(make_float2(k4.x, k4.y), x[v][0], sa[u][v]);
                        sb[u][v] = fma2(make_float2(q4.x, q4.y), x[v][0], sb[u][v]);
                        sa[u][v] = fma2(make_float2(k4.z, k4.w), x[v][1], sa[u][v]);
                        sb[u][v] = fma2(make_float2(q4.z, q4.w), x[v][1], sb[u][v]);
                    }
                }
            }
#pragma unroll
            for (int u = 0; u < 2; ++u)
#pragma unroll
                for (int v = 0; v < 2; ++v) { a[u][v] = sa[u][v].x + sa[u][v].y; b[u][v] = sb[u][v].x + sb[u][v].y; }
        }
#pragma unroll
        for (int u = 0; u < 2; ++u)
#pragma unroll
            for (int v = 0; v < 2; ++v) {
                const int r = i0 + 8 * u, c = j0 + 8 * v;
                if (c < r) N[r * NP + c] = beta[r] * a[u][v];
                if (c <= r) P[r * NP + c] = b[u][v];
            }
    }
    __syncthreads();

    const size_t at = (size_t)item * H + h;
    uint8_t* ops = p.ops + at * ops_bytes(D);
    const int pitch = op_pitch(D), op = C * pitch;
    if (tid < C) {
        // ---- the inverse's diagonal blocks, a column per thread
        const int J = tid / RB, c = tid % RB;
        float m[RB];
#pragma unroll
        for (int i = 0; i < RB; ++i) {
            float sum = 0.0f;
#pragma unroll
            for (int j = 0; j < i; ++j) sum = fmaf(N[(J * RB + i) * NP + J * RB + j], m[j], sum);
            m[i] = i == c ? 1.0f : i > c ? -sum : 0.0f;
            M[(J * RB + i) * NP + J * RB + c] = m[i];
        }
    } else {
        // ---- the operands that need no inverse
        const int w = tid - C, step = MAKE_THREADS - C;
        auto put = [&](uint8_t* to, int rest, float4 v) {              // four elements, the rests `rest` bytes behind
            uint32_t h0, l0, h1, l1;
            split2(v.x, v.y, h0, l0);
            split2(v.z, v.w, h1, l1);
            *reinterpret_cast<uint2*>(to) = make_uint2(h0, h1);
            *reinterpret_cast<uint2*>(to + rest) = make_uint2(l0, l1);
        };
        for (int e = w; e < C * per_row; e += step) {
            const int i = e / per_row, d = (e - i * per_row) * 4, J = i / RB;
            const float4 q4 = load4(qd + i * DP + d), k4 = load4(ke + i * DP + d);
            const float4 b4 = load4(base + J * D + d), n4 = load4(base + (J + 1) * D + d), l4 = load4(base + BLOCKS * D + d);
            uint8_t* to = ops + 2 * op + i * pitch + d * 2;
            put(to, op, make_float4(q4.x * ex2(b4.x), q4.y * ex2(b4.y), q4.z * ex2(b4.z), q4.w * ex2(b4.w)));
            put(to + 2 * op, op, make_float4(k4.x * ex2(l4.x - n4.x), k4.y * ex2(l4.y - n4.y), k4.z * ex2(l4.z - n4.z), k4.w * ex2(l4.w - n4.w)));
        }
        for (int e = w; e < C * C / 4; e += step) {
            const int i = e / (C / 4), j = e % (C / 4) * 4;
            put(ops + 6 * op + i * P_PITCH + j * 2, C * P_PITCH, load4(P + i * NP + j));
        }
        for (int d = w; d < D; d += step) p.last[at * D + d] = ex2(base[BLOCKS * D + d]);
    }
    __syncthreads();
    // ---- the blocks below, `apart` blocks from the diagonal
    for (int apart = 1; apart < BLOCKS; ++apart) {
        for (int e = tid; e < (BLOCKS - apart) * RB * RB; e += MAKE_THREADS) {
            const int J = e / (RB * RB), I = J + apart, i = e / RB % RB, j = e % RB;
            const float* nr = N + (I * RB + i) * NP;
            float sum = 0.0f;
            for (int k = J * RB; k < I * RB; k += 4) {
                const float4 a = load4(nr + k);
                const float* mc = M + k * NP + J * RB + j;
                sum = fmaf(a.x, mc[0], sum); sum = fmaf(a.y, mc[NP], sum); sum = fmaf(a.z, mc[2 * NP], sum); sum = fmaf(a.w, mc[3 * NP], sum);
            }
            Y[(J * RB + i) * YP + j] = sum;
        }
        __syncthreads();
        for (int e = tid; e < (BLOCKS - apart) * RB * RB; e += MAKE_THREADS) {
            const int J = e / (RB * RB), I = J + apart, i = e / RB % RB, j = e % RB;
            const float* mr = M + (I * RB + i) * NP + I * RB;
            float sum = 0.0f;
#pragma unroll
            for (int k = 0; k < RB; ++k) sum = fmaf(mr[k], Y[(J * RB + k) * YP + j], sum);
            M[(I * RB + i) * NP + J * RB + j] = -sum;
        }
        __syncthreads();
    }
    // ---- [W | U0] = M diag(beta) [k exp(G) | V] on the tensor cores
    uint8_t* t_tile = reinterpret_cast<uint8_t*>(N);                  // [hi, lo][64][P_PITCH]
    uint8_t* k_tile = reinterpret_cast<uint8_t*>(qd);                 // [hi, lo][64][pitch]
    uint8_t* v_tile = k_tile + 2 * op;                                // [hi, lo][64][v_pitch]
    const int group = min(v_group(D), (DV + 15) / 16 * 16), v_pitch = op_pitch(group);
    auto tile4 = [&](uint8_t* to, int rest, float4 v) {
        uint32_t h0, l0, h1, l1;
        split2(v.x, v.y, h0, l0);
        split2(v.z, v.w, h1, l1);
        *reinterpret_cast<uint2*>(to) = make_uint2(h0, h1);
        *reinterpret_cast<uint2*>(to + rest) = make_uint2(l0, l1);
    };
    for (int e = tid; e < C * C / 4; e += MAKE_THREADS) {
        const int i = e / (C / 4), j = e % (C / 4) * 4;
        const float4 m = load4(M + i * NP + j), b4 = load4(beta + j);
        tile4(t_tile + i * P_PITCH + j * 2, C * P_PITCH, make_float4(m.x * b4.x, m.y * b4.y, m.z * b4.z, m.w * b4.w));
    }
    for (int e = tid; e < C * per_row; e += MAKE_THREADS) {
        const int i = e / per_row, d = (e - i * per_row) * 4;
        const float4 k4 = load4(kd + i * DP + d), b4 = load4(base + i / RB * D + d);
        tile4(k_tile + i * pitch + d * 2, op, make_float4(k4.x * ex2(b4.x), k4.y * ex2(b4.y), k4.z * ex2(b4.z), k4.w * ex2(b4.w)));
    }
    float* u0 = p.u0 + at * C * DV;
    const float* v_rows = rows + 2 * p.s.G * D + (size_t)h * DV;
    const int row_tile = warp & 3, r0 = row_tile * 16 + (lane >> 2), nc = (lane & 3) * 2;
    const uint32_t ta = smem_u32(t_tile) + (row_tile * 16 + (lane & 15)) * P_PITCH + (lane >> 4) * 16;
    for (int v0 = 0; v0 < DV; v0 += group) {
        const int quads = group / 4;
        for (int e = tid; e < C * quads; e += MAKE_THREADS) {
            const int i = e / quads, c = (e - i * quads) * 4;
            float x[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
            for (int u = 0; u < 4; ++u)
                if (i < n && v0 + c + u < DV) x[u] = v_rows[(size_t)i * CH + v0 + c + u];
            tile4(v_tile + i * v_pitch + c * 2, C * v_pitch, make_float4(x[0], x[1], x[2], x[3]));
        }
        __syncthreads();
        const int w_tiles = v0 == 0 ? D / 16 : 0, all = w_tiles + group / 16;
        for (int ct = warp >> 2; ct < all; ct += MAKE_THREADS / 128) {
            const bool is_w = ct < w_tiles;
            const int col = (is_w ? ct : ct - w_tiles) * 16, bp = is_w ? pitch : v_pitch;
            const uint32_t b_hi = smem_u32(is_w ? k_tile : v_tile) + col * 2, b_lo = b_hi + C * bp;
            float acc[2][4], rest[2][4];
#pragma unroll
            for (int u = 0; u < 2; ++u)
#pragma unroll
                for (int i = 0; i < 4; ++i) acc[u][i] = rest[u][i] = 0.0f;
            for (int ks = 0; ks <= row_tile; ++ks) {                  // M is lower triangular
                uint32_t a[4], l[4], b0, b1, b2, b3, c0, c1, c2, c3;
                ldmatrix_x4(ta + ks * 32, a[0], a[1], a[2], a[3]);
                ldmatrix_x4(ta + C * P_PITCH + ks * 32, l[0], l[1], l[2], l[3]);
                const int from = (ks * 16 + (lane & 7) + (((lane >> 3) & 1) << 3)) * bp + (lane >> 4) * 16;
                ldmatrix_x4_trans(b_hi + from, b0, b1, b2, b3);
                ldmatrix_x4_trans(b_lo + from, c0, c1, c2, c3);
                mma_bf16(acc[0], a[0], a[1], a[2], a[3], b0, b1);
                mma_bf16(acc[1], a[0], a[1], a[2], a[3], b2, b3);
                mma_bf16(rest[0], l[0], l[1], l[2], l[3], b0, b1);
                mma_bf16(rest[1], l[0], l[1], l[2], l[3], b2, b3);
                mma_bf16(rest[0], a[0], a[1], a[2], a[3], c0, c1);
                mma_bf16(rest[1], a[0], a[1], a[2], a[3], c2, c3);
            }
#pragma unroll
            for (int u = 0; u < 2; ++u)
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    const int i = r0 + half * 8, c = col + u * 8 + nc;
                    const float x = acc[u][2 * half] + rest[u][2 * half], y = acc[u][2 * half + 1] + rest[u][2 * half + 1];
                    if (is_w) {
                        uint32_t hi, lo;
                        split2(x, y, hi, lo);
                        *reinterpret_cast<uint32_t*>(ops + i * pitch + c * 2) = hi;
                        *reinterpret_cast<uint32_t*>(ops + op + i * pitch + c * 2) = lo;
                    } else if (v0 + c < DV) {                         // DV is even: a pair is inside or outside
                        *reinterpret_cast<float2*>(u0 + (size_t)i * DV + v0 + c) = make_float2(x, y);
                    }
                }
        }
        if (v0 + group < DV) __syncthreads();                          // the tile is read before the next columns take its place
    }
}

constexpr int S_PITCH = NC * 2 + 16;   // bytes of a row of the S and U tiles
// W and Q of two chunks, K and P of one, S, U (each as two bfloat16 tiles), three barriers
__host__ __device__ constexpr int walk_smem(int D) { return 2 * first_bytes(D) + second_bytes(D) + 2 * D * S_PITCH + 2 * C * S_PITCH + 32; }

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
    uint64_t* bars = reinterpret_cast<uint64_t*>(smem + (u_tiles - base) + 2 * C * S_PITCH);       // W and Q (two of them), K and P
    auto load_first = [&](int c) {                             // by one thread
        const int buf = c & 1;
        ph_mbar::arrive_expect_tx(&bars[buf], (uint32_t)first_bytes(D));
        ph_mbar::bulk_copy(smem + buf * first_bytes(D), p.ops + ((size_t)(first + c) * H + h) * ops_bytes(D), (uint32_t)first_bytes(D), &bars[buf]);
    };
    auto load_second = [&](int c) {
        ph_mbar::arrive_expect_tx(&bars[2], (uint32_t)second_bytes(D));
        ph_mbar::bulk_copy(smem + 2 * first_bytes(D), p.ops + ((size_t)(first + c) * H + h) * ops_bytes(D) + first_bytes(D), (uint32_t)second_bytes(D), &bars[2]);
    };
    if (threadIdx.x == 0) {
        for (int i = 0; i < 3; ++i) ph_mbar::init(&bars[i], 1);
        ph_mbar::fence_init();
        load_first(0);
    }
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
        if (c == 0) __syncthreads();                           // the barriers are set up
        bool late = !ph_mbar::wait(&bars[c & 1], (c >> 1) & 1, p.error_flag, PH_ERR_WAIT_DELTA);
        if (__syncthreads_or(late)) return;                    // W, Q and S are there; everyone is done with the last chunk's K, P and U
        if (threadIdx.x == 0) {
            load_second(c);
            if (c + 1 < chunks) load_first(c + 1);
        }
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
        late = !ph_mbar::wait(&bars[2], c & 1, p.error_flag, PH_ERR_WAIT_DELTA);
        if (__syncthreads_or(late)) {                          // U, K and P are there; everyone is done with S
            if (threadIdx.x == 0 && c + 1 < chunks) ph_mbar::wait(&bars[(c + 1) & 1], ((c + 1) >> 1) & 1, p.error_flag, PH_ERR_WAIT_DELTA);
            return;                                            // (nothing of this block's is in flight any more)
        }
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
PH_EXPORT long long ph_delta_chunk_scratch_bytes(int D, int DV) { return (ops_bytes(D) + 4LL * C * DV + 4LL * D + 255) / 256 * 256; }

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
    p.ops = static_cast<uint8_t*>(scratch);
    p.u0 = reinterpret_cast<float*>(p.ops + units * ops_bytes(D));
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
                                  int DV, int K, float* o, int* error_flag, cudaStream_t stream) {
    if (!rows || !state || !seg_start || !seg_slot || !seg_chunks || !o || !error_flag || S < 1 || K < 1 || splits < 1 || !valid_dtype(rows_dtype) || ((uintptr_t)o & 7))
        return fail(PH_ERR_ARG, "delta_chunk_walk: bad arguments (S %d)", S);
    ChunkParams p = {};
    if (int rc = fill(p, chunks, n_chunks, seg_chunks, const_cast<void*>(scratch), H, G, D, DV)) return rc;
    p.s.rows = rows; p.s.splits = splits; p.s.split_stride = split_stride; p.s.width = width; p.s.state = state; p.s.state_stride = state_stride;
    p.s.conv_at = conv_at; p.s.seg_start = seg_start; p.s.seg_slot = seg_slot; p.s.o = o; p.s.K = K; p.error_flag = error_flag;
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
