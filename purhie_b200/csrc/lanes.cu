// A residual stream of several lanes: S rows of E float32 numbers per token.
//
//   lanes_rmsnorm   for every token (or the gathered ones), in one pass over its lanes:
//                       X'[t] = sum_s mix[s][t] X[s] + out[t] y         (y the addend, its partial sums added up; without
//                                                                        an addend X' = X)
//                       u     = sum_t in[t] X'[t]                        (in null: the plain sum)
//                       rows  = u * rsqrt(mean(u^2) + eps) * w           (w null: u itself)
//                   X' goes to `dst` (which may be `src`: a thread reads all lanes of its columns before it writes them).
//                   Before the first update every lane is the same row: `src` then has a lane stride of 0.
// Everything is float32; the sums over lanes run in the order of the lanes, the row's sum of squares in an order that
// depends on E and the launch shape only.
//
// Few rows (decoding): a row is spread over a cluster of up to eight CTAs that add up their sums of squares through
// distributed shared memory, so that the latency of one CTA reading S rows is not the kernel's time.
#include "common.cuh"

#include <cooperative_groups.h>
#include <math.h>

namespace {

using namespace ph;

struct LaneParams {
    const float* src; long long src_row, src_lane;
    float* dst;                                       // [T][S][E] or null
    const void* add; int splits; long long split_stride;
    const float* mix; const float* out; const float* in;
    const float* weight; float eps;
    const int32_t* rows;
    void* y;
    int E, S;
};

// SM: lanes held in registers (S <= SM; the surplus is never touched).  IT quads of columns per thread.  PARTS: partial
// sums of the addend in flight.  The grid is rows x CTAs of a row (blockIdx.x % cta_per_row).
template <typename TY, int SM, int IT, int PARTS>
__global__ void __launch_bounds__(512) lanes_rmsnorm_vec_kernel(const LaneParams p, int ctas) {
    namespace cg = cooperative_groups;
    __shared__ float scratch[32];
    __shared__ float total;
    pdl_launch_dependents();
    const int r = blockIdx.x / ctas, rank = blockIdx.x % ctas;
    const int t = p.rows ? p.rows[r] : r;
    const int quads = p.E / 4, per_cta = (quads + ctas - 1) / ctas;
    const int q0 = rank * per_cta, q1 = min(quads, q0 + per_cta);
    // weights: not written by any kernel of the step
    float in[SM], out[SM], mix[SM][SM];
#pragma unroll
    for (int s = 0; s < SM; ++s) {
        in[s] = s < p.S ? (p.in ? p.in[s] : 1.0f) : 0.0f;
        out[s] = s < p.S && p.add ? p.out[s] : 0.0f;
#pragma unroll
        for (int u = 0; u < SM; ++u) mix[s][u] = s < p.S && u < p.S && p.add ? p.mix[s * p.S + u] : 0.0f;
    }
    pdl_wait();
    float4 u[IT];
    float ss = 0.0f;
#pragma unroll
    for (int it = 0; it < IT; ++it) {
        const int q = q0 + it * blockDim.x + threadIdx.x;
        u[it] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (q >= q1) continue;
        float4 x[SM];
#pragma unroll
        for (int s = 0; s < SM; ++s)
            if (s < p.S) x[s] = *reinterpret_cast<const float4*>(p.src + (size_t)t * p.src_row + (size_t)s * p.src_lane + 4 * q);
        if (p.add) {
            const float* a = static_cast<const float*>(p.add) + (size_t)t * p.E + 4 * q;
            float4 y = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            for (int s0 = 0; s0 < p.splits; s0 += PARTS) {
                float4 part[PARTS];
#pragma unroll
                for (int j = 0; j < PARTS; ++j)
                    part[j] = s0 + j < p.splits ? *reinterpret_cast<const float4*>(a + (size_t)(s0 + j) * p.split_stride) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
                for (int j = 0; j < PARTS; ++j)
                    if (s0 + j < p.splits) { y.x += part[j].x; y.y += part[j].y; y.z += part[j].z; y.w += part[j].w; }
            }
#pragma unroll
            for (int v = 0; v < SM; ++v) {
                if (v >= p.S) break;
                float4 n = make_float4(out[v] * y.x, out[v] * y.y, out[v] * y.z, out[v] * y.w);
#pragma unroll
                for (int s = 0; s < SM; ++s)
                    if (s < p.S) {
                        n.x = fmaf(mix[s][v], x[s].x, n.x); n.y = fmaf(mix[s][v], x[s].y, n.y);
                        n.z = fmaf(mix[s][v], x[s].z, n.z); n.w = fmaf(mix[s][v], x[s].w, n.w);
                    }
                if (p.dst) *reinterpret_cast<float4*>(p.dst + ((size_t)t * p.S + v) * p.E + 4 * q) = n;
                u[it].x = fmaf(in[v], n.x, u[it].x); u[it].y = fmaf(in[v], n.y, u[it].y);
                u[it].z = fmaf(in[v], n.z, u[it].z); u[it].w = fmaf(in[v], n.w, u[it].w);
            }
        } else {
#pragma unroll
            for (int s = 0; s < SM; ++s)
                if (s < p.S) {
                    u[it].x = fmaf(in[s], x[s].x, u[it].x); u[it].y = fmaf(in[s], x[s].y, u[it].y);
                    u[it].z = fmaf(in[s], x[s].z, u[it].z); u[it].w = fmaf(in[s], x[s].w, u[it].w);
                }
        }
        ss += (u[it].x * u[it].x + u[it].y * u[it].y) + (u[it].z * u[it].z + u[it].w * u[it].w);
    }
    float inv = 1.0f;
    if (p.weight) {
        float sum = block_sum_any(ss, scratch);
        if (ctas > 1) {
            cg::cluster_group cluster = cg::this_cluster();
            if (threadIdx.x == 0) total = sum;
            cluster.sync();
            sum = 0.0f;
            for (int c = 0; c < ctas; ++c) sum += *cluster.map_shared_rank(&total, c);
            cluster.sync();                           // nobody leaves while its sum may still be read
        }
        inv = rsqrtf(sum / (float)p.E + p.eps);
    }
#pragma unroll
    for (int it = 0; it < IT; ++it) {
        const int q = q0 + it * blockDim.x + threadIdx.x;
        if (q >= q1) continue;
        float v[4] = {u[it].x * inv, u[it].y * inv, u[it].z * inv, u[it].w * inv};
        if (p.weight) {
            const float4 w = *reinterpret_cast<const float4*>(p.weight + 4 * q);
            v[0] *= w.x; v[1] *= w.y; v[2] *= w.z; v[3] *= w.w;
        }
        store4(static_cast<TY*>(p.y) + (size_t)r * p.E + 4 * q, v);
    }
}

// Any width, any number of lanes up to MAX_LANES, any type of the addend: a block per row, u in shared memory.
constexpr int MAX_LANES = 32;
template <typename TA, typename TY>
__global__ void lanes_rmsnorm_kernel(const LaneParams p) {
    extern __shared__ float row[];                    // [E]
    __shared__ float scratch[32];
    pdl_launch_dependents();
    pdl_wait();
    const int r = blockIdx.x, t = p.rows ? p.rows[r] : r;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < p.E; i += blockDim.x) {
        float x[MAX_LANES];
        for (int s = 0; s < p.S; ++s) x[s] = p.src[(size_t)t * p.src_row + (size_t)s * p.src_lane + i];
        float u = 0.0f;
        if (p.add) {
            const TA* a = static_cast<const TA*>(p.add) + (size_t)t * p.E + i;
            float y = 0.0f;
            for (int s = 0; s < p.splits; ++s) y += to_float<TA>(a[(size_t)s * p.split_stride]);
            for (int v = 0; v < p.S; ++v) {
                float n = p.out[v] * y;
                for (int s = 0; s < p.S; ++s) n = fmaf(p.mix[s * p.S + v], x[s], n);
                if (p.dst) p.dst[((size_t)t * p.S + v) * p.E + i] = n;
                u = fmaf(p.in ? p.in[v] : 1.0f, n, u);
            }
        } else {
            for (int s = 0; s < p.S; ++s) u = fmaf(p.in ? p.in[s] : 1.0f, x[s], u);
        }
        row[i] = u;
        ss += u * u;
    }
    const float inv = p.weight ? rsqrtf(block_sum_any(ss, scratch) / (float)p.E + p.eps) : 1.0f;
    TY* y = static_cast<TY*>(p.y) + (size_t)r * p.E;
    for (int i = threadIdx.x; i < p.E; i += blockDim.x) y[i] = from_float<TY>(p.weight ? row[i] * inv * p.weight[i] : row[i]);
}

template <typename TY, int SM, int IT, int PARTS>
cudaError_t launch_vec(const LaneParams& p, int n, int ctas, int threads, cudaStream_t stream) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3((unsigned)n * ctas);
    cfg.blockDim = dim3(threads);
    cfg.stream = stream;
    cudaLaunchAttribute attr[2];
    int k = 0;
    if (pdl_enabled()) {
        attr[k].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr[k++].val.programmaticStreamSerializationAllowed = 1;
    }
    if (ctas > 1) {
        attr[k].id = cudaLaunchAttributeClusterDimension;
        attr[k].val.clusterDim.x = ctas; attr[k].val.clusterDim.y = 1; attr[k].val.clusterDim.z = 1;
        ++k;
    }
    cfg.attrs = attr;
    cfg.numAttrs = k;
    return cudaLaunchKernelEx(&cfg, lanes_rmsnorm_vec_kernel<TY, SM, IT, PARTS>, p, ctas);
}

template <typename TY, int SM>
cudaError_t launch_vec_shape(const LaneParams& p, int n, int ctas, int threads, int it, cudaStream_t stream) {
    const bool one = !p.add || p.splits == 1;
#define SHAPE(IT) (one ? launch_vec<TY, SM, IT, 1>(p, n, ctas, threads, stream) : launch_vec<TY, SM, IT, 8>(p, n, ctas, threads, stream))
    return it == 1 ? SHAPE(1) : it == 2 ? SHAPE(2) : SHAPE(4);
#undef SHAPE
}

}  // namespace

// src: lane s of token t at src + t * src_row + s * src_lane (src_lane 0: all lanes are one row).  dst [T][S][E] or null;
// add [splits][T][E] or null (then mix [S][S], indexed [from][to], and out [S] are not read, and dst is not written).
// in [S] or null (ones); weight [E] or null.  rows: the n gathered token rows, or null for rows 0 .. n - 1.  y [n][E].
PH_EXPORT int ph_lanes_rmsnorm(const float* src, long long src_row, long long src_lane, float* dst, const void* add, int add_dtype,
                               int add_splits, long long add_split_stride, const float* mix, const float* out, const float* in,
                               const float* weight, float eps, const int32_t* rows, int n, int E, int S, void* y, int y_dtype,
                               cudaStream_t stream) {
    if (!src || !y || n < 0 || E < 1 || S < 1 || src_row < E || src_lane < 0 || (src_lane && src_lane < E) || !valid_dtype(y_dtype) ||
        (add && (!mix || !out || add_splits < 1 || !valid_dtype(add_dtype))))
        return fail(PH_ERR_ARG, "lanes_rmsnorm: bad arguments (rows %d, width %d, lanes %d)", n, E, S);
    if (S > MAX_LANES) return fail(PH_ERR_UNSUPPORTED, "lanes_rmsnorm: %d lanes exceed the supported %d", S, MAX_LANES);
    if (rows && dst && add) return fail(PH_ERR_ARG, "lanes_rmsnorm: a gathered launch cannot write the lanes back");
    if (n == 0) return PH_OK;
    LaneParams p;
    p.src = src; p.src_row = src_row; p.src_lane = src_lane; p.dst = add ? dst : nullptr; p.add = add; p.splits = add_splits;
    p.split_stride = add_split_stride; p.mix = mix; p.out = out; p.in = in; p.weight = weight; p.eps = eps; p.rows = rows; p.y = y;
    p.E = E; p.S = S;
    const bool vec = S <= 8 && E % 4 == 0 && E <= 8192 && (!add || (add_dtype == PH_F32 && add_split_stride % 4 == 0)) && src_row % 4 == 0 &&
                     src_lane % 4 == 0 && (((uintptr_t)src | (uintptr_t)dst | (uintptr_t)add | (uintptr_t)weight | (uintptr_t)y) & 15) == 0;
    if (vec) {
        const int quads = E / 4;
        // few rows: a cluster per row with about a quad per thread; many rows: a CTA per row
        int ctas = 1;
        if (n <= 64) while (ctas < 8 && quads / ctas > 128) ctas *= 2;
        const int per_cta = (quads + ctas - 1) / ctas;
        int threads = (per_cta + 31) / 32 * 32;
        const int most = n > 64 ? 256 : 512;
        if (threads > most) threads = most;
        int it = (per_cta + threads - 1) / threads;
        if (it > 4) { threads = 512; it = (per_cta + threads - 1) / threads; }
        cudaError_t e;
#define LANES(SM) PH_DISPATCH(y_dtype, TY, e = (launch_vec_shape<TY, SM>(p, n, ctas, threads, it, stream)))
        if (S <= 2) LANES(2); else if (S == 3) LANES(3); else if (S == 4) LANES(4); else LANES(8);
#undef LANES
        if (e != cudaSuccess) return fail(PH_ERR_LAUNCH, "lanes_rmsnorm: %s", cudaGetErrorString(e));
        return check_launch("lanes_rmsnorm");
    }
    const size_t smem = (size_t)E * sizeof(float);
    if (smem > 200 * 1024) return fail(PH_ERR_UNSUPPORTED, "lanes_rmsnorm: width %d exceeds the supported 51200", E);
    const int threads = E >= 1024 ? 256 : 128;
#define PLAIN(TA, TY)                                                                                                             \
    do {                                                                                                                          \
        auto kern = lanes_rmsnorm_kernel<TA, TY>;                                                                                 \
        if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                 \
        launch_overlapped(kern, dim3(n), dim3(threads), smem, stream, p);                                                         \
    } while (0)
    PH_DISPATCH(add ? add_dtype : PH_F32, TA, PH_DISPATCH(y_dtype, TY, PLAIN(TA, TY)));
#undef PLAIN
    return check_launch("lanes_rmsnorm");
}
