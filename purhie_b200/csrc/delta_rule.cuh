// What the two forms of the delta rule's recurrence (delta_rule.cu, delta_chunk.cu) share.
#pragma once

#include "common.cuh"

namespace ph_delta {

using namespace ph;

__device__ __forceinline__ float softplus(float v) { return log1pf(expf(-fabsf(v))) + fmaxf(v, 0.0f); }

struct ScanParams {
    const float* qkv;                                           // [T, 2 G D + H DV]: what delta_prepare left
    const float* beta;                                          // [T, H]
    const float* log_decay;                                     // [T, H]: one decay per head, or null
    const float* z; long long z_stride; const float* z_bias;    // [T, H D] and [H D]: the logits of a decay per channel, or null
    const float* rate;                                          // [H]: -exp(A_log)
    const void* rows; int splits; long long split_stride, width;        // the projections' rows, for the convolution's inputs
    float* state; long long state_stride, conv_at;
    const int32_t* seg_start; const int32_t* seg_slot;
    float* o;                                                   // [T, H DV]
    int H, G, D, DV, K;
    int rows_from, rows_to;                                     // this launch takes the requests whose portion has rows_from .. rows_to rows
};

// The last K - 1 inputs of the convolution, oldest first: from this step's rows, or moved up from what was kept.  The
// channels are spread over the `blocks` groups of `threads` threads that work on a request.
template <typename TI>
__device__ __forceinline__ void move_conv_inputs(const ScanParams& p, float* st, int row0, int n, int block, int blocks, int thread, int threads) {
    const int CH = 2 * p.G * p.D + p.H * p.DV;
    float* past = st + p.conv_at;
    const TI* src = static_cast<const TI*>(p.rows);
    for (int c = block * threads + thread; c < CH; c += blocks * threads)
        for (int k = 0; k < p.K - 1; ++k) {
            const int i = n - (p.K - 1) + k;
            float v;
            if (i >= 0) {
                const TI* at = src + (size_t)(row0 + i) * p.width + c;
                v = to_float<TI>(*at);
                for (int s = 1; s < p.splits; ++s) v += to_float<TI>(at[(size_t)s * p.split_stride]);
            } else {
                v = past[(size_t)(k + n) * CH + c];
            }
            past[(size_t)k * CH + c] = v;
        }
}

}  // namespace ph_delta
