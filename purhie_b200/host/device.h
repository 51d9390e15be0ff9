// Device memory, scratch space and the kernel libraries, as the host library sees them.
//
// All device memory is plain cudaMalloc memory owned by a DeviceBuffer; a Workspace hands out named scratch
// tensors that keep their address from step to step (what a captured CUDA graph needs).  The kernels live in
// separate shared objects (libpurhie_core.so, libpurhie_flash.so, libpurhie_gemm100.so) that are opened by
// need from the folder this library was loaded from: a float32 model never touches the tensor-core libraries.
// A missing library is an error that says how to build it; there is no other implementation to fall back to.
#pragma once

#include <cuda_runtime.h>

#include <map>
#include <memory>
#include <string>
#include <vector>

#include "common.h"

namespace qe {

#define QE_CUDA(expr)                                                                                  \
    do {                                                                                               \
        cudaError_t qe_e_ = (expr);                                                                    \
        if (qe_e_ != cudaSuccess)                                                                      \
            throw ::qe::Error(qe_e_ == cudaErrorMemoryAllocation ? ::qe::kOutOfMemory : ::qe::kKernelLaunch, \
                              std::string(#expr) + ": " + cudaGetErrorString(qe_e_));                 \
    } while (0)

// Owns one cudaMalloc allocation.
class QE_API DeviceBuffer {
public:
    DeviceBuffer() = default;
    explicit DeviceBuffer(size_t bytes);
    ~DeviceBuffer();
    DeviceBuffer(const DeviceBuffer&) = delete;
    DeviceBuffer& operator=(const DeviceBuffer&) = delete;
    DeviceBuffer(DeviceBuffer&& o) noexcept : p_(o.p_), n_(o.n_) { o.p_ = nullptr; o.n_ = 0; }
    DeviceBuffer& operator=(DeviceBuffer&& o) noexcept;
    void* data() const { return p_; }
    size_t bytes() const { return n_; }
    void reset();
private:
    void* p_ = nullptr;
    size_t n_ = 0;
};

// Page-locked host memory.
class QE_API PinnedBuffer {
public:
    PinnedBuffer() = default;
    explicit PinnedBuffer(size_t bytes);
    ~PinnedBuffer();
    PinnedBuffer(const PinnedBuffer&) = delete;
    PinnedBuffer& operator=(const PinnedBuffer&) = delete;
    void* data() const { return p_; }
    size_t bytes() const { return n_; }
    void ensure(size_t bytes);          // grows (contents are lost)
private:
    void* p_ = nullptr;
    size_t n_ = 0;
};

// Device tensors that somebody keeps for good (weights and what parts derive from them).
class QE_API DeviceArena {
public:
    Tensor alloc(DType dtype, std::vector<int64_t> shape);
    void release(const Tensor& t);      // give one allocation back early (a temporary made while binding)
    size_t bytes() const { return bytes_; }
private:
    std::map<void*, DeviceBuffer> bufs_;
    size_t bytes_ = 0;
};

// Scratch tensors by name, reused from step to step and grown on demand.  A tensor of a given name keeps its
// address as long as requests do not outgrow it; `frozen` turns growth into an error (a captured graph points
// at these addresses).
class QE_API Workspace {
public:
    Workspace() = default;
    Tensor get(const std::string& name, std::vector<int64_t> shape, DType dtype);
    size_t bytes() const;
    bool frozen = false;
    cudaStream_t stream = nullptr;      // growing waits for this stream before the old block is freed
private:
    std::map<std::string, DeviceBuffer> bufs_;
};

// ---- kernel libraries ---------------------------------------------------------------------------------------
// Launcher prototypes (see the .cu files under csrc/).  Every launcher returns 0 or a status with a text.
struct CoreKernels {
    int (*embed_gather)(const void*, int, const int32_t*, float*, int, int, int, cudaStream_t);
    int (*add_rmsnorm)(float*, const void*, int, int, long long, const float*, float, const int32_t*, int, int, void*, int,
                       int, cudaStream_t);
    int (*swiglu)(const void*, int, int, long long, void*, int, int, int, cudaStream_t);
    int (*cast)(const void*, int, void*, int, long long, cudaStream_t);
    int (*qk_norm_rope_kv_write)(const void*, int, int, long long, const float*, const float*, const float*, float,
                                 const float*, int, int, const int32_t*, const int32_t*, void*, int, void*, void*, int,
                                 long long, int, int, int, int, int, int, const float*, int, int, float, int, float*,
                                 const float*, int, cudaStream_t);
    // the same over rows that go on behind v, with the gate's logits there added up and stored
    int (*qk_norm_rope_gate_kv_write)(const void*, int, int, long long, const float*, const float*, const float*, float,
                                      const float*, int, int, const int32_t*, const int32_t*, void*, int, void*, void*, int,
                                      long long, int, int, int, int, int, int, const float*, int, int, float, int, float*,
                                      const float*, int, long long, void*, cudaStream_t);
    int (*add_weight_sumsq)(float*, const void*, int, int, long long, const float*, int, int, void*, int, float*, int, cudaStream_t);
    int (*attention_generic)(const void*, int, const void*, const void*, int, long long, int, const int32_t*, int,
                             const int32_t*, const int32_t*, void*, int, int, int, int, int, int, float, int, int, int, cudaStream_t);
    int (*gemm_simple)(const void*, int, const void*, int, void*, int, int, int, int, cudaStream_t);
    int (*argmax)(const float*, int, int, int32_t*, void*, long long, cudaStream_t);   // several CTAs per row, with scratch
    long long (*argmax_scratch_bytes)(int);
    int (*sample_temperature)(const float*, int, int, const float*, const double*, float, int32_t*, cudaStream_t);
    int (*sample_chain)(const float*, int, int, const void*, int32_t*, cudaStream_t);
    int (*sample_chain_max_k)(void);
    int (*random_fill)(void*, int, long long, unsigned long long, int, double, double, cudaStream_t);
    // layer norm with the residual add and a transform of the addend in front; an embedding gather with a factor
    int (*add_layernorm)(float*, const void*, int, int, long long, const float*, const float*, float, float, const float*,
                         const float*, float, const int32_t*, int, int, void*, int, int, cudaStream_t);
    int (*embed_gather_scaled)(const void*, int, const int32_t*, float*, int, int, int, float, cudaStream_t);
    // gated activations by kind (0 silu, 1 clamped swish with alpha, limit, shift)
    int (*glu)(const void*, int, int, long long, void*, int, int, int, int, float, float, float, cudaStream_t);
    int (*glu_scaled)(const void*, int, int, long long, void*, int, int, int, int, float, float, float, const float*, const int32_t*,
                      cudaStream_t);     // with a factor per row in front of the activation
    // activations of one argument over plain rows (0 silu, 1 the square of relu)
    int (*unary_act)(const void*, int, int, long long, void*, int, long long, int, cudaStream_t);
    // gated linear attention: the decayed matrix state token by token with the head norm and gate behind it; two mixers'
    // outputs, each RMS-normed over the width, combined
    int (*decayed_scan)(const void*, const void*, const void*, const void*, int, long long, const float*, long long, const float*, float,
                        float, const float*, float, float*, long long, const int32_t*, const int32_t*, int, int, int, int, int,
                        const int32_t*, int, const int32_t*, float*, float*, float*, void*, const float*, int, int, cudaStream_t);
    // a float32 row RMS-normed over its whole width, times silu or sigmoid of a gate
    int (*rms_gate)(const float*, const float*, float, const void*, int, long long, int, void*, int, int, int, cudaStream_t);
    int (*rms_pair_mean)(const void*, int, int, long long, const float*, const void*, int, int, long long, const float*, float, float,
                         float*, int, int, cudaStream_t);
    // selective state-space mixer: convolution + silu, and the scan
    int (*causal_conv_silu)(const void*, int, long long, int, const float*, const float*, int, const float*, long long, long long,
                            const int32_t*, const int32_t*, const int32_t*, void*, int, int, cudaStream_t);
    int (*selective_scan)(const void*, const float*, const float*, const void*, long long, int, int, int, const float*,
                          const float*, const void*, long long, int, int, float*, long long, const int32_t*, const int32_t*, int,
                          const int32_t*, int, const int32_t*, float*, float*, void*, int, cudaStream_t);
    // routing: router logits and top-k (softmax over the chosen, or sigmoid scores with a correction and runs of experts),
    // sort by expert, products by expert, weighted sum (on top of a base addend)
    int (*route)(const void*, int, const float*, const float*, int, int, int, int, int32_t*, float*, int, const float*, int, int,
                 float, const float*, float*, cudaStream_t);
    int (*route_max_tiles)(int, int);
    int (*route_sort)(const int32_t*, int, int, int32_t*, int32_t*, int32_t*, int, int32_t*, cudaStream_t);
    int (*route_tile_rows)(int, int);          // the sort with every expert's rows at a multiple of the product's tile
    int (*route_sort_tiles)(const int32_t*, const float*, int, int, int, int32_t*, int32_t*, int32_t*, float*, cudaStream_t);
    int (*gemm_grouped)(const void*, int, const int32_t*, int, const void*, int, const int32_t*, int, void*, int, int, int,
                        cudaStream_t);
    int (*gemv_grouped)(const void*, int, const int32_t*, int, const void*, int, const int32_t*, int, void*, int, int, int,
                        cudaStream_t);
    int (*route_gather)(const void*, int, const int32_t*, int, void*, int, int, cudaStream_t);
    int (*route_combine)(const void*, int, const int32_t*, const float*, int, int, int, float*, const float*, int, long long, const float*,
                         cudaStream_t);
    // dynamic tanh with the residual add (two addends) in front; the stream re-started from [x | what the embedding gave]
    int (*add_dyntanh)(float*, const void*, int, int, long long, const void*, int, int, long long, const float*, const float*, const float*,
                       const int32_t*, int, int, void*, int, int, cudaStream_t);
    int (*concat_restart)(float*, const void*, int, int, long long, const void*, int, int, long long, const float*, const float*, void*, int,
                          int, int, cudaStream_t);
    // attention through a latent: norms, rotation and the cache row; the key expansion folded into q; the value expansion
    int (*latent_prepare)(const void*, int, long long, int, int, int, const float*, const float*, float, const float*, int, int,
                          const int32_t*, const int32_t*, void*, int, void*, int, long long, int, int, cudaStream_t);
    int (*latent_absorb)(const void*, int, long long, const void*, int, const float*, int, int, const int32_t*, void*, int, int, int, int, int,
                         int, cudaStream_t);
    int (*latent_expand)(const void*, int, const void*, int, const void*, int, long long, int, void*, int, int, int, int, int, cudaStream_t);
    int (*latent_gather)(const void*, int, long long, int, const int32_t*, int, const int32_t*, int, const int32_t*, const int32_t*, int, void*,
                         int, int, cudaStream_t);
    // attention with a sink in the softmax's denominator (the plain kernel); attention whose heads' scores are capped,
    // biased by the distance and mixed before the softmax, with the kernel that norms q and k over their whole width and
    // writes the cache rows in front of it
    // (the plain kernel: a sink, a distance bias and an output gate, each optional)
    int (*attention_generic_biased)(const void*, int, const void*, const void*, int, long long, int, const int32_t*, int,
                                    const int32_t*, const int32_t*, void*, int, int, int, int, int, int, float, int, int, int, const float*,
                                    const float*, const void*, long long, cudaStream_t);
    // (the same with a cap on the scores)
    int (*attention_generic_capped)(const void*, int, const void*, const void*, int, long long, int, const int32_t*, int,
                                    const int32_t*, const int32_t*, void*, int, int, int, int, int, int, float, int, int, int, const float*,
                                    const float*, const void*, long long, float, cudaStream_t);
    int (*attention_talking)(const void*, int, const void*, const void*, int, long long, int, const int32_t*, int, const int32_t*,
                             const int32_t*, void*, int, int, int, int, int, int, int, int, float, float, const float*, const float*,
                             const float*, const float*, const void*, int, long long, cudaStream_t);
    // the same attention on the tensor cores (bfloat16), a tile of 16 rows and all heads per CTA
    int (*attention_talking_mma)(const void*, const void*, const void*, long long, int, const int32_t*, int, const int32_t*, const int32_t*,
                                 const int32_t*, const int32_t*, int, void*, int, int, int, int, int, int, float, float, const float*,
                                 const float*, const float*, const float*, const void*, long long, int, int, float*, float*, cudaStream_t);
    int (*attention_talking_mma_supports)(int, int, int, int);
    int (*attention_talking_mma_ctas_per_sm)(int, int, int, int);
    int (*joint_norm_kv_write)(const void*, int, int, long long, long long, const float*, const float*, float, const int32_t*, void*, int,
                               void*, void*, int, long long, int, int, int, int, int, int, int, cudaStream_t);
    // the same with a bias, a rotation, a row's missing factor and the gate's logits
    int (*joint_norm_rope_kv_write)(const void*, int, int, long long, long long, const float*, const float*, float, const int32_t*, void*, int,
                                    void*, void*, int, long long, int, int, int, int, int, int, const float*, const float*, int, int,
                                    const int32_t*, int, const float*, int, int, float, void*, int, cudaStream_t);
    // a minimal gated recurrent unit over the rows of each request; the weighted sum of two mixers' outputs
    int (*min_gru_scan)(const void*, int, int, long long, long long, const float*, const float*, float*, const int32_t*, const int32_t*,
                        int, int, int, const int32_t*, int, const int32_t*, float*, void*, int, cudaStream_t);
    int (*pair_sum)(const void*, int, int, long long, float, const void*, int, int, long long, float, float*, long long, cudaStream_t);
    // add_rmsnorm with a factor on the addend
    int (*add_scaled_rmsnorm)(float*, const void*, int, int, long long, const float*, float, const int32_t*, int, int, void*, int, int, float,
                              cudaStream_t);
    // a residual of several lanes: the addend mixed in, the lanes read, the RMS norm of what was read
    int (*lanes_rmsnorm)(const float*, long long, long long, float*, const void*, int, int, long long, const float*, const float*, const float*,
                         const float*, float, const int32_t*, int, int, int, void*, int, cudaStream_t);
    // the second Mamba form: the scan token by token, the scan in chunks on the tensor cores, the gated norm in parts
    int (*ssd_scan)(const void*, const void*, int, long long, int, int, const float*, const float*, const float*, float*, long long,
                    const int32_t*, const int32_t*, int, int, int, int, int, int, int, int, float*, cudaStream_t);
    int (*ssd_chunk)(const void*, const void*, long long, int, int, const float*, const float*, const float*, float*, long long,
                     const int32_t*, const int32_t*, int, int, int, int, int, int, int, int, float*, cudaStream_t);
    int (*ssd_chunk_supports)(int, int, int);
    int (*gate_rms)(const float*, const void*, int, long long, const float*, float, void*, int, int, int, int, cudaStream_t);
    // the gated delta rule: convolutions, unit norms and step sizes in front of it; the recurrence token by token; the head norm
    // with its gate behind it
    int (*delta_prepare)(const void*, int, int, long long, long long, const float*, int, const float*, long long, long long, const int32_t*,
                         const int32_t*, const int32_t*, int, int, int, int, int, float, float*, int, float*, int, const float*, const float*,
                         float*, int, int, void*, int, int, void*, int, cudaStream_t);
    int (*delta_scan)(const float*, const float*, const float*, const float*, long long, const float*, const float*, const void*, int, int,
                      long long, long long, float*, long long, long long, const int32_t*, const int32_t*, int, int, int, int, int, int, int, int,
                      float*, cudaStream_t);
    // (long portions of a bfloat16 model: in chunks on the tensor cores)
    int (*delta_chunk_make)(const float*, const float*, const float*, const float*, long long, const float*, const float*, const int32_t*, int,
                            void*, int, int, int, int, cudaStream_t);
    int (*delta_chunk_walk)(const void*, int, int, long long, long long, float*, long long, long long, const int32_t*, const int32_t*, int,
                            const int32_t*, int, const int32_t*, const void*, int, int, int, int, int, float*, int*, cudaStream_t);
    int (*delta_chunk_supports)(int, int);
    int (*delta_chunk_tokens)(void);
    long long (*delta_chunk_scratch_bytes)(int, int);
    int (*head_norm_gate)(const float*, const float*, float, const void*, int, long long, int, void*, int, int, int, int, cudaStream_t);
    // logits scaled and softly capped in place
    int (*scale_softcap)(float*, long long, float, float, cudaStream_t);
    const char* (*last_error)(void);
};
struct FlashKernels {
    int (*prefill)(const void*, const void*, const void*, long long, int, const int32_t*, int, const int32_t*,
                   const int32_t*, const int32_t*, const int32_t*, int, void*, int, int, int, int, int, float, cudaStream_t);
    int (*decode)(const void*, const void*, const void*, long long, int, const int32_t*, int, const int32_t*, int,
                  const int32_t*, const int32_t*, float*, float*, void*, int, int, int, int, int, int, float, cudaStream_t);
    int (*decode_bulk)(const void*, const void*, const void*, long long, int, int, const int32_t*, int, const int32_t*, int,
                       const int32_t*, const int32_t*, float*, float*, void*, int, int, int, int, int, int, float, int, int*,
                       cudaStream_t);
    int (*prefill_tc5)(const void*, int, const void*, const void*, long long, int, int, const int32_t*, int, const int32_t*,
                       const int32_t*, const int32_t*, const int32_t*, int, void*, int, int, int, int, int, float, int, float*,
                       float*, int*, cudaStream_t);
    // the two kernels above with a sink in the softmax's denominator, a distance bias, an output gate and a cap on the scores,
    // each optional (a bias and a cap exclude each other)
    int (*decode_bulk_capped)(const void*, const void*, const void*, long long, int, int, const int32_t*, int, const int32_t*, int,
                              const int32_t*, const int32_t*, float*, float*, void*, int, int, int, int, int, int, float, int, int*,
                              const float*, const float*, const void*, long long, float, cudaStream_t);
    int (*prefill_tc5_capped)(const void*, int, const void*, const void*, long long, int, int, const int32_t*, int, const int32_t*,
                              const int32_t*, const int32_t*, const int32_t*, int, void*, int, int, int, int, int, float, int, float*,
                              float*, int*, const float*, const float*, const void*, long long, float, cudaStream_t);
    // the prompt kernel over dense keys and values, a row per token with the heads side by side
    int (*prefill_tc5_dense)(const void*, long long, int, const void*, const void*, long long, int, const int32_t*, const int32_t*,
                             const int32_t*, const int32_t*, const int32_t*, int, void*, int, int, float, int, float*, float*, int*, const void*,
                             long long, cudaStream_t);
    const char* (*last_error)(void);
};
// attention over cached latent rows on the tensor cores (latent_attention_mma.cu)
struct LatentKernels {
    int (*supports)(int, int);
    int (*attention)(const void*, const void*, long long, int, const int32_t*, int, const int32_t*, const int32_t*, const int32_t*,
                     const int32_t*, int, void*, float*, float*, int, int, int, int, float, int, cudaStream_t);
    // the products per head in front of and behind it
    int (*latent_absorb)(const void*, long long, const void*, const float*, int, int, const int32_t*, void*, int, int, int, int, int,
                         cudaStream_t);
    int (*latent_expand)(const void*, const void*, const void*, long long, int, void*, int, int, int, int, cudaStream_t);
    const char* (*last_error)(void);
};
struct GemmKernels {
    int (*gemm)(const void*, const void*, void*, int, int, int, int, int, int, int, int, int, const float*, int, const float*, int, int,
                float, const float*, void*, float*, int*, cudaStream_t);
    int (*gemm_pair)(const void*, const void*, void*, int, int, int, int, int, int, int, const float*, int, const float*, int, int, float,
                     const float*, void*, float*, int*, cudaStream_t);
    // several weights in one launch, a weight per tile of 256 rows
    int (*gemm_experts)(const void*, const void*, void*, int, int, int, int, int, const int32_t*, int, const float*, const float*, int*,
                        cudaStream_t);
    const char* (*last_error)(void);
};

// Folder the kernel libraries are opened from: set_library_dir(), else $PURHIE_B200_LIB_DIR, else the folder
// this library itself was loaded from.
QE_API void set_library_dir(const std::string& dir);
QE_API std::string library_dir();
QE_API const CoreKernels& core_kernels();
QE_API const FlashKernels& flash_kernels();
QE_API const GemmKernels& gemm_kernels();
QE_API const LatentKernels& latent_kernels();
QE_API void require_library(const std::string& name);      // "core", "flash", "gemm100", "latent": open it now
QE_API extern long long g_launches;                          // launcher calls so far (for the bench's count)

// Time per kernel class, for finding out where a step's time goes (the reference prints such a breakdown under
// QWEN_PROFILE=1: src/qwen_model.cpp:393-423, 2795-2818).  Off unless PURHIE_PROFILE=1 is in the environment (or
// set_enabled): then every launcher call is bracketed by CUDA events on the engine's stream, batches of single
// tokens are launched kernel by kernel instead of replayed as graphs, and report() gives, per launcher name, the
// calls, the device milliseconds and, where the caller noted them, the bytes and flops of its launches.  The
// events serialise nothing, but a profiled step is a little slower than an unprofiled one.
class QE_API LaunchProfile {
public:
    static LaunchProfile& get();
    bool on() const { return enabled_; }
    void set_enabled(bool on) { enabled_ = on; }
    void set_stream(cudaStream_t s) { stream_ = s; }
    void forget_stream(cudaStream_t s) { if (stream_ == s) stream_ = nullptr; }      // before s is destroyed
    void note_cost(double bytes, double flops) { pending_bytes_ = bytes; pending_flops_ = flops; }   // of the next launch
    void begin(const char* call_text);
    void end();
    // {"name": {"calls", "ms", "bytes", "flops"}} over everything since the last reset; waits for the stream.
    std::string report_json(bool reset);
private:
    static std::string launcher_name(const char* call_text);
    LaunchProfile();
    struct Record { std::string name; cudaEvent_t start, stop; double bytes, flops; };
    bool enabled_ = false;
    cudaStream_t stream_ = nullptr;
    double pending_bytes_ = 0, pending_flops_ = 0;
    std::vector<Record> records_;
    std::vector<std::pair<cudaEvent_t, cudaEvent_t>> spare_;
    struct Sum { long long calls = 0; double ms = 0, bytes = 0, flops = 0; };
    std::map<std::string, Sum> sums_;
    void fold();
};
struct LaunchScope {
    bool on;
    explicit LaunchScope(const char* call_text) : on(LaunchProfile::get().on()) { if (on) LaunchProfile::get().begin(call_text); }
    ~LaunchScope() { if (on) LaunchProfile::get().end(); }
};

// Run a launcher; a non-zero status becomes a KernelError with the library's text.
#define QE_LAUNCH(lib, call)                                                                     \
    do {                                                                                         \
        ::qe::g_launches++;                                                                      \
        ::qe::LaunchScope qe_scope_(#call);                                                      \
        if ((call) != 0) throw ::qe::KernelError((lib).last_error());                           \
    } while (0)

QE_API int sm_count();                                      // of the current device

}  // namespace qe
