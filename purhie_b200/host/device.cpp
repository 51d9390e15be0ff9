#include "device.h"

#include <dlfcn.h>

#include <mutex>

namespace qe {

long long g_launches = 0;

// ---- memory -------------------------------------------------------------------------------------------------
DeviceBuffer::DeviceBuffer(size_t bytes) : n_(bytes) {
    if (bytes) {
        cudaError_t e = cudaMalloc(&p_, bytes);
        if (e != cudaSuccess) {
            p_ = nullptr;
            n_ = 0;
            throw Error(e == cudaErrorMemoryAllocation ? kOutOfMemory : kKernelLaunch,
                        "cudaMalloc of " + std::to_string(bytes) + " bytes: " + cudaGetErrorString(e));
        }
    }
}
DeviceBuffer::~DeviceBuffer() { reset(); }
DeviceBuffer& DeviceBuffer::operator=(DeviceBuffer&& o) noexcept {
    if (this != &o) {
        reset();
        p_ = o.p_; n_ = o.n_;
        o.p_ = nullptr; o.n_ = 0;
    }
    return *this;
}
void DeviceBuffer::reset() {
    if (p_) cudaFree(p_);
    p_ = nullptr;
    n_ = 0;
}

PinnedBuffer::PinnedBuffer(size_t bytes) { ensure(bytes); }
PinnedBuffer::~PinnedBuffer() { if (p_) cudaFreeHost(p_); }
void PinnedBuffer::ensure(size_t bytes) {
    if (bytes <= n_) return;
    if (p_) cudaFreeHost(p_);
    p_ = nullptr; n_ = 0;
    QE_CUDA(cudaMallocHost(&p_, bytes));
    n_ = bytes;
}

Tensor DeviceArena::alloc(DType dtype, std::vector<int64_t> shape) {
    Tensor t(nullptr, dtype, std::move(shape));
    DeviceBuffer b(std::max<size_t>(t.bytes(), 16));
    t.data = b.data();
    bytes_ += b.bytes();
    bufs_.emplace(t.data, std::move(b));
    return t;
}
void DeviceArena::release(const Tensor& t) {
    auto it = bufs_.find(t.data);
    if (it == bufs_.end()) return;
    bytes_ -= it->second.bytes();
    bufs_.erase(it);
}

Tensor Workspace::get(const std::string& name, std::vector<int64_t> shape, DType dtype) {
    Tensor t(nullptr, dtype, std::move(shape));
    size_t need = std::max<size_t>(t.bytes(), 16);
    auto it = bufs_.find(name);
    if (it == bufs_.end() || it->second.bytes() < need) {
        if (frozen) throw Error(kInvalidState, "workspace buffer '" + name + "' would have to grow while frozen");
        if (it != bufs_.end()) {
            QE_CUDA(cudaStreamSynchronize(stream));        // a kernel in flight may still use the old block
            bufs_.erase(it);
        }
        it = bufs_.emplace(name, DeviceBuffer(need)).first;
    }
    t.data = it->second.data();
    return t;
}
size_t Workspace::bytes() const {
    size_t n = 0;
    for (const auto& kv : bufs_) n += kv.second.bytes();
    return n;
}

// ---- kernel libraries -----------------------------------------------------------------------------------------
namespace {
std::mutex g_lib_mutex;
std::string g_lib_dir;
std::map<std::string, void*> g_handles;
CoreKernels g_core{};
FlashKernels g_flash{};
GemmKernels g_gemm{};
LatentKernels g_latent{};
bool g_core_ok = false, g_flash_ok = false, g_gemm_ok = false, g_latent_ok = false;

std::string own_dir() {
    Dl_info info;
    if (dladdr((void*)&own_dir, &info) && info.dli_fname) {
        std::string p(info.dli_fname);
        size_t slash = p.rfind('/');
        return slash == std::string::npos ? "." : p.substr(0, slash);
    }
    return ".";
}

void* open_library(const std::string& name) {
    auto it = g_handles.find(name);
    if (it != g_handles.end()) return it->second;
    std::string dir = g_lib_dir;
    if (dir.empty()) {
        const char* e = getenv("PURHIE_B200_LIB_DIR");
        dir = (e && *e) ? e : own_dir();
    }
    std::string path = dir + "/libpurhie_" + name + ".so";
    void* h = dlopen(path.c_str(), RTLD_NOW | RTLD_LOCAL);
    if (!h)
        throw KernelError("the '" + name + "' kernel library is missing (" + std::string(dlerror() ? dlerror() : path) +
                          "); build it with `python -m purhie_b200.csrc.build " + name +
                          "`. There is no other implementation of these kernels.");
    g_handles[name] = h;
    return h;
}

template <typename F> void bind(void* h, const std::string& lib, const char* sym, F& out) {
    void* p = dlsym(h, sym);
    if (!p) throw KernelError("libpurhie_" + lib + ".so does not export " + sym + " (stale build?)");
    out = reinterpret_cast<F>(p);
}
}  // namespace

void set_library_dir(const std::string& dir) {
    std::lock_guard<std::mutex> lock(g_lib_mutex);
    g_lib_dir = dir;
}
std::string library_dir() {
    std::lock_guard<std::mutex> lock(g_lib_mutex);
    if (!g_lib_dir.empty()) return g_lib_dir;
    const char* e = getenv("PURHIE_B200_LIB_DIR");
    return (e && *e) ? e : own_dir();
}

const CoreKernels& core_kernels() {
    if (g_core_ok) return g_core;
    std::lock_guard<std::mutex> lock(g_lib_mutex);
    if (g_core_ok) return g_core;
    void* h = open_library("core");
    bind(h, "core", "ph_embed_gather", g_core.embed_gather);
    bind(h, "core", "ph_add_rmsnorm", g_core.add_rmsnorm);
    bind(h, "core", "ph_swiglu", g_core.swiglu);
    bind(h, "core", "ph_cast", g_core.cast);
    bind(h, "core", "ph_qk_norm_rope_kv_write", g_core.qk_norm_rope_kv_write);
    bind(h, "core", "ph_add_weight_sumsq", g_core.add_weight_sumsq);
    bind(h, "core", "ph_attention_generic", g_core.attention_generic);
    bind(h, "core", "ph_gemm_simple", g_core.gemm_simple);
    bind(h, "core", "ph_argmax_parts", g_core.argmax);
    bind(h, "core", "ph_argmax_scratch_bytes", g_core.argmax_scratch_bytes);
    bind(h, "core", "ph_sample_temperature", g_core.sample_temperature);
    bind(h, "core", "ph_sample_chain", g_core.sample_chain);
    bind(h, "core", "ph_sample_chain_max_k", g_core.sample_chain_max_k);
    bind(h, "core", "ph_random_fill", g_core.random_fill);
    bind(h, "core", "ph_add_layernorm", g_core.add_layernorm);
    bind(h, "core", "ph_embed_gather_scaled", g_core.embed_gather_scaled);
    bind(h, "core", "ph_glu", g_core.glu);
    bind(h, "core", "ph_glu_scaled", g_core.glu_scaled);
    bind(h, "core", "ph_unary_act", g_core.unary_act);
    bind(h, "core", "ph_decayed_scan", g_core.decayed_scan);
    bind(h, "core", "ph_rms_pair_mean", g_core.rms_pair_mean);
    bind(h, "core", "ph_causal_conv_silu", g_core.causal_conv_silu);
    bind(h, "core", "ph_selective_scan", g_core.selective_scan);
    bind(h, "core", "ph_route", g_core.route);
    bind(h, "core", "ph_route_max_tiles", g_core.route_max_tiles);
    bind(h, "core", "ph_route_sort", g_core.route_sort);
    bind(h, "core", "ph_route_tile_rows", g_core.route_tile_rows);
    bind(h, "core", "ph_route_sort_tiles", g_core.route_sort_tiles);
    bind(h, "core", "ph_gemm_grouped", g_core.gemm_grouped);
    bind(h, "core", "ph_gemv_grouped", g_core.gemv_grouped);
    bind(h, "core", "ph_route_gather", g_core.route_gather);
    bind(h, "core", "ph_route_combine", g_core.route_combine);
    bind(h, "core", "ph_rms_gate", g_core.rms_gate);
    bind(h, "core", "ph_add_dyntanh", g_core.add_dyntanh);
    bind(h, "core", "ph_concat_restart", g_core.concat_restart);
    bind(h, "core", "ph_latent_prepare", g_core.latent_prepare);
    bind(h, "core", "ph_latent_absorb", g_core.latent_absorb);
    bind(h, "core", "ph_latent_expand", g_core.latent_expand);
    bind(h, "core", "ph_latent_gather", g_core.latent_gather);
    bind(h, "core", "ph_attention_generic_biased", g_core.attention_generic_biased);
    bind(h, "core", "ph_qk_norm_rope_gate_kv_write", g_core.qk_norm_rope_gate_kv_write);
    bind(h, "core", "ph_lanes_rmsnorm", g_core.lanes_rmsnorm);
    bind(h, "core", "ph_ssd_scan", g_core.ssd_scan);
    bind(h, "core", "ph_ssd_chunk", g_core.ssd_chunk);
    bind(h, "core", "ph_ssd_chunk_supports", g_core.ssd_chunk_supports);
    bind(h, "core", "ph_gate_rms", g_core.gate_rms);
    bind(h, "core", "ph_attention_talking", g_core.attention_talking);
    bind(h, "core", "ph_attention_talking_mma", g_core.attention_talking_mma);
    bind(h, "core", "ph_attention_talking_mma_supports", g_core.attention_talking_mma_supports);
    bind(h, "core", "ph_attention_talking_mma_ctas_per_sm", g_core.attention_talking_mma_ctas_per_sm);
    bind(h, "core", "ph_joint_norm_kv_write", g_core.joint_norm_kv_write);
    bind(h, "core", "ph_joint_norm_rope_kv_write", g_core.joint_norm_rope_kv_write);
    bind(h, "core", "ph_attention_generic_capped", g_core.attention_generic_capped);
    bind(h, "core", "ph_min_gru_scan", g_core.min_gru_scan);
    bind(h, "core", "ph_pair_sum", g_core.pair_sum);
    bind(h, "core", "ph_add_scaled_rmsnorm", g_core.add_scaled_rmsnorm);
    bind(h, "core", "ph_delta_prepare", g_core.delta_prepare);
    bind(h, "core", "ph_delta_scan", g_core.delta_scan);
    bind(h, "core", "ph_delta_chunk_make", g_core.delta_chunk_make);
    bind(h, "core", "ph_delta_chunk_walk", g_core.delta_chunk_walk);
    bind(h, "core", "ph_delta_chunk_supports", g_core.delta_chunk_supports);
    bind(h, "core", "ph_delta_chunk_tokens", g_core.delta_chunk_tokens);
    bind(h, "core", "ph_delta_chunk_scratch_bytes", g_core.delta_chunk_scratch_bytes);
    bind(h, "core", "ph_head_norm_gate", g_core.head_norm_gate);
    bind(h, "core", "ph_scale_softcap", g_core.scale_softcap);
    bind(h, "core", "ph_core_last_error", g_core.last_error);
    g_core_ok = true;
    return g_core;
}

const FlashKernels& flash_kernels() {
    if (g_flash_ok) return g_flash;
    std::lock_guard<std::mutex> lock(g_lib_mutex);
    if (g_flash_ok) return g_flash;
    void* h = open_library("flash");
    bind(h, "flash", "ph_attention_prefill", g_flash.prefill);
    bind(h, "flash", "ph_attention_decode", g_flash.decode);
    bind(h, "flash", "ph_attention_decode_bulk", g_flash.decode_bulk);
    bind(h, "flash", "ph_attention_prefill_tc5", g_flash.prefill_tc5);
    bind(h, "flash", "ph_attention_decode_bulk_capped", g_flash.decode_bulk_capped);
    bind(h, "flash", "ph_attention_prefill_tc5_capped", g_flash.prefill_tc5_capped);
    bind(h, "flash", "ph_attention_prefill_tc5_dense", g_flash.prefill_tc5_dense);
    bind(h, "flash", "ph_flash_last_error", g_flash.last_error);
    g_flash_ok = true;
    return g_flash;
}

const GemmKernels& gemm_kernels() {
    if (g_gemm_ok) return g_gemm;
    std::lock_guard<std::mutex> lock(g_lib_mutex);
    if (g_gemm_ok) return g_gemm;
    void* h = open_library("gemm100");
    bind(h, "gemm100", "ph_gemm_bf16_tcgen05", g_gemm.gemm);
    bind(h, "gemm100", "ph_gemm_bf16_tcgen05_pair", g_gemm.gemm_pair);
    bind(h, "gemm100", "ph_gemm_bf16_tcgen05_grouped", g_gemm.gemm_experts);
    bind(h, "gemm100", "ph_gemm100_last_error", g_gemm.last_error);
    g_gemm_ok = true;
    return g_gemm;
}

const LatentKernels& latent_kernels() {
    if (g_latent_ok) return g_latent;
    std::lock_guard<std::mutex> lock(g_lib_mutex);
    if (g_latent_ok) return g_latent;
    void* h = open_library("latent");
    bind(h, "latent", "ph_latent_attention_supports", g_latent.supports);
    bind(h, "latent", "ph_latent_attention", g_latent.attention);
    bind(h, "latent", "ph_latent_absorb_mma", g_latent.latent_absorb);
    bind(h, "latent", "ph_latent_expand_mma", g_latent.latent_expand);
    bind(h, "latent", "ph_latent_last_error", g_latent.last_error);
    g_latent_ok = true;
    return g_latent;
}

void require_library(const std::string& name) {
    if (name == "core") core_kernels();
    else if (name == "flash") flash_kernels();
    else if (name == "gemm100") gemm_kernels();
    else if (name == "latent") latent_kernels();
    else {
        std::lock_guard<std::mutex> lock(g_lib_mutex);
        open_library(name);
    }
}

// ---- time per kernel class ----------------------------------------------------------------------------------------
LaunchProfile::LaunchProfile() {
    const char* e = getenv("PURHIE_PROFILE");
    enabled_ = e && *e && *e != '0';
}
LaunchProfile& LaunchProfile::get() {
    static LaunchProfile p;
    return p;
}
std::string LaunchProfile::launcher_name(const char* call_text) {
    // "k.add_rmsnorm(stream.x, ...)" -> "add_rmsnorm"
    std::string name(call_text);
    size_t paren = name.find('(');
    if (paren != std::string::npos) name.resize(paren);
    size_t dot = name.rfind('.');
    if (dot != std::string::npos) name = name.substr(dot + 1);
    return name;
}
void LaunchProfile::begin(const char* call_text) {
    Record r;
    r.name = launcher_name(call_text);
    r.bytes = pending_bytes_; r.flops = pending_flops_;
    pending_bytes_ = pending_flops_ = 0;
    if (spare_.empty()) {
        cudaEventCreate(&r.start);
        cudaEventCreate(&r.stop);
    } else {
        r.start = spare_.back().first; r.stop = spare_.back().second;
        spare_.pop_back();
    }
    cudaEventRecord(r.start, stream_);
    records_.push_back(r);
    if (records_.size() > 65536) fold();
}
void LaunchProfile::end() {
    if (!records_.empty()) cudaEventRecord(records_.back().stop, stream_);
}
void LaunchProfile::fold() {
    // waits on the events, not on the stream: the engine whose stream they were recorded on may be gone by now
    for (Record& r : records_) {
        float ms = 0;
        if (cudaEventSynchronize(r.stop) == cudaSuccess && cudaEventElapsedTime(&ms, r.start, r.stop) == cudaSuccess) {
            Sum& s = sums_[r.name];
            s.calls++; s.ms += ms; s.bytes += r.bytes; s.flops += r.flops;
        }
        spare_.emplace_back(r.start, r.stop);
    }
    records_.clear();
}
std::string LaunchProfile::report_json(bool reset) {
    fold();
    std::string out = "{";
    bool first = true;
    for (const auto& kv : sums_) {
        char buf[256];
        snprintf(buf, sizeof buf, "%s\"%s\": {\"calls\": %lld, \"ms\": %.6f, \"bytes\": %.0f, \"flops\": %.0f}", first ? "" : ", ",
                 kv.first.c_str(), kv.second.calls, kv.second.ms, kv.second.bytes, kv.second.flops);
        out += buf;
        first = false;
    }
    out += "}";
    if (reset) sums_.clear();
    return out;
}

int sm_count() {
    static int cached[64] = {0};
    int dev = 0;
    QE_CUDA(cudaGetDevice(&dev));
    if (dev < 0 || dev >= 64) dev = 0;
    if (!cached[dev]) QE_CUDA(cudaDeviceGetAttribute(&cached[dev], cudaDevAttrMultiProcessorCount, dev));
    return cached[dev];
}

}  // namespace qe
