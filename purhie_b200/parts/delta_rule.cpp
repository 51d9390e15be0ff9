// The gated delta rule: a matrix state per head that decays and is then corrected towards a value along a key.
//
//   q = Wq h, k = Wk h (kv_heads heads of dim), v = Wv h (heads of value_dim); each passes a causal convolution per channel over
//   its last `conv` inputs (no bias, zeros before a request's start) and silu; q and k are divided by
//   sqrt(sum of squares + 1e-6) per head, q also by sqrt(dim); head h uses q / k head h / (heads / kv_heads).
//   beta = sigmoid(Wb h) per head;  decay a = exp(-exp(A_log) softplus(z + dt_bias)), z per key channel of a head ("decay":
//   "channel") or one number per head ("head").
//   S <- diag(a) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//   y = Wo (o / sqrt(mean over the head of o^2 + eps) * norm * act(g)), act sigmoid or silu ("gate").
// z comes from one matrix (names.decay_proj) or through a low rank (names.decay_down, decay_up); g likewise (gate_proj, or
// gate_down and gate_up).  A low rank of -1 is what the stored matrices say.
//
// What a request carries is S (float32, [heads][value_dim][dim]) and the last conv - 1 inputs of the convolution, one state
// slot of the cache manager, zero at admission.  A prompt cut anywhere walks the same recurrence.  The convolutions, the unit
// norms, beta, the decays, S, the read-out, the head norm and the gate are float32 in every mode; the products follow the
// model's dtype, what the low-rank products give is float32.
//
// One product gives the rows [q | k | v | (g) | (low) | beta | (z)]: low is decay_down's and gate_down's rows side by side,
// which one product over a matrix with decay_up and gate_up on its diagonal turns into [z | g].  Columns without a weight
// (zero rows) bring the widths to multiples of 8.
//
// In a bfloat16 model a portion of kChunkRows tokens or more runs in chunks on the tensor cores (csrc/delta_chunk.cu), every
// other one token by token; the chunk list is the mixer's own step metadata.
#include <algorithm>
#include <cmath>

#include "linear.h"
#include "parts.h"

namespace qe {

namespace {
int64_t round8(int64_t n) { return (n + 7) / 8 * 8; }
}  // namespace

// params: hidden_size, num_heads, num_kv_heads, head_dim, value_dim, conv, norm_eps, decay ("head" | "channel"), gate ("silu" |
// "sigmoid"), decay_rank and gate_rank (where a low rank is used; null: the stored matrices' inner size),
// names{q_proj, k_proj, v_proj, q_conv, k_conv, v_conv, beta_proj, a_log, dt_bias, norm, o_proj, and decay_proj or {decay_down,
// decay_up}, and gate_proj or {gate_down, gate_up}}.
class DeltaRule : public Mixer {
public:
    DeltaRule(const Json& p, BuildContext& b) : Mixer(p, b) {
        hidden_ = p.at("hidden_size").as_int();
        heads_ = (int)p.at("num_heads").as_int();
        kv_heads_ = (int)p.at("num_kv_heads").as_int();
        dim_ = (int)p.at("head_dim").as_int();
        vdim_ = (int)p.at("value_dim").as_int();
        taps_ = (int)p.at("conv").as_int();
        eps_ = p.at("norm_eps").as_double();
        if (heads_ < 1 || kv_heads_ < 1 || dim_ < 1 || vdim_ < 1 || taps_ < 1)
            throw ConfigError("delta_rule: num_heads, num_kv_heads, head_dim, value_dim and conv must be positive");
        if (heads_ % kv_heads_) throw ConfigError("delta_rule: " + std::to_string(heads_) + " heads do not share " + std::to_string(kv_heads_) + " key heads evenly");
        const std::string decay = p.at("decay").as_string(), gate = p.at("gate").as_string();
        if (decay != "head" && decay != "channel") throw ConfigError("delta_rule: decay is 'head' or 'channel', got '" + decay + "'");
        if (gate != "silu" && gate != "sigmoid") throw ConfigError("delta_rule: gate is 'silu' or 'sigmoid', got '" + gate + "'");
        per_channel_ = decay == "channel";
        gate_act_ = gate == "sigmoid" ? 1 : 0;
        low_decay_ = names_.count("decay_down") != 0;
        low_gate_ = names_.count("gate_down") != 0;
        if (per_channel_ != low_decay_)
            throw ConfigError("delta_rule: a decay per channel comes through decay_down and decay_up, a decay per head from decay_proj");
        decay_rank_ = low_decay_ ? p.get_int("decay_rank", -1) : 0;
        gate_rank_ = low_gate_ ? p.get_int("gate_rank", -1) : 0;
        gemm_ = b.options.get_string("gemm", "auto");
        qk_width_ = (int64_t)kv_heads_ * dim_;
        v_width_ = (int64_t)heads_ * vdim_;
        decay_width_ = per_channel_ ? (int64_t)heads_ * dim_ : heads_;
        channels_ = 2 * qk_width_ + v_width_;
    }

    std::vector<TensorSpec> tensor_specs() const override {
        std::vector<TensorSpec> s = {{name_of("q_proj"), {qk_width_, hidden_}, Role::Matrix, Init::Normal},
                                     {name_of("k_proj"), {qk_width_, hidden_}, Role::Matrix, Init::Normal},
                                     {name_of("v_proj"), {v_width_, hidden_}, Role::Matrix, Init::Normal},
                                     {name_of("q_conv"), {qk_width_, taps_}, Role::Vector, Init::Normal},
                                     {name_of("k_conv"), {qk_width_, taps_}, Role::Vector, Init::Normal},
                                     {name_of("v_conv"), {v_width_, taps_}, Role::Vector, Init::Normal},
                                     {name_of("beta_proj"), {heads_, hidden_}, Role::Matrix, Init::Normal},
                                     {name_of("a_log"), {heads_}, Role::Vector, Init::Normal},
                                     {name_of("dt_bias"), {decay_width_}, Role::Vector, Init::Normal},
                                     {name_of("norm"), {vdim_}, Role::Vector, Init::Scale},
                                     {name_of("o_proj"), {hidden_, v_width_}, Role::Matrix, Init::Normal}};
        if (low_decay_) {
            s.push_back({name_of("decay_down"), {decay_rank_, hidden_}, Role::Matrix, Init::Normal});
            s.push_back({name_of("decay_up"), {decay_width_, decay_rank_}, Role::Matrix, Init::Normal});
        } else {
            s.push_back({name_of("decay_proj"), {decay_width_, hidden_}, Role::Matrix, Init::Normal});
        }
        if (low_gate_) {
            s.push_back({name_of("gate_down"), {gate_rank_, hidden_}, Role::Matrix, Init::Normal});
            s.push_back({name_of("gate_up"), {v_width_, gate_rank_}, Role::Matrix, Init::Normal});
        } else {
            s.push_back({name_of("gate_proj"), {v_width_, hidden_}, Role::Matrix, Init::Normal});
        }
        return s;
    }

    void bind(WeightSource& src) override {
        cudaStream_t stream = src.stream();
        auto rank_of = [&](const std::string& down, const std::string& up, const Tensor& d, const Tensor& u) {
            if (d.shape[0] != u.shape[1])
                throw WeightError(name_of(down) + " gives " + std::to_string(d.shape[0]) + " values, " + name_of(up) + " takes " + std::to_string(u.shape[1]));
            return d.shape[0];
        };
        // the stacked matrix: every projection of h (a layout choice only)
        std::vector<std::pair<Tensor, int64_t>> parts;                   // a matrix and its first row
        int64_t at = 0;
        auto stack = [&](const std::string& role) {
            Tensor t = src.fetch(name_of(role));
            parts.push_back({t, at});
            at += t.shape[0];
            return parts.back().second;
        };
        stack("q_proj"); stack("k_proj"); stack("v_proj");
        Tensor decay_up, gate_up;
        int64_t decay_rank = 0, gate_rank = 0;
        if (!low_gate_) { at = round8(at); gate_col_ = stack("gate_proj"); }
        at = round8(at);
        low_col_ = at;
        if (low_decay_) { stack("decay_down"); decay_up = src.fetch(name_of("decay_up")); decay_rank = rank_of("decay_down", "decay_up", parts.back().first, decay_up); }
        if (low_gate_) { stack("gate_down"); gate_up = src.fetch(name_of("gate_up")); gate_rank = rank_of("gate_down", "gate_up", parts.back().first, gate_up); }
        low_width_ = round8(decay_rank + gate_rank);
        at = low_col_ + low_width_;
        beta_col_ = stack("beta_proj");
        if (!low_decay_) decay_col_ = stack("decay_proj");
        width_ = round8(at);
        const DType dt = parts[0].first.dtype;
        for (auto& part : parts)
            if (part.first.dtype != dt) throw WeightError("the projections of " + name_of("q_proj") + "'s mixer are stored in different precisions");
        const size_t es = dtype_size(dt);
        Tensor all = src.arena().alloc(dt, {width_, hidden_});
        QE_CUDA(cudaMemsetAsync(all.data, 0, all.bytes(), stream));
        for (auto& part : parts)
            QE_CUDA(cudaMemcpyAsync(static_cast<char*>(all.data) + (size_t)part.second * hidden_ * es, part.first.data, part.first.bytes(),
                                    cudaMemcpyDeviceToDevice, stream));
        QE_CUDA(cudaStreamSynchronize(stream));
        for (auto& part : parts) src.release(part.first);
        in_proj_ = Linear(all, "delta_in", gemm_);
        if (low_width_) {
            // decay_up and gate_up on the diagonal: rows [z | g], columns [decay's low | gate's low | none]
            const DType ut = low_decay_ ? decay_up.dtype : gate_up.dtype;
            if ((low_decay_ && decay_up.dtype != ut) || (low_gate_ && gate_up.dtype != ut))
                throw WeightError("the low-rank products of " + name_of("q_proj") + "'s mixer are stored in different precisions");
            const size_t us = dtype_size(ut);
            up_width_ = (low_decay_ ? decay_width_ : 0) + (low_gate_ ? v_width_ : 0);
            Tensor up = src.arena().alloc(ut, {up_width_, low_width_});
            QE_CUDA(cudaMemsetAsync(up.data, 0, up.bytes(), stream));
            auto place = [&](const Tensor& t, int64_t row, int64_t col) {
                QE_CUDA(cudaMemcpy2DAsync(static_cast<char*>(up.data) + ((size_t)row * low_width_ + col) * us, (size_t)low_width_ * us, t.data,
                                          (size_t)t.shape[1] * us, (size_t)t.shape[1] * us, (size_t)t.shape[0], cudaMemcpyDeviceToDevice, stream));
            };
            if (low_decay_) place(decay_up, 0, 0);
            if (low_gate_) place(gate_up, low_decay_ ? decay_width_ : 0, decay_rank);
            QE_CUDA(cudaStreamSynchronize(stream));
            if (low_decay_) src.release(decay_up);
            if (low_gate_) src.release(gate_up);
            up_proj_ = Linear(up, "delta_up", gemm_);
        }
        // the convolution's taps, the channels of q, k and v side by side: [taps][channels]
        std::vector<float> taps((size_t)taps_ * channels_);
        int64_t first = 0;
        for (const char* role : {"q_conv", "k_conv", "v_conv"}) {
            Tensor t = src.fetch(name_of(role));
            std::vector<float> host((size_t)t.numel());
            QE_CUDA(cudaMemcpy(host.data(), t.data, host.size() * sizeof(float), cudaMemcpyDeviceToHost));
            for (int64_t c = 0; c < t.shape[0]; c++)
                for (int k = 0; k < taps_; k++) taps[(size_t)k * channels_ + first + c] = host[(size_t)c * taps_ + k];
            first += t.shape[0];
            src.release(t);
        }
        conv_ = upload(src, taps);
        // -exp(A_log), once, in float32
        Tensor a_log = src.fetch(name_of("a_log"));
        std::vector<float> rate((size_t)heads_);
        QE_CUDA(cudaMemcpy(rate.data(), a_log.data, rate.size() * sizeof(float), cudaMemcpyDeviceToHost));
        for (float& v : rate) v = -std::exp(v);
        src.release(a_log);
        rate_ = upload(src, rate);
        dt_bias_ = src.fetch(name_of("dt_bias"));
        norm_ = src.fetch(name_of("norm"));
        o_proj_ = Linear(src.fetch(name_of("o_proj")), "o_proj", gemm_);
    }

    std::vector<std::string> required_libraries() const override {
        const bool fast = in_proj_.fast() || o_proj_.fast() || (up_proj_.defined() && up_proj_.fast());
        return fast ? std::vector<std::string>{"core", "gemm100"} : std::vector<std::string>{"core"};
    }
    int preferred_row_multiple() const override { return (in_proj_.fast() || o_proj_.fast()) ? 256 : 0; }
    CacheNeed cache_need() const override { return CacheNeed::state({state_floats()}, DType::F32); }

    // first row and rows of every chunk of the portions that run in chunks, and where each request's chunks start
    void prepare_step(StepPlan& plan) override {
        if (compute_dtype != DType::BF16 || plan.has("delta.chunks")) return;
        const int chunk = core_kernels().delta_chunk_tokens();
        std::vector<int32_t> items, seg_items = {0};
        int row = 0;
        for (int s = 0; s < plan.S; s++) {
            const int n = plan.q_lens[s];
            if (n >= kChunkRows)
                for (int at = 0; at < n; at += chunk) { items.push_back(row + at); items.push_back(std::min(chunk, n - at)); }
            row += n;
            seg_items.push_back((int32_t)(items.size() / 2));
        }
        if (items.empty()) return;
        plan.add("delta.chunks", std::move(items));
        plan.add("delta.seg_chunks", std::move(seg_items));
    }

    Addend forward(const Tensor& x, StepContext& ctx, const CacheView& cache) override {
        if (!cache.state.defined() || cache.state.dtype != DType::F32 || cache.state.shape.size() != 2 || cache.state.shape[1] != state_floats())
            throw Error(kInvalidState, "delta_rule: the cache manager gave no state of this mixer's shape");
        const int T = ctx.T;
        const DType dt = compute_dtype;
        Workspace& ws = *ctx.workspace;
        const CoreKernels& k = core_kernels();
        const LaunchProfile& profile = LaunchProfile::get();
        const double es = (double)dtype_size(dt);
        float* state = cache.state.as<float>();
        Addend in = in_proj_(x, ctx, "delta_in", dt, T, true);                                  // [T, width], maybe in parts
        const double row_bytes = (double)in.splits * dtype_size(in.tensor.dtype);
        const long long split_stride = (long long)T * width_;
        Tensor qkv = ws.get("delta_qkv", {T, channels_}, DType::F32);
        Tensor beta = ws.get("delta_beta", {T, heads_}, DType::F32);
        Tensor log_decay, low, gate_rows;
        if (!low_decay_) log_decay = ws.get("delta_log_decay", {T, heads_}, DType::F32);
        if (low_width_) low = ws.get("delta_low", {T, low_width_}, dt);
        const bool gate_in_parts = !low_gate_ && (in.splits > 1 || in.tensor.dtype != dt);
        if (gate_in_parts) gate_rows = ws.get("delta_gate", {T, v_width_}, dt);
        if (profile.on())
            LaunchProfile::get().note_cost((double)T * ((channels_ + low_width_ + heads_ + (gate_in_parts ? v_width_ : 0)) * row_bytes + channels_ * 4.0 +
                                                        (low_width_ + (gate_in_parts ? v_width_ : 0)) * es),
                                           2.0 * T * channels_ * taps_);
        QE_LAUNCH(k, k.delta_prepare(in.tensor.data, in.tensor.code(), in.splits, split_stride, width_, conv_.as<float>(), taps_, state,
                                     state_floats(), conv_at(), ctx.row_seg, ctx.seg_start, ctx.seg_slot, T, heads_, kv_heads_, dim_, vdim_,
                                     (float)(1.0 / std::sqrt((double)dim_)), qkv.as<float>(), (int)beta_col_, beta.as<float>(),
                                     low_decay_ ? -1 : (int)decay_col_, rate_.as<float>(), low_decay_ ? nullptr : dt_bias_.as<float>(),
                                     low_decay_ ? nullptr : log_decay.as<float>(), (int)low_col_, (int)low_width_, low_width_ ? low.data : nullptr,
                                     (int)gate_col_, gate_in_parts ? (int)v_width_ : 0, gate_in_parts ? gate_rows.data : nullptr,
                                     dt == DType::BF16 ? 1 : 0, ctx.stream));
        // [z | g] float32 behind the low-rank products
        Tensor up;
        if (low_width_) up = up_proj_(low, ctx, "delta_up", DType::F32, T).tensor;
        const float* z = low_decay_ ? up.as<float>() : nullptr;
        const void* gate = nullptr;
        int gate_code = 0;
        long long gate_stride = 0;
        if (low_gate_) { gate = up.as<float>() + (low_decay_ ? decay_width_ : 0); gate_stride = up_width_; }
        else if (gate_in_parts) { gate = gate_rows.data; gate_code = gate_rows.code(); gate_stride = v_width_; }
        else { gate = static_cast<const char*>(in.tensor.data) + (size_t)gate_col_ * dtype_size(dt); gate_code = in.tensor.code(); gate_stride = width_; }
        Tensor o = ws.get("delta_o", {T, v_width_}, DType::F32);
        auto note = [&](int requests, int rows) {       // q, k, v, the decays and beta in, o out, the state in and out
            if (profile.on())
                LaunchProfile::get().note_cost((double)rows * 4.0 * (channels_ + (low_decay_ ? decay_width_ : heads_) + heads_ + v_width_) +
                                                   2.0 * requests * (double)state_floats() * 4.0,
                                               (double)rows * heads_ * dim_ * vdim_ * 7.0);
        };
        // long portions in chunks on the tensor cores, the others token by token (the option "delta": "scan" keeps all of them there)
        const StepArray chunks = ctx.array("delta.chunks"), seg_chunks = ctx.array("delta.seg_chunks");
        const int n_chunks = ctx.option("delta") != "scan" && channels_ % 4 == 0 && k.delta_chunk_supports(dim_, vdim_) ? chunks.count / 2 : 0;
        int n_long = 0, rows_long = 0;
        if (n_chunks) {
            for (int n : ctx.q_lens)
                if (n >= kChunkRows) { n_long++; rows_long += n; }
            Tensor scratch = ws.get("delta_scratch", {(int64_t)n_chunks * heads_ * k.delta_chunk_scratch_bytes(dim_, vdim_)}, DType::U8);
            // (q, k, v and the decays in, the operands out; the operands in, o out, the state in and out)
            const double made = (double)n_chunks * heads_ * k.delta_chunk_scratch_bytes(dim_, vdim_);
            if (profile.on())
                LaunchProfile::get().note_cost(rows_long * 4.0 * (channels_ + (low_decay_ ? decay_width_ : heads_) + heads_) + made,
                                               (double)rows_long * heads_ * 64.0 * (2.0 * dim_ + dim_ + vdim_));
            QE_LAUNCH(k, k.delta_chunk_make(qkv.as<float>(), beta.as<float>(), low_decay_ ? nullptr : log_decay.as<float>(), z, up_width_,
                                            low_decay_ ? dt_bias_.as<float>() : nullptr, rate_.as<float>(), chunks.data, n_chunks, scratch.data,
                                            heads_, kv_heads_, dim_, vdim_, ctx.stream));
            if (profile.on())
                LaunchProfile::get().note_cost(made + rows_long * 4.0 * v_width_ + 2.0 * n_long * (double)state_floats() * 4.0,
                                               (double)rows_long * heads_ * vdim_ * (6.0 * dim_ + 64.0));
            QE_LAUNCH(k, k.delta_chunk_walk(in.tensor.data, in.tensor.code(), in.splits, split_stride, width_, state, state_floats(), conv_at(),
                                            ctx.seg_start, ctx.seg_slot, ctx.S, chunks.data, n_chunks, seg_chunks.data, scratch.data, heads_,
                                            kv_heads_, dim_, vdim_, taps_, o.as<float>(), ctx.gemm_error, ctx.stream));
        }
        if (n_long < ctx.S) {
            note(ctx.S - n_long, T - rows_long);
            QE_LAUNCH(k, k.delta_scan(qkv.as<float>(), beta.as<float>(), low_decay_ ? nullptr : log_decay.as<float>(), z, up_width_,
                                  low_decay_ ? dt_bias_.as<float>() : nullptr, rate_.as<float>(), in.tensor.data, in.tensor.code(), in.splits,
                                  split_stride, width_, state, state_floats(), conv_at(), ctx.seg_start, ctx.seg_slot, ctx.S, heads_, kv_heads_,
                                  dim_, vdim_, taps_, 0, n_long ? kChunkRows - 1 : 0, o.as<float>(), ctx.stream));
        }
        Tensor y = ws.get("delta_y", {T, v_width_}, dt);
        if (profile.on()) LaunchProfile::get().note_cost((double)T * v_width_ * (4.0 + (gate_code ? 2.0 : 4.0) + es), 0.0);
        QE_LAUNCH(k, k.head_norm_gate(o.as<float>(), norm_.as<float>(), (float)eps_, gate, gate_code, gate_stride, gate_act_, y.data, y.code(), T,
                                      heads_, vdim_, ctx.stream));
        return o_proj_(y, ctx, "delta_out", DType::F32, T, true, false, ctx.residual, nullptr, &ctx.norm_ahead);
    }

private:
    static constexpr int kChunkRows = 32;       // the shortest portion that runs in chunks
    static Tensor upload(WeightSource& src, const std::vector<float>& values) {
        Tensor t = src.arena().alloc(DType::F32, {(int64_t)values.size()});
        QE_CUDA(cudaMemcpyAsync(t.data, values.data(), values.size() * sizeof(float), cudaMemcpyHostToDevice, src.stream()));
        QE_CUDA(cudaStreamSynchronize(src.stream()));
        return t;
    }
    int64_t conv_at() const { return ((int64_t)heads_ * vdim_ * dim_ + 3) / 4 * 4; }
    int64_t state_floats() const { return (conv_at() + (int64_t)(taps_ - 1) * channels_ + 3) / 4 * 4; }

    int64_t hidden_, qk_width_, v_width_, decay_width_, channels_, decay_rank_, gate_rank_;
    int64_t width_ = 0, gate_col_ = 0, low_col_ = 0, low_width_ = 0, beta_col_ = 0, decay_col_ = 0, up_width_ = 0;
    int heads_, kv_heads_, dim_, vdim_, taps_, gate_act_;
    bool per_channel_, low_decay_, low_gate_;
    double eps_;
    std::string gemm_;
    Linear in_proj_, up_proj_, o_proj_;
    Tensor conv_, rate_, dt_bias_, norm_;
};

void register_delta_parts() {
    register_part("mixer", "delta_rule", [](const Json& p, BuildContext& b) { return std::make_shared<DeltaRule>(p, b); });
}

}  // namespace qe
