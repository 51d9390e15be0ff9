// The Noditar design: a decoder whose residual is several streams per token that every part reads as one weighted sum and
// that are mixed with each other at every addition, with three kinds of mixers.
//
//     X[s] = embed[token] for every stream s
//     a part f (mixer, feed-forward) with vectors a, b and a matrix M:   u = sum_s a[s] X[s],  y = f(rms(u; norm)),
//         X[t] <- sum_s M[s, t] X[s] + b[t] y
//     logits = head rms(sum_s X[s]; final.norm)
//   mixer "latent_attention": q = W_q h; a latent c = rms(W_dkv h) per token, keys W_uk c and values W_uv c per head, no
//     positions; the heads times sigmoid(W_g h), element by element; W_o.
//   mixer "attention": grouped-query attention with q and k divided by their root mean square per head, a bias of
//     2^(-8 (h + 1) / heads) per position of distance, a softmax with one added to its denominator, the same gate.
//   mixer "mamba2": the second Mamba form (parts/mamba.cpp).
//   feed-forward "dense": g' sigmoid(1.702 g') (u' + 1) with g' = min(g, limit), u' = clamp(u, -limit, limit).
//
// config.json keys, all read here and nowhere else:
//   architecture ("Noditar"), vocab, width, streams, norm.eps, layers[i].type ("latent_attention" | "attention" | "mamba2"),
//   layers[i].mixer, layers[i].mlp (null: no feed-forward; kind "dense": ff, limit);
//   latent_attention: heads, dim, vdim, kv_rank, scale;  attention: heads, kv_heads, dim, vdim, scale;
//   mamba2: heads, vdim, state, groups, conv, norm_groups;
//   max_position (optional): the longest sequence that is taken.
// Tensor names: embed, head, final.norm, and per layer i: l<i>.norm1, l<i>.norm2, l<i>.hc1.{in, out, mix}, l<i>.hc2.{in, out,
// mix}, l<i>.mix.{q, dkv, dkv.norm, uk, uv, g, o} or {q, k, v, g, o} or {in, conv, conv.b, dt_bias, A_log, D, norm, o},
// l<i>.mlp.{gate, up, down}.
//
// What the design fixes and the code therefore states: plain RMS norms; the slopes of the distance bias; the sink's score
// of 0; sigmoid gates of one logit per value; the gate's constants 1.702 and 1.
#include <cmath>

#include "config.h"

namespace qe {

namespace {
constexpr long long kDefaultMaxPosition = 65536;
constexpr double kGateAlpha = 1.702, kGateShift = 1.0;
constexpr double kSlopeRange = 8.0;          // the heads' slopes run down to 2^-8
constexpr double kSinkScore = 0.0;
constexpr long long kMaxStreams = 32;

Json names(std::initializer_list<std::pair<const char*, std::string>> list) {
    Json n = Json::object();
    for (const auto& kv : list) n.set(kv.first, kv.second);
    return n;
}
const Json& object_at(const Json& d, const std::string& key, const std::string& where) {
    const Json* v = d.find(key);
    if (!v || !v->is_object()) throw ConfigError("config.json: " + where + "'" + key + "' must be an object");
    return *v;
}
void check_multiple(const Json& m, const std::string& where, const char* what, const char* of) {
    if (take_int(m, what) % take_int(m, of))
        throw ConfigError("config.json: " + where + what + " " + std::to_string(take_int(m, what)) + " is no multiple of " + of + " " + std::to_string(take_int(m, of)));
}
}  // namespace

class NoditarConfig : public ModelConfig {
public:
    Json source;                        // config.json as read (checked)
    long long vocab = 0, width = 0, streams = 0, max_position = kDefaultMaxPosition;
    double eps = 0.0;

    static std::unique_ptr<ModelConfig> read(const Json& d) {
        std::unique_ptr<NoditarConfig> c(new NoditarConfig());
        c->architecture = "Noditar";
        c->source = d;
        c->vocab = take_int(d, "vocab");
        c->width = take_int(d, "width");
        c->streams = take_int(d, "streams");
        if (c->streams > kMaxStreams) throw ConfigError("config.json: streams " + std::to_string(c->streams) + " exceeds the supported " + std::to_string(kMaxStreams));
        c->eps = take_float(object_at(d, "norm", ""), "eps");
        if (!(c->eps > 0.0)) throw ConfigError("config.json: norm.eps must be positive");
        c->max_position = take_int(d, "max_position", kDefaultMaxPosition, 1);
        const Json* layers = d.find("layers");
        if (!layers || !layers->is_array() || layers->size() == 0) throw ConfigError("config.json: 'layers' must be a non-empty list");
        for (size_t i = 0; i < layers->size(); i++) {
            const Json& l = (*layers)[i];
            const std::string where = "layers[" + std::to_string(i) + "].";
            if (!l.is_object()) throw ConfigError("config.json: " + where + " must be an object");
            const std::string type = l.get_string("type", "");
            const Json& m = object_at(l, "mixer", where);
            const std::string in_mixer = where + "mixer.";
            if (type == "latent_attention" || type == "attention") {
                take_int(m, "heads"); take_int(m, "dim"); take_int(m, "vdim");
                if (type == "attention") check_multiple(m, in_mixer, "heads", "kv_heads");
                else take_int(m, "kv_rank");
                if (!(take_float(m, "scale") > 0.0)) throw ConfigError("config.json: " + in_mixer + "scale must be positive");
            } else if (type == "mamba2") {
                take_int(m, "vdim"); take_int(m, "state"); take_int(m, "conv");
                check_multiple(m, in_mixer, "heads", "groups");
                const long long inner = take_int(m, "heads") * take_int(m, "vdim"), parts = take_int(m, "norm_groups");
                if (inner % parts)
                    throw ConfigError("config.json: " + in_mixer + "norm_groups " + std::to_string(parts) + " does not divide the " + std::to_string(inner) + " channels");
            } else {
                throw ConfigError("config.json: " + where + "type '" + type + "' is not known (latent_attention, attention, mamba2)");
            }
            if (has_value(l, "mlp")) {
                const Json& f = object_at(l, "mlp", where);
                const std::string kind = f.get_string("kind", "");
                if (kind != "dense") throw ConfigError("config.json: " + where + "mlp.kind '" + kind + "' is not known (dense)");
                take_int(f, "ff");
                if (!(take_float(f, "limit") > 0.0)) throw ConfigError("config.json: " + where + "mlp.limit must be positive");
            }
        }
        return std::unique_ptr<ModelConfig>(c.release());
    }

    Json to_json() const override {
        Json d = source;
        d.set("architecture", "Noditar");
        return d;
    }

    ModelSpec build_spec() const override {
        auto norm = [&](const std::string& name) {
            Json p = Json::object();
            p.set("size", width);
            p.set("eps", eps);
            p.set("names", names({{"weight", name}}));
            return PartSpec("rmsnorm", p);
        };
        ModelSpec spec;
        spec.hidden_size = width;
        spec.vocab_size = vocab;
        spec.max_position = max_position;
        spec.residual_lanes = (int)streams;
        const Json& layers = source.at("layers");
        for (size_t i = 0; i < layers.size(); i++) {
            const Json& l = layers[i];
            const std::string p = "l" + std::to_string(i) + ".";
            auto lane_names = [&](const std::string& q) { return names({{"in", p + q + ".in"}, {"out", p + q + ".out"}, {"mix", p + q + ".mix"}}); };
            LayerSpec layer;
            layer.arrangement = "hyper_connection";
            layer.params.set("lanes", streams);
            layer.params.set("mixer_names", lane_names("hc1"));
            layer.parts.push_back({"mixer_norm", norm(p + "norm1")});
            layer.parts.push_back({"mixer", mixer(l.at("type").as_string(), l.at("mixer"), p + "mix.")});
            if (has_value(l, "mlp")) {
                const Json& f = l.at("mlp");
                Json gate = Json::object();
                gate.set("kind", "clamped_swish");
                gate.set("alpha", kGateAlpha);
                gate.set("limit", f.at("limit"));
                gate.set("shift", kGateShift);
                Json g = Json::object();
                g.set("hidden_size", width);
                g.set("intermediate_size", f.at("ff"));
                g.set("activation", gate);
                g.set("names", names({{"gate_proj", p + "mlp.gate"}, {"up_proj", p + "mlp.up"}, {"down_proj", p + "mlp.down"}}));
                layer.params.set("feed_forward_names", lane_names("hc2"));
                layer.parts.push_back({"feed_forward_norm", norm(p + "norm2")});
                layer.parts.push_back({"feed_forward", PartSpec("swiglu", g)});
            }
            spec.layers.push_back(std::move(layer));
            spec.schedule.push_back(LayerCall{(int)i, -1, 0});
        }
        Json e = Json::object();
        e.set("vocab_size", vocab);
        e.set("hidden_size", width);
        e.set("names", names({{"weight", "embed"}}));
        spec.embedding = PartSpec("embedding", e);
        Json h = Json::object();
        h.set("hidden_size", width);
        h.set("vocab_size", vocab);
        h.set("names", names({{"weight", "head"}}));
        spec.head = PartSpec("lm_head", h);
        spec.final_norm = norm("final.norm");
        spec.validate();
        return spec;
    }

private:
    PartSpec mixer(const std::string& type, const Json& m, const std::string& mp) const {
        Json a = Json::object();
        a.set("hidden_size", width);
        a.set("num_heads", m.at("heads"));
        a.set("value_dim", m.at("vdim"));
        if (type == "mamba2") {
            a.set("state", m.at("state"));
            a.set("groups", m.at("groups"));
            a.set("conv", m.at("conv"));
            a.set("norm_groups", m.at("norm_groups"));
            a.set("norm_eps", eps);
            a.set("names", names({{"in_proj", mp + "in"}, {"conv_weight", mp + "conv"}, {"conv_bias", mp + "conv.b"}, {"dt_bias", mp + "dt_bias"},
                                  {"a_log", mp + "A_log"}, {"d", mp + "D"}, {"norm", mp + "norm"}, {"out_proj", mp + "o"}}));
            return PartSpec("mamba2", a);
        }
        a.set("head_dim", m.at("dim"));
        a.set("scale", m.at("scale"));
        a.set("window", Json(0));
        a.set("position", Json());
        if (type == "latent_attention") {
            a.set("rot_dim", Json(0));
            a.set("q_rank", Json());
            a.set("kv_rank", m.at("kv_rank"));
            a.set("norm_eps", eps);
            a.set("gate", "values");
            a.set("names", names({{"q_proj", mp + "q"}, {"kv_down", mp + "dkv"}, {"kv_norm", mp + "dkv.norm"}, {"k_up", mp + "uk"}, {"v_up", mp + "uv"},
                                  {"gate", mp + "g"}, {"o_proj", mp + "o"}}));
            return PartSpec("latent_attention", a);
        }
        const long long heads = take_int(m, "heads");
        Json slopes = Json::array();
        for (long long h = 0; h < heads; h++) slopes.push(std::exp2(-kSlopeRange * (double)(h + 1) / (double)heads));
        a.set("num_kv_heads", m.at("kv_heads"));
        a.set("qk_norm_eps", eps);
        a.set("qk_norm_weight", false);
        a.set("bias", false);
        a.set("distance_slopes", slopes);
        a.set("sink_value", kSinkScore);
        a.set("names", names({{"q_proj", mp + "q"}, {"k_proj", mp + "k"}, {"v_proj", mp + "v"}, {"gate_proj", mp + "g"}, {"o_proj", mp + "o"}}));
        return PartSpec("attention", a);
    }
};

void register_noditar_architecture() { register_architecture("Noditar", NoditarConfig::read); }

}  // namespace qe
