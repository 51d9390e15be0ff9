// The Defapel design: pre-norm layers whose mixer is a gated delta rule with a decay per key channel, or attention over a
// window beside a gated delta rule with a decay per head, and whose feed-forward is a mixture of gated experts that take
// their weight on the input.
//
//     x <- x + mixer(rms(x) (1 + w1));  x <- x + experts(rms(x) (1 + w2));  logits = logit_scale * embed (rms(x) (1 + wf))
//
// config.json keys, all read here and nowhere else:
//   architecture ("Defapel"), vocab, width, norm.eps, logit_scale, layers[i].type ("channel_delta" | "parallel"),
//   layers[i].mixer, layers[i].mlp (null: the layer has no feed-forward);
//   channel_delta: heads, kv_heads, dim, vdim, conv; decay_rank and gate_rank (optional: the inner sizes of the two low-rank
//     products; without them the stored matrices give them, and only a folder can be loaded);
//   parallel: left {heads, kv_heads, dim, vdim, mask {size}, rot {base, dims, scaling {factor, low, high, original} or null},
//     scale, softcap}, right {heads, kv_heads, dim, vdim, conv}, left_scale, right_scale;
//   mlp: kind ("moe"), expert {ff}, router {experts, top};
//   max_position (optional): the longest sequence the rotary table is made for.
// Tensor names: embed, final.norm, and per layer i: l<i>.norm1, l<i>.norm2, of a delta rule under l<i>.mix. or l<i>.mix.right.:
// q, k, v, q.conv, k.conv, v.conv, b, A_log, dt_bias, norm, o, and a1, a2, g1, g2 (decay per channel) or a, g (per head); of the
// attention under l<i>.mix.left.: q, k, v, q.b, k.b, v.b, q.norm, k.norm, g, o; l<i>.mlp.{router, e<j>.gate, e<j>.up, e<j>.down}.
//
// What the design fixes and the code therefore states: norm weights are stored around zero; the attention's q, k and v have
// biases, its q and k are RMS-normed over all heads at once in front of the rotation, rotary pairs are (2i, 2i + 1), its heads
// are gated by sigmoids; the delta rule's gate is a sigmoid through a low rank where the decay is per channel, silu of one
// matrix where it is per head; router scores are sigmoids, chosen by themselves and not renormalised; experts use silu; the
// head is the embedding table.
#include "config.h"

namespace qe {

namespace {
constexpr long long kDefaultMaxPosition = 65536;

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
void check_heads(const Json& m, const std::string& where) {
    const long long heads = take_int(m, "heads"), kv = take_int(m, "kv_heads");
    if (heads % kv) throw ConfigError("config.json: " + where + std::to_string(heads) + " heads are not a multiple of " + std::to_string(kv) + " kv_heads");
    take_int(m, "dim");
    take_int(m, "vdim");
}
double positive(const Json& d, const std::string& key, const std::string& where) {
    const double v = take_float(d, key);
    if (!(v > 0.0)) throw ConfigError("config.json: " + where + key + " must be positive");
    return v;
}
}  // namespace

class DefapelConfig : public ModelConfig {
public:
    Json source;                        // config.json as read (checked)
    long long vocab = 0, width = 0, max_position = kDefaultMaxPosition;
    double eps = 0.0, logit_scale = 1.0;

    static std::unique_ptr<ModelConfig> read(const Json& d) {
        std::unique_ptr<DefapelConfig> c(new DefapelConfig());
        c->architecture = "Defapel";
        c->source = d;
        c->vocab = take_int(d, "vocab");
        c->width = take_int(d, "width");
        c->eps = positive(object_at(d, "norm", ""), "eps", "norm.");
        c->logit_scale = take_float(d, "logit_scale");
        c->max_position = take_int(d, "max_position", kDefaultMaxPosition, 1);
        const Json* layers = d.find("layers");
        if (!layers || !layers->is_array() || layers->size() == 0) throw ConfigError("config.json: 'layers' must be a non-empty list");
        for (size_t i = 0; i < layers->size(); i++) {
            const Json& l = (*layers)[i];
            const std::string where = "layers[" + std::to_string(i) + "].";
            if (!l.is_object()) throw ConfigError("config.json: " + where + " must be an object");
            const std::string type = l.get_string("type", "");
            const Json& m = object_at(l, "mixer", where);
            if (type == "channel_delta") {
                check_heads(m, where + "mixer: ");
                take_int(m, "conv");
                take_int(m, "decay_rank", 1, 1);
                take_int(m, "gate_rank", 1, 1);
            } else if (type == "parallel") {
                const Json& left = object_at(m, "left", where + "mixer.");
                const Json& right = object_at(m, "right", where + "mixer.");
                const std::string in_left = where + "mixer.left.";
                check_heads(left, in_left);
                take_int(object_at(left, "mask", in_left), "size");
                positive(left, "scale", in_left);
                positive(left, "softcap", in_left);
                const Json& rot = object_at(left, "rot", in_left);
                const long long dims = take_int(rot, "dims", 0);          // 0: no dimension is rotated
                if (dims % 2 || dims > take_int(left, "dim")) throw ConfigError("config.json: " + in_left + "rot.dims must be even and at most dim");
                positive(rot, "base", in_left + "rot.");
                if (has_value(rot, "scaling")) {
                    const Json& s = object_at(rot, "scaling", in_left + "rot.");
                    const std::string in_scaling = in_left + "rot.scaling.";
                    positive(s, "factor", in_scaling);
                    positive(s, "original", in_scaling);
                    if (positive(s, "low", in_scaling) > positive(s, "high", in_scaling))
                        throw ConfigError("config.json: " + in_scaling + "low exceeds high");
                }
                check_heads(right, where + "mixer.right: ");
                take_int(right, "conv");
                take_float(m, "left_scale");
                take_float(m, "right_scale");
            } else {
                throw ConfigError("config.json: " + where + "type '" + type + "' is not known (channel_delta, parallel)");
            }
            if (has_value(l, "mlp")) {
                const Json& f = object_at(l, "mlp", where);
                const std::string kind = f.get_string("kind", "");
                if (kind != "moe") throw ConfigError("config.json: " + where + "mlp.kind '" + kind + "' is not known (moe)");
                take_int(object_at(f, "expert", where + "mlp."), "ff");
                const Json& r = object_at(f, "router", where + "mlp.");
                if (take_int(r, "top") > take_int(r, "experts"))
                    throw ConfigError("config.json: " + where + "mlp.router: top " + std::to_string(take_int(r, "top")) + " of " +
                                      std::to_string(take_int(r, "experts")) + " experts cannot be chosen");
            }
        }
        return std::unique_ptr<ModelConfig>(c.release());
    }

    Json to_json() const override {
        Json d = source;
        d.set("architecture", "Defapel");
        return d;
    }

    ModelSpec build_spec() const override {
        auto norm = [&](const std::string& name) {
            Json p = Json::object();
            p.set("size", width);
            p.set("eps", eps);
            p.set("weight_offset", 1.0);
            p.set("names", names({{"weight", name}}));
            return PartSpec("rmsnorm", p);
        };
        ModelSpec spec;
        spec.hidden_size = width;
        spec.vocab_size = vocab;
        spec.max_position = max_position;
        const Json& layers = source.at("layers");
        for (size_t i = 0; i < layers.size(); i++) {
            const Json& l = layers[i];
            const Json& m = l.at("mixer");
            const std::string p = "l" + std::to_string(i) + ".";
            LayerSpec layer;
            layer.parts.push_back({"mixer_norm", norm(p + "norm1")});
            if (l.at("type").as_string() == "channel_delta") {
                layer.parts.push_back({"mixer", delta(m, p + "mix.", true)});
            } else {
                Json both = Json::object();
                both.set("hidden_size", width);
                both.set("combine", "weighted_sum");
                both.set("left_factor", m.at("left_scale"));
                both.set("right_factor", m.at("right_scale"));
                both.set("left", attention(m.at("left"), p + "mix.left.").to_json());
                both.set("right", delta(m.at("right"), p + "mix.right.", false).to_json());
                layer.parts.push_back({"mixer", PartSpec("side_by_side", both)});
            }
            if (has_value(l, "mlp")) {
                layer.parts.push_back({"feed_forward_norm", norm(p + "norm2")});
                layer.parts.push_back({"feed_forward", experts(l.at("mlp"), p + "mlp.")});
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
        h.set("tied_to", "embed");
        h.set("scale", logit_scale);
        spec.head = PartSpec("lm_head", h);
        spec.final_norm = norm("final.norm");
        spec.validate();
        return spec;
    }

private:
    PartSpec delta(const Json& m, const std::string& mp, bool per_channel) const {
        Json a = Json::object();
        a.set("hidden_size", width);
        a.set("num_heads", m.at("heads"));
        a.set("num_kv_heads", m.at("kv_heads"));
        a.set("head_dim", m.at("dim"));
        a.set("value_dim", m.at("vdim"));
        a.set("conv", m.at("conv"));
        a.set("norm_eps", eps);
        a.set("decay", per_channel ? "channel" : "head");
        a.set("gate", per_channel ? "sigmoid" : "silu");
        Json n = names({{"q_proj", mp + "q"}, {"k_proj", mp + "k"}, {"v_proj", mp + "v"}, {"q_conv", mp + "q.conv"}, {"k_conv", mp + "k.conv"},
                        {"v_conv", mp + "v.conv"}, {"beta_proj", mp + "b"}, {"a_log", mp + "A_log"}, {"dt_bias", mp + "dt_bias"},
                        {"norm", mp + "norm"}, {"o_proj", mp + "o"}});
        if (per_channel) {
            a.set("decay_rank", has_value(m, "decay_rank") ? m.at("decay_rank") : Json());
            a.set("gate_rank", has_value(m, "gate_rank") ? m.at("gate_rank") : Json());
            n.set("decay_down", mp + "a1");
            n.set("decay_up", mp + "a2");
            n.set("gate_down", mp + "g1");
            n.set("gate_up", mp + "g2");
        } else {
            n.set("decay_proj", mp + "a");
            n.set("gate_proj", mp + "g");
        }
        a.set("names", n);
        return PartSpec("delta_rule", a);
    }

    PartSpec attention(const Json& m, const std::string& mp) const {
        Json a = Json::object();
        a.set("hidden_size", width);
        a.set("num_heads", m.at("heads"));
        a.set("num_kv_heads", m.at("kv_heads"));
        a.set("head_dim", m.at("dim"));
        a.set("value_dim", m.at("vdim"));
        a.set("qk_norm_eps", eps);
        a.set("qk_norm_over", "row");
        a.set("bias", true);
        a.set("window", m.at("mask").at("size"));
        a.set("scale", m.at("scale"));
        a.set("softcap", m.at("softcap"));
        const Json& rot = m.at("rot");
        if (rot.at("dims").as_int() > 0) {
            Json pos = Json::object();
            pos.set("theta", rot.at("base"));
            pos.set("n_rot", rot.at("dims"));
            pos.set("max_position", max_position);
            pos.set("pairing", "interleaved");
            if (has_value(rot, "scaling")) {
                const Json& s = rot.at("scaling");
                Json scaling = Json::object();
                scaling.set("kind", "wavelength");
                for (const char* key : {"factor", "low", "high", "original"}) scaling.set(key, s.at(key));
                pos.set("scaling", scaling);
            }
            a.set("position", PartSpec("rope_neox", pos).to_json());
        } else {
            a.set("position", Json());
        }
        a.set("names", names({{"q_proj", mp + "q"}, {"k_proj", mp + "k"}, {"v_proj", mp + "v"}, {"o_proj", mp + "o"}, {"q_bias", mp + "q.b"},
                              {"k_bias", mp + "k.b"}, {"v_bias", mp + "v.b"}, {"q_norm", mp + "q.norm"}, {"k_norm", mp + "k.norm"},
                              {"gate_proj", mp + "g"}}));
        return PartSpec("attention", a);
    }

    PartSpec experts(const Json& f, const std::string& fp) const {
        const Json& router = f.at("router");
        Json g = Json::object();
        g.set("hidden_size", width);
        g.set("intermediate_size", f.at("expert").at("ff"));
        g.set("experts", router.at("experts"));
        g.set("top", router.at("top"));
        Json scoring = Json::object();
        scoring.set("kind", "sigmoid");
        g.set("scoring", scoring);
        g.set("weight_on", "input");
        g.set("names", names({{"router", fp + "router"}}));
        Json list = Json::array();
        for (long long e = 0; e < router.at("experts").as_int(); e++) {
            const std::string ep = fp + "e" + std::to_string(e) + ".";
            list.push(names({{"gate_proj", ep + "gate"}, {"up_proj", ep + "up"}, {"down_proj", ep + "down"}}));
        }
        g.set("expert_names", list);
        return PartSpec("routed_glu", g);
    }
};

void register_defapel_architecture() { register_architecture("Defapel", DefapelConfig::read); }

}  // namespace qe
