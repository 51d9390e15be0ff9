// Rotary position encoding, rotate-half pairing.
//
// For pair i < n_rot/2 the angle at position p is p * theta^(-2i/n_rot) (times an optional per-pair frequency
// factor); (x_i, x_{i+n_rot/2}) turns by it; dimensions >= n_rot are left alone.  Angles are computed in double
// precision on the host and stored as float32 cosines and sines.  Reference: src/qwen_ops.cpp:15-24 (double
// theta), src/attention.hip:225-240 (the device version); base and width: src/inference.cpp:1358-1359; the
// frequency factors and the interleaved pairing are the reference's knobs of src/attention.h:69, 84-95.
//
// Scaling for contexts longer than the trained one ("scaling": {"kind": "yarn", factor, original, fast, slow}): the
// pair whose wavelength makes t turns over `original` positions is pair(t) = n_rot * ln(original / (2 pi t)) / (2 ln
// theta); with lo = max(floor(pair(fast)), 0), hi = min(ceil(pair(slow)), n_rot - 1) and ramp_i = clamp((i - lo) /
// max(hi - lo, 0.001), 0, 1), pair i turns with f_i / factor * ramp_i + f_i * (1 - ramp_i) (fast pairs keep their
// frequency, slow ones are stretched by the factor), and every cosine and sine is multiplied by 0.1 ln(factor) + 1.
// Scaling by wavelength ("scaling": {"kind": "wavelength", factor, low, high, original}): a pair of frequency f makes
// t = original f / (2 pi) turns over `original` positions; it keeps f when t > high, turns with f / factor when t < low, and
// in between with ((1 - s) / factor + s) f, s = (t - low) / (high - low).  Cosines and sines are not stretched.
#include <algorithm>
#include <cmath>

#include "parts.h"

namespace qe {

// params: theta, n_rot, max_position; optional pairing ("half" | "interleaved"), freq_factors [n_rot/2] (each
// pair's frequency is divided by its factor), scaling (null, or {"kind": "yarn" | "wavelength", ...} as above),
// position_column.
class RotaryTable : public PositionEncoding {
public:
    RotaryTable(const Json& p, BuildContext& b) : PositionEncoding(p, b) {
        theta_ = p.at("theta").as_double();
        n_rot_ = (int)p.at("n_rot").as_int();
        max_position_ = p.at("max_position").as_int();
        interleaved_ = p.get_string("pairing", "half") == "interleaved";
        column_ = (int)p.get_int("position_column", 0);
        if (n_rot_ % 2 || n_rot_ < 2) throw ConfigError("rotary width " + std::to_string(n_rot_) + " must be even and at least 2");
        if (!(theta_ > 0) || max_position_ < 1) throw ConfigError("rotary: theta must be positive and max_position at least 1");
        if (const Json* f = p.find("freq_factors")) {
            if (!f->is_null()) {
                if (!f->is_array() || (int)f->size() != n_rot_ / 2) throw ConfigError("rotary: freq_factors must list n_rot/2 numbers");
                for (const Json& v : f->items()) factors_.push_back(v.as_double());
            }
        }
        if (const Json* sc = p.find("scaling")) {
            if (!sc->is_null()) {
                const std::string kind = sc->get_string("kind", "");
                if (kind != "yarn" && kind != "wavelength")
                    throw ConfigError("rotary: scaling of kind '" + kind + "' is not known (yarn, wavelength)");
                factor_ = sc->at("factor").as_double();
                original_ = sc->at("original").as_double();
                if (kind == "wavelength") {
                    wavelength_ = true;
                    low_ = sc->at("low").as_double();
                    high_ = sc->at("high").as_double();
                    if (!(factor_ > 0) || !(original_ > 0) || !(low_ > 0) || !(high_ >= low_))
                        throw ConfigError("rotary: wavelength scaling needs positive factor, original and low, and high not below low");
                    return;
                }
                yarn_ = true;
                fast_ = sc->at("fast").as_double();
                slow_ = sc->at("slow").as_double();
                if (!(factor_ > 0) || !(original_ > 0) || !(fast_ > 0) || !(slow_ > 0) || !(theta_ != 1.0))
                    throw ConfigError("rotary: yarn scaling needs positive factor, original, fast and slow");
            }
        }
    }
    int n_rot() const override { return n_rot_; }
    bool interleaved() const override { return interleaved_; }
    int position_column() const override { return column_; }

    void bind(WeightSource& src) override {
        if (table_.defined()) return;                     // shared by all layers: made once
        const int half = n_rot_ / 2;
        std::vector<float> host((size_t)max_position_ * n_rot_);
        std::vector<double> inv(half);
        for (int i = 0; i < half; i++) {
            inv[i] = std::pow(theta_, -2.0 * i / n_rot_);
            if (!factors_.empty()) inv[i] /= factors_[i];
        }
        double stretch = 1.0;
        const double kPi = 3.14159265358979323846;
        if (wavelength_)
            for (int i = 0; i < half; i++) {
                const double wave = 2.0 * kPi / inv[i];
                if (wave < original_ / high_) continue;
                if (wave > original_ / low_) { inv[i] /= factor_; continue; }
                const double s = high_ > low_ ? (original_ / wave - low_) / (high_ - low_) : 1.0;
                inv[i] = (1.0 - s) * inv[i] / factor_ + s * inv[i];
            }
        if (yarn_) {
            auto pair_of = [&](double turns) { return n_rot_ * std::log(original_ / (2.0 * kPi * turns)) / (2.0 * std::log(theta_)); };
            const double lo = std::max(std::floor(pair_of(fast_)), 0.0), hi = std::min(std::ceil(pair_of(slow_)), (double)n_rot_ - 1.0);
            for (int i = 0; i < half; i++) {
                const double ramp = std::min(std::max(((double)i - lo) / std::max(hi - lo, 0.001), 0.0), 1.0);
                inv[i] = inv[i] / factor_ * ramp + inv[i] * (1.0 - ramp);
            }
            stretch = 0.1 * std::log(factor_) + 1.0;
        }
        for (int64_t pos = 0; pos < max_position_; pos++)
            for (int i = 0; i < half; i++) {
                const double a = (double)pos * inv[i];
                host[(size_t)pos * n_rot_ + i] = (float)(std::cos(a) * stretch);
                host[(size_t)pos * n_rot_ + half + i] = (float)(std::sin(a) * stretch);
            }
        table_ = src.arena().alloc(DType::F32, {max_position_, n_rot_});
        QE_CUDA(cudaMemcpy(table_.data, host.data(), host.size() * sizeof(float), cudaMemcpyHostToDevice));
    }
    Tensor rotation_table() override { return table_; }

private:
    double theta_;
    int n_rot_, column_;
    int64_t max_position_;
    bool interleaved_;
    bool yarn_ = false, wavelength_ = false;
    double factor_ = 1.0, original_ = 0.0, fast_ = 0.0, slow_ = 0.0, low_ = 0.0, high_ = 0.0;
    std::vector<double> factors_;
    Tensor table_;
};

void register_position_parts() {
    register_part("position", "rope_neox", [](const Json& p, BuildContext& b) { return std::make_shared<RotaryTable>(p, b); });
}

}  // namespace qe
