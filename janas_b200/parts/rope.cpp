// NeoX ("rotate half") rotary position encoding.
//
// theta(p, i) = (float)p * powf(theta, -2 i / rotary_dim), i < rotary_dim / 2; the
// pair (i, i + half) of a head is rotated by it (src/llm/model.c:100-113,
// src/llm/model_attn.c:31-39).  The powers are computed once on the host in double
// and rounded to float, as the reference's powf does (src/llm/jmath.c:131-134);
// the table of cos and sin is filled on the device from double-precision sincos of
// the float angle (src/llm/jmath.c:163-200) when the cache's size is known.
//
// rope_pairs is the same table for the layout that rotates neighbours: the pair
// (2i, 2i + 1) turns by theta(p, i) = (float)p * (float)(theta ^ (-2 i / rotary_dim)),
// the power taken in double and rounded once.  A mixer's own kernel applies it
// (csrc/latent.cu); rotary_dim may be shorter than what it is applied to.
//
// The rotation itself is applied by the attention kernel that also normalizes the
// heads and appends K and V (csrc/rope.cu); this part owns the constants and the
// table.  Only the whole head can be rotated (rotary_dim == head size); the
// reference's partial rotation (n_rot < head size) is not built.
#include <algorithm>
#include <cmath>

#include "part.h"

namespace jb {

namespace {

// params: rotary_dim, theta, max_positions, scaling (optional): {factor, low, high, original}, or
// yarn (optional): {factor, original, fast, slow}, or linear_factor (optional): every frequency is divided by it
class RopeNeox : public PositionEncoding {
public:
    RopeNeox(const PartSpec &s, DType dt, Device *d, bool pairs = false) : PositionEncoding(s, dt, d), pairs_(pairs) {
        rotary_dim_ = (int)s.get_int("rotary_dim");
        theta_ = s.get_double("theta");
        max_positions_ = s.get_int("max_positions");
        if (rotary_dim_ <= 0 || rotary_dim_ % 2) config_error("rope_neox: rotary_dim must be even and positive");
        int half = rotary_dim_ / 2;
        inv_freq_.resize((size_t)half);
        for (int i = 0; i < half; i++) {
            // the exponent in float arithmetic, the power in double, rounded once
            float expo = -2.0f * (float)i / (float)rotary_dim_;
            inv_freq_[(size_t)i] = pairs ? (float)std::pow(theta_, -2.0 * (double)i / (double)rotary_dim_)
                                         : (float)std::pow((double)(float)theta_, (double)expo);
        }
        if (s.has("scaling")) {
            // long wavelengths are stretched: with l = 2 pi / f, f stays where l < original / high,
            // becomes f / factor where l > original / low, and in between is the mix
            // (1 - t) f / factor + t f with t = (original / l - low) / (high - low)
            PartSpec sc{"", s.params.get("scaling")};
            double factor = sc.get_double("factor"), low = sc.get_double("low"), high = sc.get_double("high");
            double original = sc.get_double("original");
            if (factor <= 0 || original <= 0 || low <= 0 || high <= low)
                config_error("rope: scaling needs factor > 0, original > 0 and 0 < low < high");
            const double two_pi = 6.283185307179586476925286766559;
            for (int i = 0; i < half; i++) {
                double f = std::pow(theta_, -2.0 * (double)i / (double)rotary_dim_);
                double wavelength = two_pi / f;
                if (wavelength > original / low) {
                    f = f / factor;
                } else if (!(wavelength < original / high)) {
                    double t = (original / wavelength - low) / (high - low);
                    f = (1.0 - t) * f / factor + t * f;
                }
                inv_freq_[(size_t)i] = (float)f;
            }
        }
        if (s.has("linear_factor")) {
            double factor = s.get_double("linear_factor");
            if (s.has("scaling") || s.has("yarn")) config_error("rope: linear_factor excludes scaling and yarn");
            if (factor <= 0) config_error("rope: linear_factor must be positive");
            for (int i = 0; i < half; i++)
                inv_freq_[(size_t)i] = (float)(std::pow(theta_, -2.0 * (double)i / (double)rotary_dim_) / factor);
        }
        if (s.has("yarn")) {
            // YaRN ("YaRN: Efficient Context Window Extension of Large Language Models", Peng, Quesnelle,
            // Fan, Shippole): the frequency at index i turns `original` positions into t(i) full turns;
            // from the index of `fast` turns to the index of `slow` turns (both made whole) the
            // frequencies go over from f to f / factor along a straight ramp, and cos and sin are
            // multiplied by 0.1 ln(factor) + 1.
            if (s.has("scaling")) config_error("rope: scaling and yarn exclude each other");
            PartSpec yn{"", s.params.get("yarn")};
            double factor = yn.get_double("factor"), original = yn.get_double("original");
            double fast = yn.get_double("fast"), slow = yn.get_double("slow");
            if (factor <= 0 || original <= 0 || fast <= 0 || slow <= 0 || theta_ <= 0 || theta_ == 1.0)
                config_error("rope: yarn needs factor, original, fast, slow and theta above 0 and theta other than 1");
            const double two_pi = 6.283185307179586476925286766559;
            auto index_of = [&](double turns) {
                return (double)rotary_dim_ * std::log(original / (two_pi * turns)) / (2.0 * std::log(theta_));
            };
            double lo = std::max(std::floor(index_of(fast)), 0.0);
            double hi = std::min(std::ceil(index_of(slow)), (double)(rotary_dim_ - 1));
            for (int i = 0; i < half; i++) {
                double f = std::pow(theta_, -2.0 * (double)i / (double)rotary_dim_);
                double ramp = std::min(std::max(((double)i - lo) / std::max(hi - lo, 0.001), 0.0), 1.0);
                inv_freq_[(size_t)i] = (float)(f / factor * ramp + f * (1.0 - ramp));
            }
            amplitude_ = 0.1 * std::log(factor) + 1.0;
        }
    }

    void prepare(long long n_positions) override {
        long long n = std::min(n_positions, max_positions_);
        if (n <= n_) return;
        if (!dev) fail(JB_LLM_EFAIL, "rope_neox: no device to fill the table on");
        dev->make_current();
        int half = rotary_dim_ / 2;
        DevTensor inv = dev->tensor(F32, {half});
        cuda_check(cudaMemcpy(inv.ptr, inv_freq_.data(), (size_t)half * 4, cudaMemcpyHostToDevice),
                   "copying the rotation's frequencies");
        DevTensor c = dev->tensor(F32, {n, half}), s = dev->tensor(F32, {n, half});
        ops::rope_table(*dev, (const float *)inv.ptr, half, n, (float *)c.ptr, (float *)s.ptr, amplitude_);
        dev->sync();
        cos_ = c;
        sin_ = s;
        n_ = n;
    }

    const float *cos() const override { return (const float *)cos_.ptr; }
    const float *sin() const override { return (const float *)sin_.ptr; }
    int rotary_dim() const override { return rotary_dim_; }
    bool pairs() const override { return pairs_; }
    long long n_positions() const override { return n_; }

    Json info() const override {
        Json o = Json::object();
        o.set("rotary_dim", rotary_dim_);
        o.set("n_positions", n_);
        o.set("cos", (unsigned long long)(uintptr_t)cos_.ptr);
        o.set("sin", (unsigned long long)(uintptr_t)sin_.ptr);
        return o;
    }

private:
    int rotary_dim_;
    bool pairs_ = false;
    double theta_, amplitude_ = 1.0;     // amplitude: a factor on cos and sin
    long long max_positions_;
    std::vector<float> inv_freq_;
    DevTensor cos_, sin_;
    long long n_ = 0;
};

// No position encoding: q and k are used as they are.
class NoPosition : public PositionEncoding {
public:
    using PositionEncoding::PositionEncoding;
};

}  // namespace

void register_builtin_positions() {
    register_part("position", "rope_neox", [](const PartSpec &s, DType dt, Device *d) {
        return std::unique_ptr<Part>(new RopeNeox(s, dt, d));
    });
    register_part("position", "rope_pairs", [](const PartSpec &s, DType dt, Device *d) {
        return std::unique_ptr<Part>(new RopeNeox(s, dt, d, true));
    });
    register_part("position", "none", [](const PartSpec &s, DType dt, Device *d) {
        return std::unique_ptr<Part>(new NoPosition(s, dt, d));
    });
}

}  // namespace jb
