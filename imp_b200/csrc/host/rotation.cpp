#include "rotation.hpp"

#include <algorithm>
#include <cmath>

namespace imp {

namespace {
constexpr double PI = 3.14159265358979323846;

double need(const Json& j, const char* key, const char* part) {
    const Json* v = j.find(key);
    if (!v || !v->is_number()) fail(IMP_ERROR_INVALID_MODEL, std::string(part) + ": rot_scaling lacks '" + key + "'");
    return v->as_double();
}

void slow_long_wavelengths(std::vector<double>& f, const Json& sc, const char* part) {
    const double factor = need(sc, "factor", part), low = need(sc, "low", part), high = need(sc, "high", part), original = need(sc, "original", part);
    if (!(factor > 0) || !(high > low) || !(low > 0) || !(original > 0))
        fail(IMP_ERROR_INVALID_MODEL, std::string(part) + ": rot_scaling needs factor > 0, 0 < low < high and original > 0");
    for (double& v : f) {
        const double wave = 2 * PI / v;
        if (wave > original / low) {
            v /= factor;
        } else if (!(wave < original / high)) {
            const double s = (original / wave - low) / (high - low);
            v = (1.0 - s) * v / factor + s * v;
        }
    }
}

void yarn(Rotation& r, const Json& sc, double base, int dims, const char* part) {
    const double factor = need(sc, "factor", part), original = need(sc, "original", part), fast = need(sc, "fast", part), slow = need(sc, "slow", part);
    if (!(factor > 0) || !(original > 0) || !(fast > 0) || !(slow > 0) || base == 1.0)
        fail(IMP_ERROR_INVALID_MODEL, std::string(part) + ": rot_scaling needs positive factor, original, fast and slow, and a base other than 1");
    // the (real) index of the pair that turns `turns` times over `original` positions
    auto index_of = [&](double turns) { return dims * std::log(original / (2 * PI * turns)) / (2 * std::log(base)); };
    const double lo = std::max(std::floor(index_of(fast)), 0.0), hi = std::min(std::ceil(index_of(slow)), dims - 1.0);
    for (size_t i = 0; i < r.freq.size(); ++i) {
        const double ramp = std::min(std::max(((double)i - lo) / std::max(hi - lo, 0.001), 0.0), 1.0);
        r.freq[i] = r.freq[i] / factor * ramp + r.freq[i] * (1.0 - ramp);
    }
    r.mult = 0.1 * std::log(factor) + 1.0;
}
}  // namespace

std::vector<float> Rotation::turns() const {
    const size_t n = freq.size();
    std::vector<float> t(2 * n);
    for (size_t i = 0; i < n; ++i) {
        const double v = freq[i] / (2 * PI);
        t[i] = (float)v;
        t[n + i] = (float)(v - (double)t[i]);
    }
    return t;
}

Rotation rotation_frequencies(const Json& params, int dims, const char* part) {
    Rotation r;
    const double base = params.get_double("rot_base", 10000.0);
    if (!(base > 0)) fail(IMP_ERROR_INVALID_MODEL, std::string(part) + ": rot_base must be positive");
    for (int i = 0; i < dims / 2; ++i) r.freq.push_back(std::pow(base, -2.0 * i / dims));
    const Json* sc = params.find("rot_scaling");
    if (!sc || !sc->is_object()) return r;
    const std::string kind = sc->get_string("kind", "wavelengths");
    if (kind == "wavelengths") slow_long_wavelengths(r.freq, *sc, part);
    else if (kind == "yarn") yarn(r, *sc, base, dims, part);
    else fail(IMP_ERROR_INVALID_MODEL, std::string(part) + ": unknown rot_scaling kind '" + kind + "' (known: wavelengths, yarn)");
    return r;
}

}  // namespace imp
