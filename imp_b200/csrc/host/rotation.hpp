// Frequencies of rotary positions with their optional scalings, shared by the mixers that rotate.
#pragma once

#include <string>
#include <vector>

#include "parts.hpp"

namespace imp {

// Frequencies f_i (radians per position, i < dims / 2) and a factor on cos and sin.
struct Rotation {
    std::vector<double> freq;
    double mult = 1.0;
    // What the kernels read: [2][dims / 2] float32, a pair's turns per position (f_i / 2 pi) as the sum of two floats.
    std::vector<float> turns() const;
};

// f_i = rot_base^(-2i/dims), with params' optional `rot_scaling`:
//   {"factor", "low", "high", "original"}: long wavelengths slowed down; f kept where 2 pi / f < original / high, f / factor
//     where 2 pi / f > original / low, blended linearly in original / wavelength in between;
//   {"kind": "yarn", "factor", "original", "fast", "slow"}: blended linearly in the pair's index, from the pair that turns `fast`
//     times over `original` positions (f kept) to the one that turns `slow` times (f / factor); cos and sin times
//     0.1 ln(factor) + 1.
// `part` names the caller in errors.
Rotation rotation_frequencies(const Json& params, int dims, const char* part);

}  // namespace imp
