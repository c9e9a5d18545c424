// Angles of rotary positions.  position * frequency is formed in float64 and brought into
// [-pi, pi] there (in float32 its rounding grows with the position); the sine and cosine of the
// reduced angle are float32.
#pragma once

#include "common.cuh"

namespace somi {

// (cosine, sine) of pos * freq
__device__ __forceinline__ float2 turn_by(double pos, double freq) {
    double angle = pos * freq;
    angle -= 6.283185307179586476925286766559 * rint(angle * 0.15915494309189533576888376337251);
    float sn, cs;
    sincosf(static_cast<float>(angle), &sn, &cs);
    return make_float2(cs, sn);
}

}  // namespace somi
