// Rotary positions: pair i of a head's first `dims` elements, (x_i, x_(i + dims / 2)), turns by position * base^(-2 i / dims).
//
// Angles are kept in turns: the host divides each pair's frequency by 2 pi in double precision, the device multiplies by the position and drops
// whole turns in double precision, and only the remaining fraction becomes a 32-bit number. Its sine and cosine are then as accurate at a far
// position as at a near one.
#pragma once
#include <cmath>
#include <vector>

namespace qtb {

inline std::vector<double> rotation_turns(int dims, double base) {
    std::vector<double> t(dims / 2);
    for (int i = 0; i < dims / 2; ++i) t[i] = std::pow(base, -2.0 * i / dims) / (2.0 * 3.141592653589793238462643);
    return t;
}

// cosine and sine of a pair's angle at a position
__device__ __forceinline__ float2 rotation(double turns, unsigned int pos) {
    double t = turns * static_cast<double>(pos);
    t -= rint(t);
    float s, c;
    sincospif(2.0f * static_cast<float>(t), &s, &c);
    return make_float2(c, s);
}
__device__ __forceinline__ float2 rotate_pair(float u, float v, float2 cs) { return make_float2(u * cs.x - v * cs.y, v * cs.x + u * cs.y); }

}  // namespace qtb
