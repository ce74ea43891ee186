// Angles of rotated positions.
#pragma once

#include <cuda_runtime.h>

namespace ps {

// sine and cosine of pos * freq: the angle is reduced to one turn in double precision
__device__ __forceinline__ void turn_angle(int pos, double freq, float* s, float* c) {
    const double a = (double)pos * freq;
    sincosf((float)(a - 6.283185307179586 * rint(a * 0.15915494309189535)), s, c);
}

}  // namespace ps
