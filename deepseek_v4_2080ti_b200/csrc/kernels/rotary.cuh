// Rotary angles of a position: the product with the fp64 frequency is reduced to one turn in fp64, sine and cosine are fp32.
#pragma once

namespace b200 {

__device__ __forceinline__ void rotary_angle(int position, double freq, float mscale, float& c, float& s) {
  const double turn = 6.283185307179586476925286766559;
  double a = (double)position * freq;
  a -= turn * rint(a / turn);
  sincosf((float)a, &s, &c);
  c *= mscale;
  s *= mscale;
}

}  // namespace b200
