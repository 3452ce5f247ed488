// Sine and cosine of a rotary angle.  The angle is formed and brought into [-pi, pi] in double precision, its sine and cosine
// are taken in float32: a float32 product of a position in the thousands and a frequency near one is already off by 1e-4.
#pragma once

__device__ __forceinline__ void rotary_sincos(int position, double freq, float factor, float& sn, float& cs) {
  double angle = (double)position * freq;
  angle -= 6.283185307179586 * rint(angle * 0.15915494309189535);
  float s, c;
  sincosf((float)angle, &s, &c);
  sn = s * factor;
  cs = c * factor;
}
