// Rotation by position, shared by the kernels that turn a part of a head.
#pragma once

#include "rb_common.cuh"

// position * frequency in float64, brought into (-pi, pi] before the float32 sine and cosine
__device__ __forceinline__ void angle_sincos(int pos, double freq, float magnitude, float* sn, float* cs) {
  const double a = (double)pos * freq;
  const double turns = rint(a * 0.15915494309189535);
  const float r = (float)fma(-turns, 6.283185307179586, a);
  sincosf(r, sn, cs);
  *sn *= magnitude;
  *cs *= magnitude;
}

// value e of a head after the rotation of its first rot_dim values; val(i) gives the head's value i before it
template <typename F>
__device__ __forceinline__ float turned(F val, int e, int rot_dim, int interleaved, const float* s_sincos) {
  if (e >= rot_dim) return val(e);
  const int rhalf = rot_dim >> 1;
  int pair, other;
  bool first;
  if (interleaved) { pair = e >> 1; first = (e & 1) == 0; other = first ? e + 1 : e - 1; }
  else { first = e < rhalf; pair = first ? e : e - rhalf; other = first ? e + rhalf : e - rhalf; }
  const float sn = s_sincos[pair], cs = s_sincos[rhalf + pair];
  const float me = val(e), ot = val(other);
  return first ? me * cs - ot * sn : me * cs + ot * sn;
}
