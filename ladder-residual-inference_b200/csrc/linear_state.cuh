// Recurrences over a matrix state with a decay per key channel, per sequence and head:
//
//   gated linear attention   S <- g * S + k v^T                                                    o = S^T q
//   gated delta rule         S <- g * S;  u = beta (v - S^T k);  S <- S + k u^T                    o = S^T q
//
// g acts on the rows of S (key channels).  State, decays, step sizes and unit vectors are fp32 everywhere.
#pragma once

#include "common.cuh"

namespace lri {

__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
// exp(-exp(a_log) softplus(z))
__device__ __forceinline__ float delta_decay_f(float z, float a_log) { return expf(-expf(a_log) * softplus_f(z)); }
// sigmoid(z)^(1 / tau)
__device__ __forceinline__ float logistic_decay_f(float z, float inv_tau) { return expf(-softplus_f(-z) * inv_tau); }

constexpr int kMaxTaps = 16;

// Causal convolution over time of one channel: inputs at earlier positions come from the call's own rows or, before the
// call's first token, from the ring (the input of position q in slot q % taps); positions below 0 count as zero.
struct ConvInput {
  const float* proj;  // first row of the sequence in this call
  int64_t ld;
  const float* ring;  // [taps, channels] of the sequence
  int64_t ring_ld;
  int taps;
};
template <typename T>
__device__ __forceinline__ float short_conv(const ConvInput& c, const T* w, int64_t off, int64_t channel, int s, int64_t pos) {
  float y = 0.f;
  for (int j = c.taps - 1; j >= 0; --j) {  // j tokens back, oldest first
    float x = 0.f;
    if (s - j >= 0)
      x = c.proj[(s - j) * c.ld + off];
    else if (pos - j >= 0)
      x = c.ring[(pos - j) % c.taps * c.ring_ld + channel];
    y = fmaf(Num<T>::to_f(w[c.taps - 1 - j]), x, y);
  }
  return y;
}

}  // namespace lri
