// Recurrences over a matrix state with a decay per key channel, per sequence and head:
//
//   gated linear attention   S <- g * S + k v^T                                                    o = S^T q
//   gated delta rule         S <- g * S;  u = beta (v - S^T k);  S <- S + k u^T                    o = S^T q
//
// g acts on the rows of S (key channels).  State, decays, step sizes and unit vectors are fp32 everywhere.
//
// Tokens are taken in blocks of T = 4.  With S the state before a block and products of decays over tokens of the block,
//   q'_t = q_t prod_{1..t} g      k'_t = k_t prod_{1..t} g      k"_s = k_s prod_{s+1..T} g      G = prod_{1..T} g
//   A[t, s] = k_t . (prod_{s+1..t} g * k_s)  (s < t)            B[t, s] = q_t . (prod_{s+1..t} g * k_s)  (s <= t)
// the block is, with u_t = v_t for gated linear attention,
//   u_t = beta_t (v_t - S^T k'_t - sum_{s<t} A[t, s] u_s)       o_t = S^T q'_t + sum_{s<=t} B[t, s] u_s
//   S <- G * S + sum_s k"_s u_s^T
// so the sums over the rows of S of all its tokens are independent.  Every product of decays is a running product, never a
// quotient or a difference of logarithms, so small decays are harmless.
#pragma once

#include "common.cuh"

namespace lri {

constexpr int kStateBlock = 4;  // tokens of a block
// coefficients of a block and head: beta_t, then A[t, s] (s < t), then B[t, s] as rows of four (zero for s > t)
constexpr int kCoef = 32, kCoefA = 4, kCoefB = 12;

// ---- packed fp32 pairs ---------------------------------------------------------------------------------
using f2 = unsigned long long;
__device__ __forceinline__ f2 mul2(f2 a, f2 b) {
  f2 d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ f2 fma2(f2 a, f2 b, f2 c) {
  f2 d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ f2 pack_f2(float lo, float hi) {
  f2 d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ void unpack_f2(f2 v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }
__device__ __forceinline__ f2 add2(f2 a, f2 b) {
  f2 d;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ float sum_f2(f2 v) {
  float a, b;
  unpack_f2(v, a, b);
  return a + b;
}

__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
// exp(-a softplus(z))
__device__ __forceinline__ float delta_decay_f(float z, float a) { return expf(-a * softplus_f(z)); }
// sigmoid(z)^(1 / tau)
__device__ __forceinline__ float logistic_decay_f(float z, float inv_tau) { return expf(-softplus_f(-z) * inv_tau); }

constexpr int kMaxTaps = 16;
constexpr float kUnitEps = 1e-6f;

}  // namespace lri
