// What stands in front of the matrix-state recurrences (linear_state.cuh) when several tokens are fed:
//
//   delta_blocks   short convolutions over time, silu, unit queries and keys, decays, step sizes; block vectors and
//                  coefficients of the gated delta rule
//   gla_blocks     decays, block vectors and coefficients of gated linear attention
//   conv_ring      the last convolution inputs of the call become state
//   round_columns  columns of fp32 projections in the storage type (inputs of low-rank second projections)
#include "linear_state.cuh"

namespace lri {
namespace {

constexpr int kT = kStateBlock;

// Sums of N values (a power of two) over the warp; the lanes that share lane / (32 / N) get the sum of that value.
template <int N>
__device__ __forceinline__ float reduce_scatter(float (&a)[N], int lane) {
  int o = 16;
#pragma unroll
  for (int n = N / 2; n >= 1; n >>= 1, o >>= 1) {
    const bool up = lane & o;
#pragma unroll
    for (int i = 0; i < n; ++i) {
      const float give = up ? a[i] : a[i + n];
      a[i] = (up ? a[i + n] : a[i]) + __shfl_xor_sync(0xffffffffu, give, o);
    }
  }
#pragma unroll
  for (; o >= 1; o >>= 1) a[0] += __shfl_xor_sync(0xffffffffu, a[0], o);
  return a[0];
}

// Block vectors of one channel: q, k, g of its tokens -> q', k', k", G, and this channel's share of A and B.
struct BlockOut {
  float *qd, *kd, *ku;  // of token 0, pitch `pitch` from token to token
  int64_t pitch;
  float* decay;
};
template <bool DELTA>
__device__ __forceinline__ void block_channel(const float (&q)[kT], const float (&k)[kT], const float (&g)[kT], int64_t at, const BlockOut& o,
                                              float (&coef)[16]) {
  float w = 1.f;
#pragma unroll
  for (int t = 0; t < kT; ++t) {
    w *= g[t];
    o.qd[at + t * o.pitch] = q[t] * w;
    if (DELTA) o.kd[at + t * o.pitch] = k[t] * w;
  }
  o.decay[at] = w;
#pragma unroll
  for (int s = 0; s < kT; ++s) {
    float ks = k[s];
    coef[6 + s * (s + 1) / 2 + s] = fmaf(q[s], ks, coef[6 + s * (s + 1) / 2 + s]);
#pragma unroll
    for (int t = s + 1; t < kT; ++t) {
      ks *= g[t];
      if (DELTA) coef[t * (t - 1) / 2 + s] = fmaf(k[t], ks, coef[t * (t - 1) / 2 + s]);
      coef[6 + t * (t + 1) / 2 + s] = fmaf(q[t], ks, coef[6 + t * (t + 1) / 2 + s]);
    }
    o.ku[at + s * o.pitch] = ks;
  }
}
// the lanes' shares of A (6) and B (10) -> coefficients of the block
__device__ __forceinline__ void store_coef(float (&coef)[16], float* dst, int lane) {
  const float x = reduce_scatter<16>(coef, lane);
  // element 6 + t (t + 1) / 2 + s of B goes to row t, column s
  const int e = lane >> 1, i = e - 6, t = i < 1 ? 0 : (i < 3 ? 1 : (i < 6 ? 2 : 3));
  if ((lane & 1) == 0) dst[e < 6 ? kCoefA + e : kCoefB + kT * t + i - t * (t + 1) / 2] = x;
  if (lane < kT * kT && lane % kT > lane / kT) dst[kCoefB + lane] = 0.f;
}

struct DeltaBlocksParams {
  const float* proj;  // [rows, ld]
  int64_t ld, q_off, k_off, v_off, b_off;
  const void *conv_q, *conv_k, *conv_v;  // [channels, taps]
  int taps;
  const float* ring;  // [B, taps, 2 G C + H E]
  const float* z;     // [rows, H, C]
  const void *a_log, *dt_bias;
  const void* input_pos;
  int pos_is_i64;
  float *qd, *kd, *ku;  // [B * blocks * 4, H, C]
  float* decay;         // [B * blocks, H, C]
  float* coef;          // [B * blocks, H, 32]
  float* v;             // [rows, H, E]
  float q_scale;
  int S, H, G, C, E;
};

// Activation of a convolution: 16-bit models take it from the special-function unit (a few units in the last place of fp32).
template <typename T>
__device__ __forceinline__ float conv_silu(float x) {
  return sizeof(T) == 4 ? silu_f(x) : x * __fdividef(1.0f, 1.0f + __expf(-x));
}

// silu of the convolution of one channel at the block's tokens (zero past the n of them).  `in` is the input of the block's
// first token, s its place in the call, pos its position; inputs before the call come from the ring, those before the
// sequence are zero.
template <typename T, int TAPS>
__device__ __forceinline__ void conv_block(const float* in, int64_t ld, const T* w, const float* ring, int64_t channels, int taps, int s,
                                           int64_t pos, int n, float (&y)[kT]) {
  float x[TAPS - 1 + kT];  // the last kT: the block's tokens
#pragma unroll
  for (int t = 0; t < kT; ++t) x[TAPS - 1 + t] = t < n ? in[t * ld] : 0.f;
  float c[TAPS];  // leading taps that do not exist have weight zero
  const bool whole = TAPS == 4 && sizeof(T) == 2 && taps == 4 && (reinterpret_cast<uintptr_t>(w) & 7u) == 0;
  if (whole) {
    if constexpr (TAPS == 4 && sizeof(T) == 2) {
      const uint2 v = *reinterpret_cast<const uint2*>(w);
      Num<T>::unpack2(v.x, c[0], c[1]);
      Num<T>::unpack2(v.y, c[2], c[3]);
    }
  } else {
#pragma unroll
    for (int j = 0; j < TAPS; ++j) c[TAPS - 1 - j] = j < taps ? Num<T>::to_f(w[taps - 1 - j]) : 0.f;
  }
#pragma unroll
  for (int j = 0; j < TAPS; ++j) {  // j tokens back
    if (j > 0) {
      float v = 0.f;
      if (j < taps) {
        if (s - j >= 0)
          v = in[-j * ld];
        else if (pos - j >= 0)
          v = ring[(pos - j) % taps * channels];
      }
      x[TAPS - 1 - j] = v;
    }
  }
#pragma unroll
  for (int t = 0; t < kT; ++t) {
    float a = 0.f;
#pragma unroll
    for (int j = 0; j < TAPS; ++j) a = fmaf(c[j], x[t + j], a);
    y[t] = t < n ? conv_silu<T>(a) : 0.f;
  }
}

// One warp per (block, value head) for the vectors over key channels, and one for the values and the step size; a lane owns
// the channels lane, lane + 32, ...  CI > 0: at most 32 CI channels, whose q and
// k stay in registers over the unit norms' sums; CI = 0: any number, computed twice.
template <typename T, int CI, int TAPS>
__global__ void __launch_bounds__(256, CI > 0 ? 3 : 1) delta_blocks_kernel(const DeltaBlocksParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31, unit = blockIdx.y * 8 + (threadIdx.x >> 5);
  if (unit >= 2 * p.H) return;
  const int h = unit < p.H ? unit : unit - p.H;
  const int blocks = (p.S + kT - 1) / kT;
  const int64_t blk = blockIdx.x, b = blk / blocks;
  const int s = static_cast<int>(blk - b * blocks) * kT;
  const int n = p.S - s < kT ? p.S - s : kT;
  const int C = p.C, E = p.E, H = p.H, G = p.G, hk = h / (H / G);
  const int64_t row = b * p.S + s, pos = load_pos(p.input_pos, p.pos_is_i64, s);
  const int64_t channels = 2ll * G * C + static_cast<int64_t>(H) * E;
  const float* ring = p.ring + b * p.taps * channels;
  const float* in = p.proj + row * p.ld;
  if (unit >= p.H) {
    if (lane < kT) p.coef[(blk * H + h) * kCoef + lane] = lane < n ? sigmoid_f(in[lane * p.ld + p.b_off + h]) : 0.f;
#pragma unroll 2
    for (int e = lane; e < E; e += 32) {
      const int64_t ch = static_cast<int64_t>(h) * E + e;
      float y[kT];
      conv_block<T, TAPS>(in + p.v_off + ch, p.ld, static_cast<const T*>(p.conv_v) + ch * p.taps, ring + 2ll * G * C + ch, channels, p.taps, s,
                          pos, n, y);
#pragma unroll
      for (int t = 0; t < kT; ++t)
        if (t < n) p.v[(row + t) * H * E + ch] = y[t];
    }
    return;
  }

  auto conv_qk = [&](int c, float (&q)[kT], float (&k)[kT]) {
    const int64_t ch = static_cast<int64_t>(hk) * C + c;
    conv_block<T, TAPS>(in + p.q_off + ch, p.ld, static_cast<const T*>(p.conv_q) + ch * p.taps, ring + ch, channels, p.taps, s, pos, n, q);
    conv_block<T, TAPS>(in + p.k_off + ch, p.ld, static_cast<const T*>(p.conv_k) + ch * p.taps, ring + static_cast<int64_t>(G) * C + ch,
                        channels, p.taps, s, pos, n, k);
  };
  float sums[2 * kT];
#pragma unroll
  for (int i = 0; i < 2 * kT; ++i) sums[i] = 0.f;
  auto add_squares = [&](const float (&q)[kT], const float (&k)[kT]) {
#pragma unroll
    for (int t = 0; t < kT; ++t) sums[t] = fmaf(q[t], q[t], sums[t]), sums[kT + t] = fmaf(k[t], k[t], sums[kT + t]);
  };
  [[maybe_unused]] float qr[CI > 0 ? CI : 1][kT], kr[CI > 0 ? CI : 1][kT];
  if constexpr (CI > 0) {
#pragma unroll
    for (int i = 0; i < CI; ++i) {
      // (channels past the end repeat the last one and count nothing)
      conv_qk(lane + 32 * i < C ? lane + 32 * i : C - 1, qr[i], kr[i]);
      if (lane + 32 * i < C) add_squares(qr[i], kr[i]);
    }
  } else {
    for (int c = lane; c < C; c += 32) {
      float q[kT], k[kT];
      conv_qk(c, q, k);
      add_squares(q, k);
    }
  }
  const float mine = 1.0f / sqrtf(reduce_scatter<2 * kT>(sums, lane) + kUnitEps);
  float iq[kT], ik[kT];
#pragma unroll
  for (int t = 0; t < kT; ++t) {
    iq[t] = __shfl_sync(0xffffffffu, mine, 4 * t) * p.q_scale;
    ik[t] = __shfl_sync(0xffffffffu, mine, 4 * (kT + t));
  }

  const int64_t hc = static_cast<int64_t>(H) * C;
  const BlockOut out{p.qd + blk * kT * hc + h * C, p.kd + blk * kT * hc + h * C, p.ku + blk * kT * hc + h * C, hc, p.decay + blk * hc + h * C};
  const float a = expf(Num<T>::to_f(static_cast<const T*>(p.a_log)[h]));
  float coef[16];
#pragma unroll
  for (int i = 0; i < 16; ++i) coef[i] = 0.f;
  auto finish = [&](int c, const float (&q0)[kT], const float (&k0)[kT]) {
    const float bias = Num<T>::to_f(static_cast<const T*>(p.dt_bias)[h * C + c]);
    float q[kT], k[kT], g[kT];
#pragma unroll
    for (int t = 0; t < kT; ++t) {
      q[t] = q0[t] * iq[t], k[t] = k0[t] * ik[t];
      g[t] = t < n ? delta_decay_f(p.z[(row + t) * hc + h * C + c] + bias, a) : 1.f;
    }
    block_channel<true>(q, k, g, c, out, coef);
  };
  if constexpr (CI > 0) {
#pragma unroll
    for (int i = 0; i < CI; ++i) {
      if (lane + 32 * i < C) finish(lane + 32 * i, qr[i], kr[i]);
    }
  } else {
    for (int c = lane; c < C; c += 32) {
      float q[kT], k[kT];
      conv_qk(c, q, k);
      finish(c, q, k);
    }
  }
  store_coef(coef, p.coef + (blk * H + h) * kCoef, lane);
}

struct GlaBlocksParams {
  const float* proj;  // [rows, ld]
  int64_t ld, q_off, k_off;
  const float* z;  // [rows, H, C]
  const void* bias;
  float inv_tau, q_scale;
  float *qd, *ku, *decay, *coef;
  int S, H, C;
};

template <typename T>
__global__ void __launch_bounds__(256) gla_blocks_kernel(const GlaBlocksParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31, h = blockIdx.y * 8 + (threadIdx.x >> 5);
  if (h >= p.H) return;
  const int blocks = (p.S + kT - 1) / kT;
  const int64_t blk = blockIdx.x, b = blk / blocks;
  const int s = static_cast<int>(blk - b * blocks) * kT;
  const int n = p.S - s < kT ? p.S - s : kT;
  const int64_t row = b * p.S + s, hc = static_cast<int64_t>(p.H) * p.C;
  const BlockOut out{p.qd + blk * kT * hc + h * p.C, nullptr, p.ku + blk * kT * hc + h * p.C, hc, p.decay + blk * hc + h * p.C};
  float coef[16];
#pragma unroll
  for (int i = 0; i < 16; ++i) coef[i] = 0.f;
  for (int c = lane; c < p.C; c += 32) {
    const int ch = h * p.C + c;
    const float bias = Num<T>::to_f(static_cast<const T*>(p.bias)[ch]);
    float q[kT], k[kT], g[kT];
#pragma unroll
    for (int t = 0; t < kT; ++t) {
      const float* in = p.proj + (row + t) * p.ld;
      q[t] = t < n ? in[p.q_off + ch] * p.q_scale : 0.f;
      k[t] = t < n ? in[p.k_off + ch] : 0.f;
      g[t] = t < n ? p.z[(row + t) * hc + ch] : 0.f;
    }
#pragma unroll
    for (int t = 0; t < kT; ++t) g[t] = t < n ? logistic_decay_f(g[t] + bias, p.inv_tau) : 1.f;
    block_channel<false>(q, k, g, c, out, coef);
  }
  store_coef(coef, p.coef + (blk * p.H + h) * kCoef, lane);
}

// The inputs of the call's last `taps` tokens into the ring.  Runs behind delta_blocks, which reads older ones from it.
__global__ void __launch_bounds__(256)
conv_ring_kernel(const float* proj, int64_t ld, int64_t q_off, int64_t k_off, int64_t v_off, int nqk, int nv, float* ring, int taps,
                 const void* input_pos, int pos_is_i64, int S) {
  pdl_launch_dependents();
  pdl_wait();
  const int channels = 2 * nqk + nv;
  const int ch = blockIdx.x * 256 + threadIdx.x;
  const int64_t b = blockIdx.z;
  const int s = S - 1 - static_cast<int>(blockIdx.y);
  if (ch >= channels || s < 0) return;
  const int64_t pos = load_pos(input_pos, pos_is_i64, s);
  if (pos < 0) return;
  const int64_t off = ch < nqk ? q_off + ch : (ch < 2 * nqk ? k_off + ch - nqk : v_off + ch - 2 * nqk);
  ring[(b * taps + pos % taps) * channels + ch] = proj[(b * S + s) * ld + off];
}

// columns [off, off + n) of fp32 rows in the storage type
template <typename T>
__global__ void __launch_bounds__(256) round_columns_kernel(const float* x, int64_t ld, int64_t off, int n, T* y, int64_t count) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t i = static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x;
  if (i >= count) return;
  const int64_t r = i / n;
  y[i] = Num<T>::from_f(x[r * ld + off + (i - r * n)]);
}

template <typename T>
int delta_blocks(const DeltaBlocksParams& p, int B, cudaStream_t st) {
  auto kern = p.taps > 4 || p.C > 128 ? delta_blocks_kernel<T, 0, kMaxTaps> : (p.C <= 64 ? delta_blocks_kernel<T, 2, 4> : delta_blocks_kernel<T, 4, 4>);
  LRI_CUDA(launch_pdl(kern, dim3(static_cast<unsigned>(B) * ((p.S + kT - 1) / kT), (2 * p.H + 7) / 8), dim3(256), 0, st, p));
  LRI_LAUNCH_CHECK("delta_blocks_kernel");
  return LRI_OK;
}
template <typename T>
int gla_blocks(const GlaBlocksParams& p, int B, cudaStream_t st) {
  LRI_CUDA(launch_pdl(gla_blocks_kernel<T>, dim3(static_cast<unsigned>(B) * ((p.S + kT - 1) / kT), (p.H + 7) / 8), dim3(256), 0, st, p));
  LRI_LAUNCH_CHECK("gla_blocks_kernel");
  return LRI_OK;
}

bool dtype_ok(int dtype) { return dtype >= LRI_BF16 && dtype <= LRI_FP32; }

}  // namespace
}  // namespace lri

using namespace lri;

#define LRI_BY_TYPE(dtype, call) ((dtype) == LRI_BF16 ? call<__nv_bfloat16> : (dtype) == LRI_FP16 ? call<__half> : call<float>)

extern "C" int64_t lri_state_blocks(int64_t S) { return (S + kT - 1) / kT; }

extern "C" int lri_delta_blocks(int dtype, const float* proj, int64_t ld, int64_t q_off, int64_t k_off, int64_t v_off, int64_t b_off,
                                const void* conv_q, const void* conv_k, const void* conv_v, int taps, float* ring, const float* z,
                                const void* a_log, const void* dt_bias, const void* input_pos, int pos_is_i64, float* qd, float* kd,
                                float* ku, float* decay, float* coef, float* v, int B, int S, int heads, int kv_heads, int dim, int vdim,
                                lri_stream_t stream) {
  LRI_REQUIRE(dtype_ok(dtype), LRI_ERR_UNSUPPORTED, "delta_blocks: dtype %d", dtype);
  LRI_REQUIRE(proj && conv_q && conv_k && conv_v && ring && z && a_log && dt_bias && input_pos && qd && kd && ku && decay && coef && v,
              LRI_ERR_ARG, "delta_blocks: NULL pointer");
  LRI_REQUIRE(B >= 0 && B <= 65535 && S >= 0 && heads > 0 && heads <= 65535 && kv_heads > 0 && heads % kv_heads == 0 && dim > 0 && vdim > 0,
              LRI_ERR_ARG, "delta_blocks: B=%d S=%d heads=%d kv_heads=%d dim=%d vdim=%d", B, S, heads, kv_heads, dim, vdim);
  LRI_REQUIRE(taps >= 1 && taps <= kMaxTaps, LRI_ERR_UNSUPPORTED, "delta_blocks: taps=%d outside 1..%d", taps, kMaxTaps);
  if (B == 0 || S == 0) return LRI_OK;
  DeltaBlocksParams p{};
  p.proj = proj, p.ld = ld, p.q_off = q_off, p.k_off = k_off, p.v_off = v_off, p.b_off = b_off;
  p.conv_q = conv_q, p.conv_k = conv_k, p.conv_v = conv_v, p.taps = taps, p.ring = ring, p.z = z, p.a_log = a_log, p.dt_bias = dt_bias;
  p.input_pos = input_pos, p.pos_is_i64 = pos_is_i64, p.qd = qd, p.kd = kd, p.ku = ku, p.decay = decay, p.coef = coef, p.v = v;
  p.q_scale = 1.0f / sqrtf(static_cast<float>(dim)), p.S = S, p.H = heads, p.G = kv_heads, p.C = dim, p.E = vdim;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int rc = LRI_BY_TYPE(dtype, delta_blocks)(p, B, st);
  if (rc != LRI_OK) return rc;
  const int nqk = kv_heads * dim, nv = heads * vdim;
  LRI_CUDA(launch_pdl(conv_ring_kernel, dim3((2 * nqk + nv + 255) / 256, taps < S ? taps : S, B), dim3(256), 0, st, proj, ld, q_off, k_off,
                      v_off, nqk, nv, ring, taps, input_pos, pos_is_i64, S));
  LRI_LAUNCH_CHECK("conv_ring_kernel");
  return LRI_OK;
}

extern "C" int lri_gla_blocks(int dtype, const float* proj, int64_t ld, int64_t q_off, int64_t k_off, const float* z, const void* bias,
                              float tau, float* qd, float* ku, float* decay, float* coef, int B, int S, int heads, int dim,
                              lri_stream_t stream) {
  LRI_REQUIRE(dtype_ok(dtype), LRI_ERR_UNSUPPORTED, "gla_blocks: dtype %d", dtype);
  LRI_REQUIRE(proj && z && bias && qd && ku && decay && coef, LRI_ERR_ARG, "gla_blocks: NULL pointer");
  LRI_REQUIRE(B >= 0 && B <= 65535 && S >= 0 && heads > 0 && heads <= 65535 && dim > 0 && tau > 0.f, LRI_ERR_ARG,
              "gla_blocks: B=%d S=%d heads=%d dim=%d tau=%g", B, S, heads, dim, tau);
  if (B == 0 || S == 0) return LRI_OK;
  GlaBlocksParams p{};
  p.proj = proj, p.ld = ld, p.q_off = q_off, p.k_off = k_off, p.z = z, p.bias = bias, p.inv_tau = 1.0f / tau;
  p.q_scale = 1.0f / sqrtf(static_cast<float>(dim)), p.qd = qd, p.ku = ku, p.decay = decay, p.coef = coef, p.S = S, p.H = heads, p.C = dim;
  return LRI_BY_TYPE(dtype, gla_blocks)(p, B, static_cast<cudaStream_t>(stream));
}

extern "C" int lri_round_columns(int dtype, const float* x, int64_t ld, int64_t off, int n, void* y, int64_t rows, lri_stream_t stream) {
  LRI_REQUIRE(dtype_ok(dtype), LRI_ERR_UNSUPPORTED, "round_columns: dtype %d", dtype);
  LRI_REQUIRE(x && y && n > 0 && rows >= 0, LRI_ERR_ARG, "round_columns: n=%d rows=%lld", n, (long long)rows);
  const int64_t count = rows * n;
  if (count == 0) return LRI_OK;
  const unsigned grid = static_cast<unsigned>((count + 255) / 256);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
#define LRI_CALL(T) LRI_CUDA(launch_pdl(round_columns_kernel<T>, dim3(grid), dim3(256), 0, st, x, ld, off, n, static_cast<T*>(y), count))
  if (dtype == LRI_BF16)
    LRI_CALL(__nv_bfloat16);
  else if (dtype == LRI_FP16)
    LRI_CALL(__half);
  else
    LRI_CALL(float);
#undef LRI_CALL
  LRI_LAUNCH_CHECK("round_columns_kernel");
  return LRI_OK;
}
