// Residual stream kept in fp32: a sublayer's result enters it through an optional elementwise gate and an optional
// RMSNorm, and the norm in front of the next sublayer is taken in the same pass.
//
//   y = sum over the row's slots of y_in                     (one slot, or the choices of a mixture of experts)
//   t = sigmoid(gate + bias) * y                              (gate may be absent)
//   r = resid + RMSNorm(t) * post_weight                      (post_weight absent: r = resid + t)
//   normed = RMSNorm(r) * next_weight                         rounded once to the storage type (next_weight absent: r)
//
// One CTA per row; the row stays in registers between the two reductions, so every array is read or
// written once.  The embedding gather that starts the stream is the same kernel without gate, post norm and residual.
#include "common.cuh"

namespace lri {
namespace {

struct GatedNormParams {
  const float* resid;       // [rows, dim] or NULL (zero); may alias resid_out
  const void* y;            // rows of `dim` elements
  const int32_t* slots;     // [rows, n_slots] row of y per slot, or NULL: row * n_slots + slot
  const int64_t* slots64;   // same, 64-bit (embedding ids)
  int n_slots;
  int64_t y_rows;           // rows of y (slot numbers are clamped into it)
  const float* gate;        // [rows, gate_ld] pre-activation, or NULL
  int64_t gate_ld;
  const void* gate_bias;    // [dim]
  const void* post_weight;  // [dim] or NULL
  float* resid_out;         // [rows, dim]
  const void* next_weight;  // [dim] or NULL
  void* normed_out;         // [rows, dim]
  float eps;
  int dim;
};

template <typename T, int VEC>
__device__ __forceinline__ void load_v(const T* p, float (&f)[VEC]) {
  if constexpr (VEC == 8) {
    load8<T>(p, f);
  } else {
    f[0] = Num<T>::to_f(p[0]);
  }
}
template <typename T, int VEC>
__device__ __forceinline__ void store_v(T* p, const float (&f)[VEC]) {
  if constexpr (VEC == 8) {
    store8<T>(p, f);
  } else {
    p[0] = Num<T>::from_f(f[0]);
  }
}

// PRE (few rows): the kernel is a chain of load latencies, so everything that can be loaded at once is.
template <typename T, int VEC, int NV, int THREADS, bool PRE>
__global__ void __launch_bounds__(THREADS) gated_norm_add_kernel(const GatedNormParams p) {
  __shared__ float part[33];
  const int64_t row = blockIdx.x;
  const int dim = p.dim, nvec = dim / VEC;
  const T* y = static_cast<const T*>(p.y);
  const T* bias = static_cast<const T*>(p.gate_bias);
  const T* wpost = static_cast<const T*>(p.post_weight);
  const T* wnext = static_cast<const T*>(p.next_weight);
  // constants of the model: fetched while the preceding kernel drains
  [[maybe_unused]] float cb[NV][VEC], cp[NV][VEC], cn[NV][VEC];
  if constexpr (PRE) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int v = threadIdx.x + i * THREADS;
      if (v >= nvec) continue;
      if (p.gate) load_v<T, VEC>(bias + v * VEC, cb[i]);
      if (wpost) load_v<T, VEC>(wpost + v * VEC, cp[i]);
      if (wnext) load_v<T, VEC>(wnext + v * VEC, cn[i]);
    }
  }
  pdl_launch_dependents();
  pdl_wait();
  float t[NV][VEC];
  [[maybe_unused]] float res[NV][VEC];
  if constexpr (PRE) {
    if (p.resid)
#pragma unroll
      for (int i = 0; i < NV; ++i)
        if (threadIdx.x + i * THREADS < nvec) load_v<float, VEC>(p.resid + row * dim + (threadIdx.x + i * THREADS) * VEC, res[i]);
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int v = threadIdx.x + i * THREADS;
    if (v >= nvec) continue;
#pragma unroll
    for (int e = 0; e < VEC; ++e) t[i][e] = 0.f;
    for (int s = 0; s < p.n_slots; ++s) {
      int64_t src = row * p.n_slots + s;
      if (p.slots) src = p.slots[src];
      if (p.slots64) src = p.slots64[src];
      src = src < 0 ? 0 : (src >= p.y_rows ? p.y_rows - 1 : src);
      float f[VEC];
      load_v<T, VEC>(y + src * dim + v * VEC, f);
#pragma unroll
      for (int e = 0; e < VEC; ++e) t[i][e] += f[e];
    }
    if (p.gate) {
      float g[VEC], b[VEC];
      load_v<float, VEC>(p.gate + row * p.gate_ld + v * VEC, g);
      if constexpr (PRE) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) b[e] = cb[i][e];
      } else {
        load_v<T, VEC>(bias + v * VEC, b);
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) t[i][e] *= sigmoid_f(g[e] + b[e]);
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) ss += t[i][e] * t[i][e];
  }
  float inv = 1.f;
  if (wpost) inv = 1.0f / sqrtf(block_sum(ss, part) / static_cast<float>(dim) + p.eps);
  ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int v = threadIdx.x + i * THREADS;
    if (v >= nvec) continue;
    if (wpost) {
      float w[VEC];
      if constexpr (PRE) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) w[e] = cp[i][e];
      } else {
        load_v<T, VEC>(wpost + v * VEC, w);
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) t[i][e] *= inv * w[e];
    }
    if (p.resid) {
      float r[VEC];
      if constexpr (PRE) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) r[e] = res[i][e];
      } else {
        load_v<float, VEC>(p.resid + row * dim + v * VEC, r);
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) t[i][e] += r[e];
    }
    if (p.resid_out) store_v<float, VEC>(p.resid_out + row * dim + v * VEC, t[i]);
#pragma unroll
    for (int e = 0; e < VEC; ++e) ss += t[i][e] * t[i][e];
  }
  if (!wnext) {
    if (!p.normed_out) return;
    T* sum_out = static_cast<T*>(p.normed_out) + row * dim;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int v = threadIdx.x + i * THREADS;
      if (v < nvec) store_v<T, VEC>(sum_out + v * VEC, t[i]);
    }
    return;
  }
  inv = 1.0f / sqrtf(block_sum(ss, part) / static_cast<float>(dim) + p.eps);
  T* out = static_cast<T*>(p.normed_out) + row * dim;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int v = threadIdx.x + i * THREADS;
    if (v >= nvec) continue;
    float w[VEC];
    if constexpr (PRE) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) w[e] = cn[i][e];
    } else {
      load_v<T, VEC>(wnext + v * VEC, w);
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) w[e] *= t[i][e] * inv;
    store_v<T, VEC>(out + v * VEC, w);
  }
}

template <typename T, int VEC, int NV, int THREADS, bool PRE = false>
int launch(const GatedNormParams& p, int64_t rows, cudaStream_t st) {
  LRI_CUDA(launch_pdl(gated_norm_add_kernel<T, VEC, NV, THREADS, PRE>, dim3(static_cast<unsigned>(rows)), dim3(THREADS), 0, st, p));
  LRI_LAUNCH_CHECK("gated_norm_add_kernel");
  return LRI_OK;
}

constexpr int kMaxDim = 16384;

template <typename T>
int dispatch(const GatedNormParams& p, int64_t rows, cudaStream_t st) {
  const bool vec = p.dim % 8 == 0 && p.gate_ld % 4 == 0 && aligned16(p.resid) && aligned16(p.y) && aligned16(p.gate) &&
                   aligned16(p.gate_bias) && aligned16(p.post_weight) && aligned16(p.resid_out) &&
                   aligned16(p.next_weight) && aligned16(p.normed_out);
  if (!vec) {
    if (p.dim <= 1024) return launch<T, 1, 4, 256>(p, rows, st);
    return launch<T, 1, 16, 1024>(p, rows, st);
  }
  const int nvec = p.dim / 8;
  if (rows <= 16 && nvec > 256) {  // few rows: the kernel is one thread's latency chain, spread the row
    if (nvec <= 512) return launch<T, 8, 1, 512, true>(p, rows, st);
    if (nvec <= 1024) return launch<T, 8, 1, 1024, true>(p, rows, st);
    return launch<T, 8, 2, 1024>(p, rows, st);
  }
  if (nvec <= 128) return launch<T, 8, 1, 128>(p, rows, st);
  if (nvec <= 256) return launch<T, 8, 1, 256>(p, rows, st);
  if (nvec <= 512) return launch<T, 8, 2, 256>(p, rows, st);
  if (nvec <= 1024) return launch<T, 8, 2, 512>(p, rows, st);
  return launch<T, 8, 4, 512>(p, rows, st);
}

int run(int dtype, const GatedNormParams& p, int64_t rows, cudaStream_t st) {
  if (dtype == LRI_BF16) return dispatch<__nv_bfloat16>(p, rows, st);
  if (dtype == LRI_FP16) return dispatch<__half>(p, rows, st);
  return dispatch<float>(p, rows, st);
}

}  // namespace
}  // namespace lri

using namespace lri;

extern "C" int lri_gated_norm_add(int dtype, const float* resid, const void* y, const int32_t* slots, int n_slots,
                                  int64_t y_rows, const float* gate, int64_t gate_ld, const void* gate_bias,
                                  const void* post_weight, float eps, float* resid_out, const void* next_weight,
                                  void* normed_out, int64_t rows, int dim, lri_stream_t stream) {
  LRI_REQUIRE(dtype >= LRI_BF16 && dtype <= LRI_FP32, LRI_ERR_UNSUPPORTED, "gated_norm_add: dtype %d", dtype);
  LRI_REQUIRE(y && (resid_out || normed_out), LRI_ERR_ARG, "gated_norm_add: NULL pointer");
  LRI_REQUIRE((gate == nullptr) == (gate_bias == nullptr), LRI_ERR_ARG, "gated_norm_add: gate and gate_bias go together");
  LRI_REQUIRE(next_weight == nullptr || normed_out != nullptr, LRI_ERR_ARG, "gated_norm_add: normed_out is NULL");
  LRI_REQUIRE(rows >= 0 && rows < (1ll << 31) && n_slots >= 1 && y_rows >= 1, LRI_ERR_ARG, "gated_norm_add: bad extent");
  LRI_REQUIRE(dim > 0 && dim <= kMaxDim, LRI_ERR_UNSUPPORTED, "gated_norm_add: dim=%d outside 1..%d", dim, kMaxDim);
  if (rows == 0) return LRI_OK;
  GatedNormParams p{};
  p.resid = resid, p.y = y, p.slots = slots, p.n_slots = n_slots, p.y_rows = y_rows;
  p.gate = gate, p.gate_ld = gate_ld, p.gate_bias = gate_bias, p.post_weight = post_weight;
  p.resid_out = resid_out, p.next_weight = next_weight, p.normed_out = normed_out, p.eps = eps, p.dim = dim;
  return run(dtype, p, rows, static_cast<cudaStream_t>(stream));
}

extern "C" int lri_embed_norm(int dtype, const void* table, const void* idx, int idx_is_i64, int64_t vocab, float* resid_out,
                              const void* weight, float eps, void* normed_out, int64_t rows, int dim, lri_stream_t stream) {
  LRI_REQUIRE(dtype >= LRI_BF16 && dtype <= LRI_FP32, LRI_ERR_UNSUPPORTED, "embed_norm: dtype %d", dtype);
  LRI_REQUIRE(table && idx && resid_out, LRI_ERR_ARG, "embed_norm: NULL pointer");
  LRI_REQUIRE((weight == nullptr) == (normed_out == nullptr), LRI_ERR_ARG, "embed_norm: weight and normed_out go together");
  LRI_REQUIRE(rows >= 0 && rows < (1ll << 31) && vocab > 0, LRI_ERR_ARG, "embed_norm: bad extent");
  LRI_REQUIRE(dim > 0 && dim <= kMaxDim, LRI_ERR_UNSUPPORTED, "embed_norm: dim=%d outside 1..%d", dim, kMaxDim);
  if (rows == 0) return LRI_OK;
  GatedNormParams p{};
  p.y = table, p.n_slots = 1, p.y_rows = vocab;
  if (idx_is_i64)
    p.slots64 = static_cast<const int64_t*>(idx);
  else
    p.slots = static_cast<const int32_t*>(idx);
  p.resid_out = resid_out, p.next_weight = weight, p.normed_out = normed_out, p.eps = eps, p.dim = dim;
  return run(dtype, p, rows, static_cast<cudaStream_t>(stream));
}
