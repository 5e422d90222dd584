// Residual held as several parallel streams (hyper-connections), fp32: a sublayer reads a weighted sum of the streams,
// and its result is written into all of them together with a mix of the old ones.
//
//   x_t' = sum_s mix[s, t] x_s + out[t] y          (old streams on the right)
//   u    = sum_s in[s] x_s'                         in: weights of the NEXT sublayer; absent: plain sum (the model's end)
//   normed = RMSNorm(u) * weight                    rounded once to the storage type
//
// One CTA per row: every stream is read and written once, u stays in registers over the reduction.  The embedding that
// starts the streams (all equal, scaled) is the same kernel with a gather in place of the mix.
#include "common.cuh"

#include <type_traits>

namespace lri {
namespace {

struct StreamParams {
  const float* x;  // [rows, streams, dim] (NULL: start from the table)
  float* x_out;    // may alias x; NULL: not written
  const void* table;
  const int32_t* idx32;
  const int64_t* idx64;
  int64_t vocab;
  float scale;
  const void* y;        // [rows, dim]
  const void* mix;      // [streams, streams], [from, to]
  const void* out;      // [streams]
  const void* in_next;  // [streams] or NULL
  const void* weight;   // [dim]
  float eps;
  void* normed;  // [rows, dim]
  int streams, dim;
};

constexpr int kVec = 4;
__device__ __forceinline__ void load_f(const float* p, float (&f)[kVec]) {
  const float4 v = *reinterpret_cast<const float4*>(p);
  f[0] = v.x, f[1] = v.y, f[2] = v.z, f[3] = v.w;
}
__device__ __forceinline__ void store_f(float* p, const float (&f)[kVec]) {
  *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
}
template <typename T>
__device__ __forceinline__ void load_t(const T* p, float (&f)[kVec]) {
  if constexpr (std::is_same<T, float>::value) {
    load_f(p, f);
  } else {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    Num<T>::unpack2(v.x, f[0], f[1]);
    Num<T>::unpack2(v.y, f[2], f[3]);
  }
}
template <typename T>
__device__ __forceinline__ void store_t(T* p, const float (&f)[kVec]) {
  if constexpr (std::is_same<T, float>::value)
    store_f(p, f);
  else
    *reinterpret_cast<uint2*>(p) = make_uint2(pack2<T>(f[0], f[1]), pack2<T>(f[2], f[3]));
}

// SM: bound of the number of streams.  NV vectors of four elements per thread.
template <typename T, int SM, int NV, int THREADS>
__global__ void __launch_bounds__(THREADS) join_streams_kernel(const StreamParams p) {
  __shared__ float part[33];
  __shared__ float mix[SM][SM], out[SM], in[SM];
  const int n = p.streams, dim = p.dim, nvec = dim / kVec;
  const int64_t row = blockIdx.x;
  if (threadIdx.x < SM) {
    const int t = threadIdx.x;
    in[t] = t < n ? (p.in_next ? Num<T>::to_f(static_cast<const T*>(p.in_next)[t]) : 1.0f) : 0.f;
    out[t] = t < n && p.out ? Num<T>::to_f(static_cast<const T*>(p.out)[t]) : 0.f;
  }
  for (int i = threadIdx.x; i < SM * SM; i += THREADS) {
    const int s = i / SM, t = i % SM;
    mix[s][t] = p.mix && s < n && t < n ? Num<T>::to_f(static_cast<const T*>(p.mix)[s * n + t]) : 0.f;
  }
  float w[NV][kVec];  // constant of the model: fetched while the preceding kernel drains
  const T* weight = static_cast<const T*>(p.weight);
#pragma unroll
  for (int i = 0; i < NV; ++i)
    if (threadIdx.x + i * THREADS < nvec) load_t<T>(weight + (threadIdx.x + i * THREADS) * kVec, w[i]);
  pdl_launch_dependents();
  pdl_wait();
  __syncthreads();
  int64_t src = 0;
  if (p.table) {
    src = p.idx32 ? p.idx32[row] : p.idx64[row];
    src = src < 0 ? 0 : (src >= p.vocab ? p.vocab - 1 : src);
  }
  const float* x = p.x + row * n * dim;
  float* xo = p.x_out + row * n * dim;
  float u[NV][kVec], ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int v = threadIdx.x + i * THREADS;
    if (v >= nvec) continue;
    const int64_t e0 = static_cast<int64_t>(v) * kVec;
#pragma unroll
    for (int e = 0; e < kVec; ++e) u[i][e] = 0.f;
    if (p.table) {
      float f[kVec];
      load_t<T>(static_cast<const T*>(p.table) + src * dim + e0, f);
#pragma unroll
      for (int e = 0; e < kVec; ++e) f[e] *= p.scale;
#pragma unroll
      for (int t = 0; t < SM; ++t) {
        if (t >= n) break;
        if (p.x_out) store_f(xo + static_cast<int64_t>(t) * dim + e0, f);
#pragma unroll
        for (int e = 0; e < kVec; ++e) u[i][e] = fmaf(in[t], f[e], u[i][e]);
      }
    } else {
      float y[kVec], old[SM][kVec];
#pragma unroll
      for (int s = 0; s < SM; ++s)
        if (s < n) load_f(x + static_cast<int64_t>(s) * dim + e0, old[s]);
      load_t<T>(static_cast<const T*>(p.y) + row * dim + e0, y);
#pragma unroll
      for (int t = 0; t < SM; ++t) {
        if (t >= n) break;
        float f[kVec];
#pragma unroll
        for (int e = 0; e < kVec; ++e) f[e] = out[t] * y[e];
#pragma unroll
        for (int s = 0; s < SM; ++s)
          if (s < n)
#pragma unroll
            for (int e = 0; e < kVec; ++e) f[e] = fmaf(mix[s][t], old[s][e], f[e]);
        if (p.x_out) store_f(xo + static_cast<int64_t>(t) * dim + e0, f);
#pragma unroll
        for (int e = 0; e < kVec; ++e) u[i][e] = fmaf(in[t], f[e], u[i][e]);
      }
    }
#pragma unroll
    for (int e = 0; e < kVec; ++e) ss += u[i][e] * u[i][e];
  }
  const float inv = 1.0f / sqrtf(block_sum(ss, part) / static_cast<float>(dim) + p.eps);
  T* dst = static_cast<T*>(p.normed) + row * dim;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int v = threadIdx.x + i * THREADS;
    if (v >= nvec) continue;
    float f[kVec];
#pragma unroll
    for (int e = 0; e < kVec; ++e) f[e] = u[i][e] * inv * w[i][e];
    store_t<T>(dst + static_cast<int64_t>(v) * kVec, f);
  }
}

template <typename T, int SM, int NV, int THREADS>
int launch(const StreamParams& p, int64_t rows, cudaStream_t st) {
  LRI_CUDA(launch_pdl(join_streams_kernel<T, SM, NV, THREADS>, dim3(static_cast<unsigned>(rows)), dim3(THREADS), 0, st, p));
  LRI_LAUNCH_CHECK("join_streams_kernel");
  return LRI_OK;
}

// Any number of streams and any width: one element at a time, u in shared memory.
constexpr int kMaxDim = 16384, kMaxStreams = 16;
template <typename T>
__global__ void __launch_bounds__(256) join_streams_generic_kernel(const StreamParams p) {
  extern __shared__ float su[];  // [dim]
  __shared__ float part[33];
  const int n = p.streams, dim = p.dim;
  const int64_t row = blockIdx.x;
  pdl_launch_dependents();
  pdl_wait();
  int64_t src = 0;
  if (p.table) {
    src = p.idx32 ? p.idx32[row] : p.idx64[row];
    src = src < 0 ? 0 : (src >= p.vocab ? p.vocab - 1 : src);
  }
  const T* mix = static_cast<const T*>(p.mix);
  float ss = 0.f;
  for (int e = threadIdx.x; e < dim; e += 256) {
    float old[kMaxStreams], u = 0.f;
    if (p.table) {
      old[0] = Num<T>::to_f(static_cast<const T*>(p.table)[src * dim + e]) * p.scale;
    } else {
      for (int s = 0; s < n; ++s) old[s] = p.x[(row * n + s) * dim + e];
    }
    for (int t = 0; t < n; ++t) {
      float f = old[0];
      if (!p.table) {
        f = Num<T>::to_f(static_cast<const T*>(p.out)[t]) * Num<T>::to_f(static_cast<const T*>(p.y)[row * dim + e]);
        for (int s = 0; s < n; ++s) f = fmaf(Num<T>::to_f(mix[s * n + t]), old[s], f);
      }
      if (p.x_out) p.x_out[(row * n + t) * dim + e] = f;
      u = fmaf(p.in_next ? Num<T>::to_f(static_cast<const T*>(p.in_next)[t]) : 1.0f, f, u);
    }
    su[e] = u;
    ss += u * u;
  }
  const float inv = 1.0f / sqrtf(block_sum(ss, part) / static_cast<float>(dim) + p.eps);
  for (int e = threadIdx.x; e < dim; e += 256)
    static_cast<T*>(p.normed)[row * dim + e] = Num<T>::from_f(su[e] * inv * Num<T>::to_f(static_cast<const T*>(p.weight)[e]));
}

template <typename T>
int launch_generic(const StreamParams& p, int64_t rows, cudaStream_t st) {
  auto kern = join_streams_generic_kernel<T>;
  static std::atomic<unsigned long long> attr_set{0};
  LRI_ONCE_PER_DEVICE(attr_set, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxDim * 4));
  LRI_CUDA(launch_pdl(kern, dim3(static_cast<unsigned>(rows)), dim3(256), static_cast<size_t>(p.dim) * 4, st, p));
  LRI_LAUNCH_CHECK("join_streams_generic_kernel");
  return LRI_OK;
}

template <typename T, int SM>
int by_size(const StreamParams& p, int64_t rows, cudaStream_t st) {
  const int nvec = p.dim / 4;
  if (nvec <= 256) return launch<T, SM, 1, 256>(p, rows, st);
  if (nvec <= 512) return launch<T, SM, 1, 512>(p, rows, st);
  if (rows <= 16 && nvec <= 1024) return launch<T, SM, 1, 1024>(p, rows, st);  // few rows: one thread's latency chain
  if (nvec <= 1024) return launch<T, SM, 4, 256>(p, rows, st);
  return launch<T, SM, 8, 512>(p, rows, st);
}

template <typename T>
int by_streams(const StreamParams& p, int64_t rows, cudaStream_t st) {
  const bool vec = p.dim % 4 == 0 && p.streams <= 8 && aligned16(p.x) && aligned16(p.x_out) && aligned16(p.table) &&
                   aligned16(p.y) && aligned16(p.weight) && aligned16(p.normed);
  if (!vec) return launch_generic<T>(p, rows, st);
  if (p.streams <= 2) return by_size<T, 2>(p, rows, st);
  if (p.streams <= 4) return by_size<T, 4>(p, rows, st);
  return by_size<T, 8>(p, rows, st);
}

int run(const char* who, int dtype, const StreamParams& p, int64_t rows, cudaStream_t st) {
  LRI_REQUIRE(dtype >= LRI_BF16 && dtype <= LRI_FP32, LRI_ERR_UNSUPPORTED, "%s: dtype %d", who, dtype);
  LRI_REQUIRE(p.weight && p.normed, LRI_ERR_ARG, "%s: NULL pointer", who);
  LRI_REQUIRE(rows >= 0 && rows < (1ll << 31), LRI_ERR_ARG, "%s: rows=%lld", who, (long long)rows);
  LRI_REQUIRE(p.streams >= 1 && p.streams <= kMaxStreams, LRI_ERR_UNSUPPORTED, "%s: streams=%d outside 1..%d", who, p.streams,
              kMaxStreams);
  LRI_REQUIRE(p.dim > 0 && p.dim <= kMaxDim, LRI_ERR_UNSUPPORTED, "%s: dim=%d outside 1..%d", who, p.dim, kMaxDim);
  if (rows == 0) return LRI_OK;
  if (dtype == LRI_BF16) return by_streams<__nv_bfloat16>(p, rows, st);
  if (dtype == LRI_FP16) return by_streams<__half>(p, rows, st);
  return by_streams<float>(p, rows, st);
}

}  // namespace
}  // namespace lri

using namespace lri;

extern "C" int lri_join_streams(int dtype, const float* x, const void* y, const void* mix, const void* out, float* x_out,
                                const void* in_next, const void* weight, float eps, void* normed, int64_t rows, int streams,
                                int dim, lri_stream_t stream) {
  LRI_REQUIRE(x && y && mix && out, LRI_ERR_ARG, "join_streams: NULL pointer");
  StreamParams p{};
  p.x = x, p.y = y, p.mix = mix, p.out = out, p.x_out = x_out, p.in_next = in_next, p.weight = weight, p.eps = eps;
  p.normed = normed, p.streams = streams, p.dim = dim;
  return run("join_streams", dtype, p, rows, static_cast<cudaStream_t>(stream));
}

extern "C" int lri_embed_streams(int dtype, const void* table, const void* idx, int idx_is_i64, int64_t vocab, float scale,
                                 float* x_out, const void* in_next, const void* weight, float eps, void* normed, int64_t rows,
                                 int streams, int dim, lri_stream_t stream) {
  LRI_REQUIRE(table && idx && vocab > 0, LRI_ERR_ARG, "embed_streams: NULL pointer or vocab=%lld", (long long)vocab);
  StreamParams p{};
  p.table = table, p.vocab = vocab, p.scale = scale;
  if (idx_is_i64)
    p.idx64 = static_cast<const int64_t*>(idx);
  else
    p.idx32 = static_cast<const int32_t*>(idx);
  p.x_out = x_out, p.in_next = in_next, p.weight = weight, p.eps = eps, p.normed = normed, p.streams = streams, p.dim = dim;
  return run("embed_streams", dtype, p, rows, static_cast<cudaStream_t>(stream));
}
