// SIMT GEMM without constraints on shape, alignment or storage type: y[m, n] = sum_k x[m, k] W[n, k] (+ addend)
// with fp32 arithmetic and y in the storage type or in fp32.  It serves fp32 models (every product and sum a true
// 32-bit operation) and projections whose K is not a multiple of 8, which the 16-byte kernels do not take.
#include "linear.cuh"

namespace lri {
namespace {

constexpr int kTile = 64, kDepth = 16;

// 64 x 64 outputs per CTA, 256 threads, 4 x 4 outputs per thread
template <typename T, typename TO>
__global__ void __launch_bounds__(256)
gemm_generic_kernel(const T* __restrict__ x, const T* __restrict__ w, const T* __restrict__ addend, TO* __restrict__ y,
                    int64_t m, int n, int k) {
  __shared__ float xs[kDepth][kTile + 1];
  __shared__ float ws[kDepth][kTile + 1];
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const int64_t m0 = static_cast<int64_t>(blockIdx.y) * kTile, n0 = static_cast<int64_t>(blockIdx.x) * kTile;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < k; k0 += kDepth) {
    for (int i = threadIdx.x; i < kTile * kDepth; i += 256) {
      const int r = i / kDepth, kk = i % kDepth;
      const bool in_k = k0 + kk < k;
      xs[kk][r] = in_k && m0 + r < m ? Num<T>::to_f(x[(m0 + r) * k + k0 + kk]) : 0.f;
      ws[kk][r] = in_k && n0 + r < n ? Num<T>::to_f(w[(n0 + r) * k + k0 + kk]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < kDepth; ++kk) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) a[i] = xs[kk][ty * 4 + i], b[i] = ws[kk][tx * 4 + i];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int64_t r = m0 + ty * 4 + i, c = n0 + tx * 4 + j;
      if (r >= m || c >= n) continue;
      float v = acc[i][j];
      if (addend) v = rnd<T>(v) + Num<T>::to_f(addend[r * n + c]);
      y[r * n + c] = Num<TO>::from_f(v);
    }
}

// Few rows: one warp per output column, lanes over K.
template <typename T, typename TO, int M>
__global__ void __launch_bounds__(256)
gemv_generic_kernel(const T* __restrict__ x, const T* __restrict__ w, const T* __restrict__ addend, TO* __restrict__ y,
                    int m, int n, int k) {
  const int64_t c = static_cast<int64_t>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (c >= n) return;
  float acc[M] = {};
  for (int i = lane; i < k; i += 32) {
    const float wv = Num<T>::to_f(w[c * k + i]);
#pragma unroll
    for (int r = 0; r < M; ++r)
      if (r < m) acc[r] = fmaf(wv, Num<T>::to_f(x[static_cast<int64_t>(r) * k + i]), acc[r]);
  }
#pragma unroll
  for (int r = 0; r < M; ++r) {
    if (r >= m) break;
    float v = warp_sum(acc[r]);
    if (lane == 0) {
      if (addend) v = rnd<T>(v) + Num<T>::to_f(addend[static_cast<int64_t>(r) * n + c]);
      y[static_cast<int64_t>(r) * n + c] = Num<TO>::from_f(v);
    }
  }
}

template <typename T, typename TO>
int launch(const void* x, const void* w, const void* addend, void* y, int64_t m, int n, int k, cudaStream_t st) {
  const T* xt = static_cast<const T*>(x);
  const T* wt = static_cast<const T*>(w);
  const T* at = static_cast<const T*>(addend);
  TO* yt = static_cast<TO*>(y);
  if (m <= 8) {
    const unsigned grid = static_cast<unsigned>((n + 7) / 8);
    if (m == 1)
      gemv_generic_kernel<T, TO, 1><<<grid, 256, 0, st>>>(xt, wt, at, yt, 1, n, k);
    else
      gemv_generic_kernel<T, TO, 8><<<grid, 256, 0, st>>>(xt, wt, at, yt, static_cast<int>(m), n, k);
  } else {
    const int64_t tiles_m = (m + kTile - 1) / kTile;
    LRI_REQUIRE(tiles_m <= 65535, LRI_ERR_UNSUPPORTED, "linear: %lld rows", (long long)m);
    gemm_generic_kernel<T, TO><<<dim3((n + kTile - 1) / kTile, static_cast<unsigned>(tiles_m)), 256, 0, st>>>(xt, wt, at, yt, m, n, k);
  }
  LRI_LAUNCH_CHECK("gemm_generic_kernel");
  return LRI_OK;
}

template <typename T>
__global__ void __launch_bounds__(256) glu_rows_kernel(const float* ug, T* h, int64_t m, int n, GluParams glu) {
  const int64_t i = static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x;
  if (i >= m * n) return;
  const int64_t r = i / n, j = i - r * n;
  h[i] = Num<T>::from_f(clamped_glu(ug[r * 2 * n + n + j], ug[r * 2 * n + j], glu));
}

}  // namespace

int glu_rows_launch(int dtype, const float* ug, void* h, int64_t m, int n, const GluParams& glu, cudaStream_t st) {
  const unsigned grid = static_cast<unsigned>((m * n + 255) / 256);
  if (dtype == LRI_FP32)
    glu_rows_kernel<float><<<grid, 256, 0, st>>>(ug, static_cast<float*>(h), m, n, glu);
  else if (dtype == LRI_BF16)
    glu_rows_kernel<__nv_bfloat16><<<grid, 256, 0, st>>>(ug, static_cast<__nv_bfloat16*>(h), m, n, glu);
  else
    glu_rows_kernel<__half><<<grid, 256, 0, st>>>(ug, static_cast<__half*>(h), m, n, glu);
  LRI_LAUNCH_CHECK("glu_rows_kernel");
  return LRI_OK;
}

int gemm_generic_launch(int dtype, const void* x, const void* w, const void* addend, void* y, bool out_f32, int64_t m,
                        int n, int k, cudaStream_t st) {
  if (dtype == LRI_FP32) return launch<float, float>(x, w, addend, y, m, n, k, st);
  if (dtype == LRI_BF16)
    return out_f32 ? launch<__nv_bfloat16, float>(x, w, addend, y, m, n, k, st)
                   : launch<__nv_bfloat16, __nv_bfloat16>(x, w, addend, y, m, n, k, st);
  return out_f32 ? launch<__half, float>(x, w, addend, y, m, n, k, st)
                 : launch<__half, __half>(x, w, addend, y, m, n, k, st);
}

}  // namespace lri
