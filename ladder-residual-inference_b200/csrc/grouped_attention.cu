// Grouped-query attention on a cache of keys and values per key head, with the steps in front of it for designs that norm
// the whole query and key projections and rotate the first part of each head:
//
//   grouped_prepare    q, k <- RMSNorm over ALL heads of the projection, rotation by halves of the first rot_dims
//                      dimensions of a head, q stored for the call, k and v written to the cache
//   grouped_attention  softmax attention over the cache inside a window and / or a chunk of positions, with an optional
//                      sink: tcgen05 for prompt portions (latent_attention_tc.cu), thread-block clusters for single tokens
//                      (attention_cluster.cu), a plain kernel for any size and type (latent_attention.cu)
#include "latent_attention.cuh"

namespace lri {
namespace {

struct PrepareParams {
  const float* proj;  // [rows, ld]: q (H heads of d), k (G heads of d), v (G heads of dv) at the offsets
  int64_t ld, q_off, k_off, v_off;
  const void* q_norm;  // [H * d]
  const void* k_norm;  // [G * d]
  const float* sums;   // [rows, 2] sums of squares of q and k over all ranks, or NULL: taken here
  int q_width, k_width;  // elements those sums (and the means) run over
  float eps;
  const float* table;  // [table_rows, rot / 2, 2] cos, sin
  int64_t table_rows;
  const void* input_pos;
  int pos_is_i64;
  void* q;        // [rows, H, d]
  void* k_cache;  // [B, G, smax, d]
  void* v_cache;  // [B, G, smax, dv]
  int64_t smax;
  int S, H, G, d, dv, rot;
};

constexpr int kThreads = 256;

// n elements of a row, normed and rotated: store(head, first element, VEC values)
template <typename T, int VEC, typename Store>
__device__ __forceinline__ void norm_rotate(const float* x, const T* w, float inv, const float* cs, int heads, int d, int rot, Store store) {
  const int half = rot >> 1, per = d / VEC;
  const bool whole = VEC == 8 && half % 8 == 0;  // 8 elements lie in one half, or behind the rotated part
  for (int i = blockIdx.y * kThreads + threadIdx.x; i < heads * per; i += kThreads * gridDim.y) {
    const int h = i / per, e0 = (i - h * per) * VEC;
    const float* xh = x + h * d;
    const T* wh = w + h * d;
    float f[VEC];
    if constexpr (VEC == 8) {
      if (whole) {
        float a[8], wa[8];
        load8<float>(xh + e0, a);
        load8<T>(wh + e0, wa);
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] = a[j] * inv * wa[j];
        if (e0 < rot) {
          const bool lower = e0 < half;
          const int other = lower ? e0 + half : e0 - half;
          const float* c = cs + 2 * (lower ? e0 : other);
          float b[8], wb[8], t0[8], t1[8];
          load8<float>(xh + other, b);
          load8<T>(wh + other, wb);
          load8<float>(c, t0);
          load8<float>(c + 8, t1);
#pragma unroll
          for (int j = 0; j < 8; ++j) {
            const float co = j < 4 ? t0[2 * j] : t1[2 * j - 8], si = j < 4 ? t0[2 * j + 1] : t1[2 * j - 7];
            const float y = b[j] * inv * wb[j];
            f[j] = lower ? f[j] * co - y * si : f[j] * co + y * si;
          }
        }
        store(h, e0, f);
        continue;
      }
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      const int e = e0 + j;
      const float a = xh[e] * inv * Num<T>::to_f(wh[e]);
      if (e < rot) {
        const int pair = e < half ? e : e - half, other = e < half ? e + half : e - half;
        const float b = xh[other] * inv * Num<T>::to_f(wh[other]);
        const float c = cs[2 * pair], s = cs[2 * pair + 1];
        f[j] = e < half ? a * c - b * s : a * c + b * s;
      } else {
        f[j] = a;
      }
    }
    store(h, e0, f);
  }
}
template <typename T, int VEC>
__device__ __forceinline__ void put(T* dst, const float (&f)[VEC]) {
  if constexpr (VEC == 8)
    store8<T>(dst, f);
  else
    dst[0] = Num<T>::from_f(f[0]);
}

// Grid (rows, slices): q and k of the row are staged in shared memory, since a norm needs all of them and a rotation both
// halves; with few rows several CTAs stage the same row and store a share of it each.
template <typename T, int VEC>
__global__ void __launch_bounds__(kThreads) grouped_prepare_kernel(const PrepareParams p) {
  extern __shared__ __align__(16) float gp_smem[];
  __shared__ float part[33];
  const int nq = p.H * p.d, nk = p.G * p.d, nv = p.G * p.dv;
  float* q = gp_smem;
  float* k = gp_smem + nq;
  pdl_launch_dependents();
  pdl_wait();
  const int64_t row = blockIdx.x;
  const int64_t b = row / p.S, s = row - b * p.S;
  const int64_t pos = load_pos(p.input_pos, p.pos_is_i64, s);
  if (pos < 0 || pos >= p.smax || pos >= p.table_rows) return;
  const float* pr = p.proj + row * p.ld;
  float sq = 0.f, sk = 0.f;
  if constexpr (VEC == 8) {
    for (int i = threadIdx.x * 4; i < nq; i += kThreads * 4) {
      const float4 v = *reinterpret_cast<const float4*>(pr + p.q_off + i);
      *reinterpret_cast<float4*>(q + i) = v;
      sq += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    for (int i = threadIdx.x * 4; i < nk; i += kThreads * 4) {
      const float4 v = *reinterpret_cast<const float4*>(pr + p.k_off + i);
      *reinterpret_cast<float4*>(k + i) = v;
      sk += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
  } else {
    for (int i = threadIdx.x; i < nq; i += kThreads) {
      q[i] = pr[p.q_off + i];
      sq += q[i] * q[i];
    }
    for (int i = threadIdx.x; i < nk; i += kThreads) {
      k[i] = pr[p.k_off + i];
      sk += k[i] * k[i];
    }
  }
  if (p.sums) {
    sq = p.sums[2 * row], sk = p.sums[2 * row + 1];
    __syncthreads();
  } else {
    sq = block_sum(sq, part);
    sk = block_sum(sk, part);
  }
  const float* cs = p.table + pos * (p.rot >> 1) * 2;
  T* qo = static_cast<T*>(p.q) + row * nq;
  T* kc = static_cast<T*>(p.k_cache) + (b * p.G * p.smax + pos) * p.d;
  T* vc = static_cast<T*>(p.v_cache) + (b * p.G * p.smax + pos) * p.dv;
  norm_rotate<T, VEC>(q, static_cast<const T*>(p.q_norm), 1.0f / sqrtf(sq / static_cast<float>(p.q_width) + p.eps), cs, p.H, p.d, p.rot,
                      [&](int h, int e, const float(&f)[VEC]) { put<T, VEC>(qo + h * p.d + e, f); });
  norm_rotate<T, VEC>(k, static_cast<const T*>(p.k_norm), 1.0f / sqrtf(sk / static_cast<float>(p.k_width) + p.eps), cs, p.G, p.d, p.rot,
                      [&](int h, int e, const float(&f)[VEC]) { put<T, VEC>(kc + h * p.smax * p.d + e, f); });
  for (int i = (blockIdx.y * kThreads + threadIdx.x) * VEC; i < nv; i += kThreads * VEC * gridDim.y) {
    const int h = i / p.dv, e = i - h * p.dv;
    float f[VEC];
    if constexpr (VEC == 8)
      load8<float>(pr + p.v_off + i, f);
    else
      f[0] = pr[p.v_off + i];
    put<T, VEC>(vc + h * p.smax * p.dv + e, f);
  }
}

// sums[row] = (sum of squares of n1 elements at off1, of n2 elements at off2)
__global__ void __launch_bounds__(kThreads)
row_squares_kernel(const float* x, int64_t ld, int64_t off1, int n1, int64_t off2, int n2, float* sums) {
  __shared__ float part[33];
  pdl_launch_dependents();
  pdl_wait();
  const float* r = x + blockIdx.x * ld;
  float a = 0.f, b = 0.f;
  for (int i = threadIdx.x; i < n1; i += kThreads) a += r[off1 + i] * r[off1 + i];
  for (int i = threadIdx.x; i < n2; i += kThreads) b += r[off2 + i] * r[off2 + i];
  a = block_sum(a, part);
  b = block_sum(b, part);
  if (threadIdx.x == 0) sums[2 * static_cast<int64_t>(blockIdx.x)] = a, sums[2 * static_cast<int64_t>(blockIdx.x) + 1] = b;
}

constexpr int kMaxStaged = 224 * 1024 / 4;  // elements of q and k of a row

template <typename T>
int prepare(const PrepareParams& p, int64_t rows, bool vec, cudaStream_t st) {
  const size_t smem = static_cast<size_t>(p.H + p.G) * p.d * sizeof(float);
  auto kern = vec ? grouped_prepare_kernel<T, 8> : grouped_prepare_kernel<T, 1>;
  static std::atomic<unsigned long long> set8{0}, set1{0};
  if (vec)
    LRI_ONCE_PER_DEVICE(set8, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxStaged * 4));
  else
    LRI_ONCE_PER_DEVICE(set1, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxStaged * 4));
  const int items = p.H * p.d / (vec ? 8 : 1);
  const unsigned slices = rows > 64 ? 1 : (items + kThreads - 1) / kThreads;
  LRI_CUDA(launch_pdl(kern, dim3(static_cast<unsigned>(rows), slices < 8 ? slices : 8), dim3(kThreads), smem, st, p));
  LRI_LAUNCH_CHECK("grouped_prepare_kernel");
  return LRI_OK;
}

}  // namespace
}  // namespace lri

using namespace lri;

extern "C" int lri_row_squares(const float* x, int64_t ld, int64_t off1, int n1, int64_t off2, int n2, float* sums, int64_t rows,
                               lri_stream_t stream) {
  LRI_REQUIRE(x && sums, LRI_ERR_ARG, "row_squares: NULL pointer");
  LRI_REQUIRE(rows >= 0 && rows < (1ll << 31) && n1 >= 0 && n2 >= 0, LRI_ERR_ARG, "row_squares: rows=%lld", (long long)rows);
  if (rows == 0) return LRI_OK;
  LRI_CUDA(launch_pdl(row_squares_kernel, dim3(static_cast<unsigned>(rows)), dim3(kThreads), 0, static_cast<cudaStream_t>(stream), x, ld,
                      off1, n1, off2, n2, sums));
  LRI_LAUNCH_CHECK("row_squares_kernel");
  return LRI_OK;
}

extern "C" int lri_grouped_prepare(int dtype, const float* proj, int64_t ld, int64_t q_off, int64_t k_off, int64_t v_off,
                                   const void* q_norm, const void* k_norm, const float* sums, int q_width, int k_width, float eps,
                                   const float* rope_table, int64_t table_rows, int rot_dims, const void* input_pos,
                                   int pos_is_i64, void* q, void* k_cache, void* v_cache, int64_t smax, int B, int S, int n_head,
                                   int n_kv, int dim, int vdim, lri_stream_t stream) {
  LRI_REQUIRE(dtype >= LRI_BF16 && dtype <= LRI_FP32, LRI_ERR_UNSUPPORTED, "grouped_prepare: dtype %d", dtype);
  LRI_REQUIRE(proj && q_norm && k_norm && rope_table && input_pos && q && k_cache && v_cache, LRI_ERR_ARG,
              "grouped_prepare: NULL pointer");
  LRI_REQUIRE(B >= 0 && S >= 0 && n_head > 0 && n_kv > 0 && dim > 0 && vdim > 0 && smax > 0 && table_rows > 0 && q_width > 0 && k_width > 0,
              LRI_ERR_ARG, "grouped_prepare: B=%d S=%d n_head=%d n_kv=%d dim=%d vdim=%d", B, S, n_head, n_kv, dim, vdim);
  LRI_REQUIRE(rot_dims >= 0 && rot_dims % 2 == 0 && rot_dims <= dim, LRI_ERR_ARG, "grouped_prepare: rot_dims=%d of dim=%d", rot_dims, dim);
  LRI_REQUIRE(static_cast<int64_t>(n_head + n_kv) * dim <= kMaxStaged, LRI_ERR_UNSUPPORTED, "grouped_prepare: %d heads of %d",
              n_head + n_kv, dim);
  const int64_t rows = static_cast<int64_t>(B) * S;
  if (rows == 0) return LRI_OK;
  PrepareParams p{};
  p.proj = proj, p.ld = ld, p.q_off = q_off, p.k_off = k_off, p.v_off = v_off, p.q_norm = q_norm, p.k_norm = k_norm, p.sums = sums;
  p.q_width = q_width, p.k_width = k_width, p.eps = eps, p.table = rope_table, p.table_rows = table_rows;
  p.input_pos = input_pos, p.pos_is_i64 = pos_is_i64, p.q = q, p.k_cache = k_cache, p.v_cache = v_cache, p.smax = smax;
  p.S = S, p.H = n_head, p.G = n_kv, p.d = dim, p.dv = vdim, p.rot = rot_dims;
  const bool vec = dim % 8 == 0 && vdim % 8 == 0 && ld % 4 == 0 && q_off % 4 == 0 && k_off % 4 == 0 && v_off % 4 == 0 &&
                   aligned16(proj) && aligned16(q) && aligned16(k_cache) && aligned16(v_cache) && aligned16(q_norm) && aligned16(k_norm) &&
                   aligned16(rope_table);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (dtype == LRI_BF16) return prepare<__nv_bfloat16>(p, rows, vec, st);
  if (dtype == LRI_FP16) return prepare<__half>(p, rows, vec, st);
  return prepare<float>(p, rows, vec, st);
}

extern "C" int lri_grouped_attention(int dtype, const void* q, const void* k_cache, const void* v_cache, const void* sink,
                                     void* out, int64_t out_ld, float out_scale, const void* input_pos, int pos_is_i64,
                                     int64_t smax, int64_t window, int64_t chunk, float scale, int B, int S, int n_head, int n_kv,
                                     int dim, int vdim, lri_stream_t stream) {
  LRI_REQUIRE(dtype >= LRI_BF16 && dtype <= LRI_FP32, LRI_ERR_UNSUPPORTED, "grouped_attention: dtype %d", dtype);
  LRI_REQUIRE(q && k_cache && v_cache && out && input_pos, LRI_ERR_ARG, "grouped_attention: NULL pointer");
  LRI_REQUIRE(B >= 0 && S >= 0 && n_head > 0 && n_kv > 0 && n_head % n_kv == 0 && dim > 0 && vdim > 0 && smax > 0, LRI_ERR_ARG,
              "grouped_attention: B=%d S=%d n_head=%d n_kv=%d dim=%d vdim=%d", B, S, n_head, n_kv, dim, vdim);
  LRI_REQUIRE(window >= 0 && chunk >= 0, LRI_ERR_ARG, "grouped_attention: window=%lld chunk=%lld", (long long)window, (long long)chunk);
  LRI_REQUIRE(vdim <= 1024 && dim <= 2048, LRI_ERR_UNSUPPORTED, "grouped_attention: dim=%d vdim=%d", dim, vdim);
  const int64_t rows = static_cast<int64_t>(B) * S;
  if (rows == 0) return LRI_OK;
  WindowParams p{};
  p.q = q, p.q_row = static_cast<int64_t>(n_head) * dim, p.q_head = dim;
  p.k = k_cache, p.k_batch = n_kv * smax * dim, p.k_row = dim, p.k_head = smax * dim;
  p.k2 = k_cache;  // no second part
  p.v = v_cache, p.v_batch = n_kv * smax * vdim, p.v_row = vdim, p.v_head = smax * vdim;
  p.group = n_head / n_kv, p.out = out, p.out_ld = out_ld, p.out_scale = out_scale, p.input_pos = input_pos, p.pos_is_i64 = pos_is_i64;
  p.history = -1, p.k_rows = smax, p.window = window > 0 ? window : (1ll << 40), p.chunk = chunk, p.sink = sink;
  p.scale = scale, p.S = S, p.H = n_head, p.d1 = dim, p.d2 = 0, p.dv = vdim;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (option(OPT_WINDOW_TC)) {
    if (attn_decode_masked_supports(dtype, p)) return attn_decode_masked_launch(dtype, p, B, st);
    if (window_attention_tc_supports(dtype, p, B)) return window_attention_tc_launch(dtype, p, B, st);
  }
  return window_attention_plain_launch(dtype, p, rows, st);
}
