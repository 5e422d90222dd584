// Latent attention: the keys and values of all heads are linear images of one normed latent per token (plus a rotated
// key part shared by the heads), and only latent and rotated part are cached: one row [latent (r) | rotated key (dr)] per
// token.
//
//   latent_prepare   from the fp32 projections of a token: rotation of q's rotated part and of the shared key part,
//                    RMSNorm of the latent, cache write
//   latent_window    the cache rows a call can see, copied to contiguous latents and rotated keys (prompt form: they
//                    are expanded to per-head keys and values by one projection)
//   head_linear      per-head matrices: q^T W_uk (the query in latent coordinates) and W_uv o (single-token form: scores
//                    and sums run on the cached latents themselves)
//   window_attention softmax attention over a sliding window for either form: tcgen05 for prompt portions
//                    (latent_attention_tc.cu), mma.sync for single tokens (latent_decode.cu), and here the plain kernel
//                    for any size and type
#include "latent_attention.cuh"
#include "linear.cuh"

namespace lri {

namespace {

// ---- rotation, norm, cache write ---------------------------------------------------------------------
struct PrepareParams {
  const float* proj;  // [rows, ld]: q at q_off (H heads of [dn | dr]), latent and key part at kv_off
  int64_t ld, q_off, kv_off;
  const void* norm_w;  // [r]
  float eps;
  const float* table;  // [table_rows, dr / 2, 2] cos, sin
  int64_t table_rows;
  const void* input_pos;
  int pos_is_i64;
  void* qn;  // unrotated part, q_n + row * qn_row + head * qn_head
  int64_t qn_row, qn_head;
  void* qr;  // rotated part
  int64_t qr_row, qr_head;
  void* cache;  // [B, smax, r + dr]
  int64_t smax;
  int S, H, dn, dr, r;
  int heads_per_cta;
  int vec;  // 8-element accesses of q are aligned
};

// Grid (rows, 1 + head groups): slice 0 writes the cache row, the others some heads of q each.
template <typename T>
__global__ void __launch_bounds__(256) latent_prepare_kernel(const PrepareParams p) {
  __shared__ float part[33];
  pdl_launch_dependents();
  pdl_wait();
  const int64_t row = blockIdx.x;
  const int64_t b = row / p.S, s = row - b * p.S;
  const int64_t pos = load_pos(p.input_pos, p.pos_is_i64, s);
  if (pos < 0 || pos >= p.smax || pos >= p.table_rows) return;
  const int half = p.dr >> 1;
  const float* cs = p.table + pos * half * 2;
  const float* pr = p.proj + row * p.ld;
  if (blockIdx.y == 0) {
    const float* kv = pr + p.kv_off;
    float ss = 0.f;
    for (int i = threadIdx.x; i < p.r; i += 256) ss += kv[i] * kv[i];
    const float inv = 1.0f / sqrtf(block_sum(ss, part) / static_cast<float>(p.r) + p.eps);
    const T* w = static_cast<const T*>(p.norm_w);
    T* dst = static_cast<T*>(p.cache) + (b * p.smax + pos) * (p.r + p.dr);
    for (int i = threadIdx.x; i < p.r; i += 256) dst[i] = Num<T>::from_f(kv[i] * inv * Num<T>::to_f(w[i]));
    for (int i = threadIdx.x; i < half; i += 256) {
      const float u = kv[p.r + i], v = kv[p.r + half + i], c = cs[2 * i], sn = cs[2 * i + 1];
      dst[p.r + i] = Num<T>::from_f(u * c - v * sn);
      dst[p.r + half + i] = Num<T>::from_f(v * c + u * sn);
    }
    return;
  }
  const int h0 = (blockIdx.y - 1) * p.heads_per_cta, h1 = min(h0 + p.heads_per_cta, p.H);
  if (p.vec) {
    // items of 8 unrotated elements, then of 4 rotated pairs
    const int plain = p.dn >> 3, per_head = plain + (half >> 2);
    for (int i = threadIdx.x; i < (h1 - h0) * per_head; i += 256) {
      const int h = h0 + i / per_head, u = i % per_head;
      const float* q = pr + p.q_off + static_cast<int64_t>(h) * (p.dn + p.dr);
      if (u < plain) {
        float f[8];
        load8<float>(q + u * 8, f);
        store8<T>(static_cast<T*>(p.qn) + row * p.qn_row + h * p.qn_head + u * 8, f);
        continue;
      }
      const int e = (u - plain) * 4;
      T* qr = static_cast<T*>(p.qr) + row * p.qr_row + h * p.qr_head;
      const float4 x = *reinterpret_cast<const float4*>(q + p.dn + e), y = *reinterpret_cast<const float4*>(q + p.dn + half + e);
      const float4 t0 = *reinterpret_cast<const float4*>(cs + 2 * e), t1 = *reinterpret_cast<const float4*>(cs + 2 * e + 4);
      const float a[4] = {x.x, x.y, x.z, x.w}, b2[4] = {y.x, y.y, y.z, y.w};
      const float c[4] = {t0.x, t0.z, t1.x, t1.z}, sn[4] = {t0.y, t0.w, t1.y, t1.w};
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        qr[e + j] = Num<T>::from_f(a[j] * c[j] - b2[j] * sn[j]);
        qr[half + e + j] = Num<T>::from_f(b2[j] * c[j] + a[j] * sn[j]);
      }
    }
    return;
  }
  for (int h = h0 + (threadIdx.x >> 5); h < h1; h += 8) {
    const int lane = threadIdx.x & 31;
    const float* q = pr + p.q_off + static_cast<int64_t>(h) * (p.dn + p.dr);
    T* qn = static_cast<T*>(p.qn) + row * p.qn_row + h * p.qn_head;
    T* qr = static_cast<T*>(p.qr) + row * p.qr_row + h * p.qr_head;
    for (int i = lane; i < p.dn; i += 32) qn[i] = Num<T>::from_f(q[i]);
    for (int i = lane; i < half; i += 32) {
      const float u = q[p.dn + i], v = q[p.dn + half + i], c = cs[2 * i], sn = cs[2 * i + 1];
      qr[i] = Num<T>::from_f(u * c - v * sn);
      qr[half + i] = Num<T>::from_f(v * c + u * sn);
    }
  }
}

// ---- cache rows of a call, contiguous -----------------------------------------------------------------
// Row j of sequence b holds position pos0 - history + j; rows before position 0 are zero.
template <typename T>
__global__ void __launch_bounds__(128)
latent_window_kernel(const T* cache, int64_t smax, int r, int dr, const void* input_pos, int pos_is_i64, int history,
                     int rows, T* lat, T* k_rot) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t j = blockIdx.x, b = blockIdx.y;
  const int64_t pos = load_pos(input_pos, pos_is_i64, 0) - history + j;
  const bool ok = pos >= 0 && pos < smax;
  const T* src = cache + (b * smax + (ok ? pos : 0)) * (r + dr);
  T* ld = lat + (b * rows + j) * r;
  T* kd = k_rot + (b * rows + j) * dr;
  if (sizeof(T) == 2 && r % 8 == 0 && dr % 8 == 0) {
    const uint4 zero = make_uint4(0, 0, 0, 0);
    for (int i = threadIdx.x; i < r / 8; i += 128)
      reinterpret_cast<uint4*>(ld)[i] = ok ? reinterpret_cast<const uint4*>(src)[i] : zero;
    for (int i = threadIdx.x; i < dr / 8; i += 128)
      reinterpret_cast<uint4*>(kd)[i] = ok ? reinterpret_cast<const uint4*>(src + r)[i] : zero;
    return;
  }
  for (int i = threadIdx.x; i < r; i += 128) ld[i] = ok ? src[i] : Num<T>::from_f(0.f);
  for (int i = threadIdx.x; i < dr; i += 128) kd[i] = ok ? src[r + i] : Num<T>::from_f(0.f);
}

// ---- per-head matrices -----------------------------------------------------------------------------------
struct HeadLinearParams {
  const void* x;  // x + row * x_row + head * x_head, `in` elements
  int64_t x_row, x_head;
  const void* w;  // [H, out, in] or, transposed, [H, in, out]
  void* y;        // y + row * y_row + head * y_head, `out` elements
  int64_t y_row, y_head;
  int rows, in, out;
};

// transposed, any shape: one thread per output
template <typename T>
__global__ void __launch_bounds__(128) head_linear_t_generic_kernel(const HeadLinearParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int j = blockIdx.x * 128 + threadIdx.x, h = blockIdx.y;
  const int64_t row = blockIdx.z;
  if (j >= p.out) return;
  const T* x = static_cast<const T*>(p.x) + row * p.x_row + h * p.x_head;
  const T* w = static_cast<const T*>(p.w) + static_cast<int64_t>(h) * p.in * p.out + j;
  float acc = 0.f;
  for (int i = 0; i < p.in; ++i) acc = fmaf(Num<T>::to_f(x[i]), Num<T>::to_f(w[static_cast<int64_t>(i) * p.out]), acc);
  (static_cast<T*>(p.y) + row * p.y_row + h * p.y_head)[j] = Num<T>::from_f(acc);
}
// rows of W contiguous, any shape: one warp per output
template <typename T>
__global__ void __launch_bounds__(256) head_linear_generic_kernel(const HeadLinearParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int j = blockIdx.x * 8 + (threadIdx.x >> 5), h = blockIdx.y, lane = threadIdx.x & 31;
  const int64_t row = blockIdx.z;
  if (j >= p.out) return;
  const T* x = static_cast<const T*>(p.x) + row * p.x_row + h * p.x_head;
  const T* w = static_cast<const T*>(p.w) + (static_cast<int64_t>(h) * p.out + j) * p.in;
  float acc = 0.f;
  for (int i = lane; i < p.in; i += 32) acc = fmaf(Num<T>::to_f(x[i]), Num<T>::to_f(w[i]), acc);
  acc = warp_sum(acc);
  if (lane == 0) (static_cast<T*>(p.y) + row * p.y_row + h * p.y_head)[j] = Num<T>::from_f(acc);
}

// transposed, 16-byte loads: a CTA owns 64 outputs of a head; 8 threads cover them with 8 outputs each, the 32 thread groups
// take the inputs i = group, group + 32, ...; M rows share the weights.  The weights of the first four inputs of a thread are requested
// before the wait for the preceding kernel.
template <typename T, int M>
__global__ void __launch_bounds__(256) head_linear_t_kernel(const HeadLinearParams p) {
  __shared__ float red[8][M][64];
  const int h = blockIdx.y, cg = threadIdx.x & 7, ig = threadIdx.x >> 3;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int j0 = blockIdx.x * 64 + cg * 8;
  const int64_t row0 = static_cast<int64_t>(blockIdx.z) * M;
  const T* w = static_cast<const T*>(p.w) + static_cast<int64_t>(h) * p.in * p.out + j0;
  const bool live = j0 < p.out;
  uint4 wv[4];
  auto load_w = [&](int i0) {
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const int i = i0 + ig + 32 * u;
      wv[u] = live && i < p.in ? ld_stream16(w + static_cast<int64_t>(i) * p.out) : make_uint4(0, 0, 0, 0);
    }
  };
  load_w(0);
  pdl_launch_dependents();
  pdl_wait();
  const T* x = static_cast<const T*>(p.x) + row0 * p.x_row + h * p.x_head;
  float acc[M][8] = {};
  for (int i0 = 0; i0 < p.in; i0 += 128) {
    if (i0 > 0) load_w(i0);
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const int i = i0 + ig + 32 * u;
      if (i >= p.in) break;
      float f[8];
      unpack8<T>(wv[u], f);
#pragma unroll
      for (int m = 0; m < M; ++m) {
        const float xv = row0 + m < p.rows ? Num<T>::to_f(x[m * p.x_row + i]) : 0.f;
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[m][e] = fmaf(f[e], xv, acc[m][e]);
      }
    }
  }
#pragma unroll
  for (int m = 0; m < M; ++m)
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      float v = acc[m][e];
      v += __shfl_xor_sync(0xffffffffu, v, 8);
      v += __shfl_xor_sync(0xffffffffu, v, 16);
      if (lane < 8) red[warp][m][cg * 8 + e] = v;
    }
  __syncthreads();
  for (int i = threadIdx.x; i < M * 64; i += 256) {
    const int m = i >> 6, c = i & 63;
    if (row0 + m >= p.rows || blockIdx.x * 64 + c >= p.out) continue;
    float v = 0.f;
#pragma unroll
    for (int wi = 0; wi < 8; ++wi) v += red[wi][m][c];
    (static_cast<T*>(p.y) + (row0 + m) * p.y_row + h * p.y_head)[blockIdx.x * 64 + c] = Num<T>::from_f(v);
  }
}

// rows of W contiguous, 16-byte loads: a warp owns 4 outputs of a head, its lanes 8 inputs each per step
template <typename T, int M>
__global__ void __launch_bounds__(256) head_linear_kernel(const HeadLinearParams p) {
  const int h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int j0 = blockIdx.x * 32 + warp * 4;
  const int64_t row0 = static_cast<int64_t>(blockIdx.z) * M;
  const T* w = static_cast<const T*>(p.w) + static_cast<int64_t>(h) * p.out * p.in;
  uint4 wv[2][4];
  auto load_w = [&](int i0) {
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int i = i0 + u * 256 + lane * 8;
#pragma unroll
      for (int r = 0; r < 4; ++r)
        wv[u][r] = j0 + r < p.out && i < p.in ? ld_stream16(w + static_cast<int64_t>(j0 + r) * p.in + i) : make_uint4(0, 0, 0, 0);
    }
  };
  load_w(0);
  pdl_launch_dependents();
  pdl_wait();
  const T* x = static_cast<const T*>(p.x) + row0 * p.x_row + h * p.x_head;
  float acc[M][4] = {};
  for (int i0 = 0; i0 < p.in; i0 += 512) {
    if (i0 > 0) load_w(i0);
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int i = i0 + u * 256 + lane * 8;
      if (i >= p.in) break;
      float xf[M][8];
#pragma unroll
      for (int m = 0; m < M; ++m) load8<T>(x + (row0 + m < p.rows ? m : 0) * p.x_row + i, xf[m]);
#pragma unroll
      for (int r = 0; r < 4; ++r) {
        float f[8];
        unpack8<T>(wv[u][r], f);
#pragma unroll
        for (int m = 0; m < M; ++m)
#pragma unroll
          for (int e = 0; e < 8; ++e) acc[m][r] = fmaf(f[e], xf[m][e], acc[m][r]);
      }
    }
  }
#pragma unroll
  for (int m = 0; m < M; ++m)
#pragma unroll
    for (int r = 0; r < 4; ++r) {
      const float v = warp_sum(acc[m][r]);
      if (lane == 0 && row0 + m < p.rows && j0 + r < p.out)
        (static_cast<T*>(p.y) + (row0 + m) * p.y_row + h * p.y_head)[j0 + r] = Num<T>::from_f(v);
    }
}

template <typename T, int M>
int launch_head_linear(const HeadLinearParams& p, int heads, bool transposed, cudaStream_t st) {
  const unsigned h = static_cast<unsigned>(heads), z = static_cast<unsigned>((p.rows + M - 1) / M);
  if (transposed)
    LRI_CUDA(launch_pdl(head_linear_t_kernel<T, M>, dim3((p.out + 63) / 64, h, z), dim3(256), 0, st, p));
  else
    LRI_CUDA(launch_pdl(head_linear_kernel<T, M>, dim3((p.out + 31) / 32, h, z), dim3(256), 0, st, p));
  LRI_LAUNCH_CHECK("head_linear_kernel");
  return LRI_OK;
}
template <typename T>
int head_linear(const HeadLinearParams& p, int heads, bool transposed, cudaStream_t st) {
  if (p.rows <= 1) return launch_head_linear<T, 1>(p, heads, transposed, st);
  if (p.rows <= 2) return launch_head_linear<T, 2>(p, heads, transposed, st);
  return launch_head_linear<T, 4>(p, heads, transposed, st);
}

// ---- attention over a sliding window, any size ---------------------------------------------------------------
// One warp per (token, head).  A lane scores one key at a time, then the warp adds the 32 keys' values, lanes over the
// value columns.
template <typename T, int NV>
__global__ void __launch_bounds__(128) window_attention_kernel(const WindowParams p, int64_t rows) {
  extern __shared__ float wa_smem[];
  pdl_launch_dependents();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int64_t item = static_cast<int64_t>(blockIdx.x) * 4 + warp;
  if (item >= rows * p.H) return;
  const int64_t row = item / p.H;
  const int h = static_cast<int>(item - row * p.H);
  const int64_t b = row / p.S, s = row - b * p.S;
  const int d = p.d1 + p.d2;
  float* q = wa_smem + warp * d;
  const T* qg = static_cast<const T*>(p.q) + row * p.q_row + h * p.q_head;
  for (int i = lane; i < d; i += 32) q[i] = Num<T>::to_f(qg[i]);
  __syncwarp();
  const int64_t qpos = load_pos(p.input_pos, p.pos_is_i64, s);
  const int64_t kpos0 = p.history < 0 ? 0 : load_pos(p.input_pos, p.pos_is_i64, 0) - p.history;
  const int64_t lo = first_visible(qpos, p.window, p.chunk);
  int64_t j0 = lo - kpos0, j1 = qpos - kpos0;  // visible key rows j0 .. j1
  j0 = j0 < 0 ? 0 : j0;
  j1 = j1 >= p.k_rows ? p.k_rows - 1 : j1;
  const T* k = static_cast<const T*>(p.k) + b * p.k_batch + (h / p.group) * p.k_head;
  const T* k2 = static_cast<const T*>(p.k2) + b * p.k2_batch;
  const T* v = static_cast<const T*>(p.v) + b * p.v_batch + (h / p.group) * p.v_head;
  float m = p.sink ? Num<T>::to_f(static_cast<const T*>(p.sink)[h]) : -INFINITY;
  float l = p.sink ? 1.f : 0.f, o[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) o[i] = 0.f;
  for (int64_t jb = j0; jb <= j1; jb += 32) {
    const int64_t j = jb + lane;
    float sc = -INFINITY;
    if (j <= j1) {
      const T* kj = k + j * p.k_row;
      const T* kj2 = k2 + j * p.k2_row;
      float acc = 0.f;
      for (int i = 0; i < p.d1; ++i) acc = fmaf(q[i], Num<T>::to_f(kj[i]), acc);
      for (int i = 0; i < p.d2; ++i) acc = fmaf(q[p.d1 + i], Num<T>::to_f(kj2[i]), acc);
      sc = acc * p.scale;
    }
    const float mn = fmaxf(m, warp_max(sc));
    const float corr = m == -INFINITY ? 0.f : expf(m - mn);
    const float pj = j <= j1 ? expf(sc - mn) : 0.f;
    l = l * corr + warp_sum(pj);
    m = mn;
#pragma unroll
    for (int i = 0; i < NV; ++i) o[i] *= corr;
    const int n = static_cast<int>(j1 - jb + 1 < 32 ? j1 - jb + 1 : 32);
    for (int jj = 0; jj < n; ++jj) {
      const float w = __shfl_sync(0xffffffffu, pj, jj);
      const T* vj = v + (jb + jj) * p.v_row;
#pragma unroll
      for (int i = 0; i < NV; ++i)
        if (lane + 32 * i < p.dv) o[i] = fmaf(w, Num<T>::to_f(vj[lane + 32 * i]), o[i]);
    }
  }
  const float inv = l > 0.f ? p.out_scale / l : 0.f;
  T* out = static_cast<T*>(p.out) + row * p.out_ld + static_cast<int64_t>(h) * p.dv;
#pragma unroll
  for (int i = 0; i < NV; ++i)
    if (lane + 32 * i < p.dv) out[lane + 32 * i] = Num<T>::from_f(o[i] * inv);
}

template <typename T, int NV>
int launch_window(const WindowParams& p, int64_t rows, cudaStream_t st) {
  const int64_t items = rows * p.H;
  const size_t smem = static_cast<size_t>(p.d1 + p.d2) * 4 * sizeof(float);
  LRI_CUDA(launch_pdl(window_attention_kernel<T, NV>, dim3(static_cast<unsigned>((items + 3) / 4)), dim3(128), smem, st, p, rows));
  LRI_LAUNCH_CHECK("window_attention_kernel");
  return LRI_OK;
}
template <typename T>
int window(const WindowParams& p, int64_t rows, cudaStream_t st) {
  const int nv = (p.dv + 31) / 32;
  if (nv <= 1) return launch_window<T, 1>(p, rows, st);
  if (nv <= 4) return launch_window<T, 4>(p, rows, st);
  if (nv <= 8) return launch_window<T, 8>(p, rows, st);
  if (nv <= 16) return launch_window<T, 16>(p, rows, st);
  return launch_window<T, 32>(p, rows, st);
}

bool dtype_ok(int dtype) { return dtype >= LRI_BF16 && dtype <= LRI_FP32; }

}  // namespace

int window_attention_plain_launch(int dtype, const WindowParams& p, int64_t rows, cudaStream_t st) {
  if (dtype == LRI_BF16) return window<__nv_bfloat16>(p, rows, st);
  if (dtype == LRI_FP16) return window<__half>(p, rows, st);
  return window<float>(p, rows, st);
}

}  // namespace lri

using namespace lri;

#define LRI_BY_TYPE(dtype, call)                                 \
  ((dtype) == LRI_BF16 ? call<__nv_bfloat16> : (dtype) == LRI_FP16 ? call<__half> : call<float>)

extern "C" int lri_latent_prepare(int dtype, const float* proj, int64_t ld, int64_t q_off, int64_t kv_off,
                                  const void* norm_weight, float eps, const float* rope_table, int64_t table_rows,
                                  const void* input_pos, int pos_is_i64, void* qn, int64_t qn_row, int64_t qn_head, void* qr,
                                  int64_t qr_row, int64_t qr_head, void* cache, int64_t smax, int B, int S, int heads, int dim,
                                  int rot_dim, int rank, lri_stream_t stream) {
  LRI_REQUIRE(dtype_ok(dtype), LRI_ERR_UNSUPPORTED, "latent_prepare: dtype %d", dtype);
  LRI_REQUIRE(proj && norm_weight && rope_table && input_pos && qn && qr && cache, LRI_ERR_ARG, "latent_prepare: NULL pointer");
  LRI_REQUIRE(B >= 0 && S >= 0 && heads > 0 && heads <= 8 * 65534 && dim > 0 && rot_dim > 0 && rot_dim % 2 == 0 && rank > 0 && smax > 0 &&
                  table_rows > 0,
              LRI_ERR_ARG, "latent_prepare: B=%d S=%d heads=%d dim=%d rot_dim=%d rank=%d", B, S, heads, dim, rot_dim, rank);
  const int64_t rows = static_cast<int64_t>(B) * S;
  if (rows == 0) return LRI_OK;
  PrepareParams p{};
  p.proj = proj, p.ld = ld, p.q_off = q_off, p.kv_off = kv_off, p.norm_w = norm_weight, p.eps = eps;
  p.table = rope_table, p.table_rows = table_rows, p.input_pos = input_pos, p.pos_is_i64 = pos_is_i64;
  p.qn = qn, p.qn_row = qn_row, p.qn_head = qn_head, p.qr = qr, p.qr_row = qr_row, p.qr_head = qr_head;
  p.cache = cache, p.smax = smax, p.S = S, p.H = heads, p.dn = dim, p.dr = rot_dim, p.r = rank;
  p.vec = dim % 8 == 0 && rot_dim % 8 == 0 && ld % 8 == 0 && q_off % 8 == 0 && qn_row % 8 == 0 && qn_head % 8 == 0 && aligned16(proj) &&
          aligned16(qn) && aligned16(rope_table);
  // many rows: one CTA takes the heads of a row (few rows: more CTAs, shorter chains)
  p.heads_per_cta = rows >= 256 ? (heads < 64 ? heads : 64) : 8;
  LRI_CUDA(launch_pdl(LRI_BY_TYPE(dtype, latent_prepare_kernel),
                      dim3(static_cast<unsigned>(rows), 1 + (heads + p.heads_per_cta - 1) / p.heads_per_cta), dim3(256), 0,
                      static_cast<cudaStream_t>(stream), p));
  LRI_LAUNCH_CHECK("latent_prepare_kernel");
  return LRI_OK;
}

extern "C" int lri_latent_window(int dtype, const void* cache, int64_t smax, int rank, int rot_dim, const void* input_pos,
                                 int pos_is_i64, int B, int history, int rows, void* latent_out, void* k_rot_out,
                                 lri_stream_t stream) {
  LRI_REQUIRE(dtype_ok(dtype), LRI_ERR_UNSUPPORTED, "latent_window: dtype %d", dtype);
  LRI_REQUIRE(cache && input_pos && latent_out && k_rot_out, LRI_ERR_ARG, "latent_window: NULL pointer");
  LRI_REQUIRE(B >= 0 && B <= 65535 && rows >= 0 && history >= 0 && rank > 0 && rot_dim > 0 && smax > 0, LRI_ERR_ARG,
              "latent_window: B=%d rows=%d history=%d", B, rows, history);
  if (B == 0 || rows == 0) return LRI_OK;
  const dim3 grid(static_cast<unsigned>(rows), static_cast<unsigned>(B));
  cudaStream_t st = static_cast<cudaStream_t>(stream);
#define LRI_CALL(T)                                                                                                       \
  LRI_CUDA(launch_pdl(latent_window_kernel<T>, grid, dim3(128), 0, st, static_cast<const T*>(cache), smax, rank, rot_dim, \
                      input_pos, pos_is_i64, history, rows, static_cast<T*>(latent_out), static_cast<T*>(k_rot_out)))
  if (dtype == LRI_BF16)
    LRI_CALL(__nv_bfloat16);
  else if (dtype == LRI_FP16)
    LRI_CALL(__half);
  else
    LRI_CALL(float);
#undef LRI_CALL
  LRI_LAUNCH_CHECK("latent_window_kernel");
  return LRI_OK;
}

extern "C" int lri_head_linear(int dtype, const void* x, int64_t x_row, int64_t x_head, const void* w, int transposed, void* y,
                               int64_t y_row, int64_t y_head, int64_t rows, int heads, int in, int out, lri_stream_t stream) {
  LRI_REQUIRE(dtype_ok(dtype), LRI_ERR_UNSUPPORTED, "head_linear: dtype %d", dtype);
  LRI_REQUIRE(x && w && y, LRI_ERR_ARG, "head_linear: NULL pointer");
  LRI_REQUIRE(rows >= 0 && rows <= 65535 && heads > 0 && heads <= 65535 && in > 0 && out > 0, LRI_ERR_ARG,
              "head_linear: rows=%lld heads=%d in=%d out=%d", (long long)rows, heads, in, out);
  if (rows == 0) return LRI_OK;
  HeadLinearParams p{};
  p.x = x, p.x_row = x_row, p.x_head = x_head, p.w = w, p.y = y, p.y_row = y_row, p.y_head = y_head;
  p.rows = static_cast<int>(rows), p.in = in, p.out = out;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (dtype != LRI_FP32 && in % 8 == 0 && out % 8 == 0 && x_row % 8 == 0 && x_head % 8 == 0 && aligned16(x) && aligned16(w))
    return dtype == LRI_BF16 ? head_linear<__nv_bfloat16>(p, heads, transposed != 0, st)
                             : head_linear<__half>(p, heads, transposed != 0, st);
  const unsigned h = static_cast<unsigned>(heads), m = static_cast<unsigned>(rows);
  if (transposed)
    LRI_CUDA(launch_pdl(LRI_BY_TYPE(dtype, head_linear_t_generic_kernel), dim3((out + 127) / 128, h, m), dim3(128), 0, st, p));
  else
    LRI_CUDA(launch_pdl(LRI_BY_TYPE(dtype, head_linear_generic_kernel), dim3((out + 7) / 8, h, m), dim3(256), 0, st, p));
  LRI_LAUNCH_CHECK("head_linear_kernel");
  return LRI_OK;
}

extern "C" size_t lri_window_attention_scratch_bytes(int B, int heads, int dv, int64_t keys) {
  return B > 0 && heads > 0 && dv > 0 && keys > 0 ? latent_decode_scratch_bytes(B, heads, dv, keys) : 0;
}

extern "C" int lri_window_attention(int dtype, const void* q, int64_t q_row, int64_t q_head, const void* k, int64_t k_batch,
                                    int64_t k_row, int64_t k_head, const void* k2, int64_t k2_batch, int64_t k2_row, const void* v,
                                    int64_t v_batch, int64_t v_row, int64_t v_head, void* out, const void* input_pos,
                                    int pos_is_i64, int history, int64_t k_rows, int64_t window_size, float scale, int B, int S,
                                    int heads, int d1, int d2, int dv, void* scratch, size_t scratch_bytes,
                                    lri_stream_t stream) {
  LRI_REQUIRE(dtype_ok(dtype), LRI_ERR_UNSUPPORTED, "window_attention: dtype %d", dtype);
  LRI_REQUIRE(q && k && k2 && v && out && input_pos, LRI_ERR_ARG, "window_attention: NULL pointer");
  LRI_REQUIRE(B >= 0 && S >= 0 && heads > 0 && d1 > 0 && d2 >= 0 && dv > 0 && k_rows > 0 && window_size > 0, LRI_ERR_ARG,
              "window_attention: B=%d S=%d heads=%d d1=%d d2=%d dv=%d", B, S, heads, d1, d2, dv);
  LRI_REQUIRE(dv <= 1024 && d1 + d2 <= 2048, LRI_ERR_UNSUPPORTED, "window_attention: dv=%d d1+d2=%d", dv, d1 + d2);
  const int64_t rows = static_cast<int64_t>(B) * S;
  if (rows == 0) return LRI_OK;
  WindowParams p{};
  p.q = q, p.q_row = q_row, p.q_head = q_head, p.k = k, p.k_batch = k_batch, p.k_row = k_row, p.k_head = k_head;
  p.k2 = k2, p.k2_batch = k2_batch, p.k2_row = k2_row, p.v = v, p.v_batch = v_batch, p.v_row = v_row, p.v_head = v_head;
  p.out = out, p.input_pos = input_pos, p.pos_is_i64 = pos_is_i64, p.history = history, p.k_rows = k_rows;
  p.window = window_size, p.scale = scale, p.S = S, p.H = heads, p.d1 = d1, p.d2 = d2, p.dv = dv;
  p.group = 1, p.out_ld = static_cast<int64_t>(heads) * dv, p.out_scale = 1.0f;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (option(OPT_WINDOW_TC)) {
    if (latent_decode_supports(dtype, p)) return latent_decode_launch(dtype, p, B, scratch, scratch_bytes, st);
    if (window_attention_tc_supports(dtype, p, B)) return window_attention_tc_launch(dtype, p, B, st);
  }
  return window_attention_plain_launch(dtype, p, rows, st);
}
