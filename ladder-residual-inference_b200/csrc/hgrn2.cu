// HGRN2 token mixer: linear attention whose forget gate, per head and channel, also scales what is written.
//
//   f = low + (1 - low) * sigmoid(f_raw + f_bias)          q = silu(q_raw)
//   S_t[c, e] = f_t[c] S_{t-1}[c, e] + (1 - f_t[c]) v_t[e]
//   o_t[e] = sum_c q_t[c] S_t[c, e]                         then RMSNorm over e, one weight for all heads
//
// Here the token-by-token form: single tokens, short portions, fp32 models and sizes the block form does not take.
// The projections arrive in fp32; gates, state and sums stay fp32, v is taken in the storage type.  The state of sequence b and head h is
// [C, E] in `state`; a call whose first position is 0 starts from zero, any other continues what the previous call left.
#include "hgrn2.cuh"

namespace lri {
namespace {

constexpr int kWarps = 8;

// Grid (column slices, heads, sequences).  A warp owns the state rows c = warp, warp + 8, ... and its lanes the
// columns of the slice, VEC each; the rows of a thread stay in registers over all tokens of the call.
template <typename T, int NR, int VEC>
__global__ void __launch_bounds__(kWarps * 32) hgrn2_steps_kernel(const Hgrn2Params p) {
  extern __shared__ float hg_smem[];
  float* qs = hg_smem;          // [C]
  float* fs = hg_smem + p.C;    // [C]
  __shared__ float red[kWarps][32 * VEC];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y, b = blockIdx.z, H = p.H, C = p.C, E = p.E;
  const int e0 = blockIdx.x * 32 * VEC + lane * VEC;
  const bool live = e0 < E;
  const T* bias = static_cast<const T*>(p.f_bias) + h * C;
  const T* lower = static_cast<const T*>(p.lower) + h * C;
  float* st_base = p.state + (static_cast<int64_t>(b) * H + h) * C * E;
  pdl_launch_dependents();
  pdl_wait();
  const bool fresh = load_pos(p.input_pos, p.pos_is_i64, 0) <= 0;
  float st[NR][VEC];
#pragma unroll
  for (int r = 0; r < NR; ++r) {
    const int c = warp + r * kWarps;
#pragma unroll
    for (int e = 0; e < VEC; ++e) st[r][e] = 0.f;
    if (!fresh && live && c < C) {
      if constexpr (VEC == 4) {
        const float4 v = *reinterpret_cast<const float4*>(st_base + static_cast<int64_t>(c) * E + e0);
        st[r][0] = v.x, st[r][1] = v.y, st[r][2] = v.z, st[r][3] = v.w;
      } else {
        st[r][0] = st_base[static_cast<int64_t>(c) * E + e0];
      }
    }
  }
  for (int t = 0; t < p.S; ++t) {
    const int64_t row = static_cast<int64_t>(b) * p.S + t;
    const float* pr = p.proj + row * p.ld;
    for (int c = threadIdx.x; c < C; c += kWarps * 32) {
      qs[c] = silu_f(pr[p.q_off + h * C + c]);
      fs[c] = forget_gate(pr[p.f_off + h * C + c], Num<T>::to_f(bias[c]), Num<T>::to_f(lower[c]));
    }
    float v[VEC], o[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      v[e] = live ? rnd<T>(pr[p.v_off + h * E + e0 + e]) : 0.f;
      o[e] = 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int r = 0; r < NR; ++r) {
      const int c = warp + r * kWarps;
      if (c < C) {
        const float f = fs[c], w = 1.0f - f, q = qs[c];
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          st[r][e] = fmaf(f, st[r][e], w * v[e]);
          o[e] = fmaf(q, st[r][e], o[e]);
        }
      }
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) red[warp][lane * VEC + e] = o[e];
    __syncthreads();
    if (warp == 0) {
      float ss = 0.f;
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        float s = 0.f;
#pragma unroll
        for (int w = 0; w < kWarps; ++w) s += red[w][lane * VEC + e];
        o[e] = live ? s : 0.f;
        ss += o[e] * o[e];
      }
      if (p.o_raw) {
        if (live)
#pragma unroll
          for (int e = 0; e < VEC; ++e) p.o_raw[(row * H + h) * E + e0 + e] = o[e];
      } else {
        const float inv = 1.0f / sqrtf(warp_sum(ss) / static_cast<float>(E) + p.eps);
        const T* w = static_cast<const T*>(p.norm_w);
        T* out = static_cast<T*>(p.out) + (row * H + h) * E + e0;
        if (live)
#pragma unroll
          for (int e = 0; e < VEC; ++e) out[e] = Num<T>::from_f(o[e] * inv * Num<T>::to_f(w[e0 + e]));
      }
    }
  }
#pragma unroll
  for (int r = 0; r < NR; ++r) {
    const int c = warp + r * kWarps;
    if (live && c < C) {
      if constexpr (VEC == 4)
        *reinterpret_cast<float4*>(st_base + static_cast<int64_t>(c) * E + e0) = make_float4(st[r][0], st[r][1], st[r][2], st[r][3]);
      else
        st_base[static_cast<int64_t>(c) * E + e0] = st[r][0];
    }
  }
}

// RMSNorm over each head's E values: one warp per (row, head)
template <typename T>
__global__ void __launch_bounds__(256)
head_rmsnorm_kernel(const float* o, const T* w, float eps, T* out, int64_t rows, int E) {
  const int64_t r = static_cast<int64_t>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  pdl_launch_dependents();
  pdl_wait();
  if (r >= rows) return;
  float ss = 0.f;
  for (int e = lane; e < E; e += 32) ss += o[r * E + e] * o[r * E + e];
  const float inv = 1.0f / sqrtf(warp_sum(ss) / static_cast<float>(E) + eps);
  for (int e = lane; e < E; e += 32) out[r * E + e] = Num<T>::from_f(o[r * E + e] * inv * Num<T>::to_f(w[e]));
}

template <typename T>
int head_norm(const Hgrn2Params& p, int64_t rows, cudaStream_t st) {
  const int64_t n = rows * p.H;
  LRI_CUDA(launch_pdl(head_rmsnorm_kernel<T>, dim3(static_cast<unsigned>((n + 7) / 8)), dim3(256), 0, st,
                      static_cast<const float*>(p.o_raw), static_cast<const T*>(p.norm_w), p.eps, static_cast<T*>(p.out), n, p.E));
  LRI_LAUNCH_CHECK("head_rmsnorm_kernel");
  return LRI_OK;
}

template <typename T, int NR, int VEC>
int launch_steps(const Hgrn2Params& p, int B, int slices, cudaStream_t st) {
  LRI_CUDA(launch_pdl(hgrn2_steps_kernel<T, NR, VEC>, dim3(slices, p.H, B), dim3(kWarps * 32),
                      2 * static_cast<size_t>(p.C) * sizeof(float), st, p));
  LRI_LAUNCH_CHECK("hgrn2_steps_kernel");
  return LRI_OK;
}

// Form that takes any size: columns cut so that a warp's lanes cover a slice.
bool wide_columns(const Hgrn2Params& p) { return p.E % 4 == 0 && p.E >= 64 && p.C <= 256; }
int column_slices(const Hgrn2Params& p) {
  const int per = wide_columns(p) ? 128 : 32;
  return (p.E + per - 1) / per;
}

template <typename T>
int steps(Hgrn2Params p, int B, cudaStream_t st) {
  const int slices = column_slices(p);
  if (slices == 1) p.o_raw = nullptr;
  int rc;
  if (wide_columns(p)) {
    if (p.C <= 64)
      rc = launch_steps<T, 8, 4>(p, B, slices, st);
    else if (p.C <= 128)
      rc = launch_steps<T, 16, 4>(p, B, slices, st);
    else
      rc = launch_steps<T, 32, 4>(p, B, slices, st);
  } else {
    if (p.C <= 64)
      rc = launch_steps<T, 8, 1>(p, B, slices, st);
    else if (p.C <= 256)
      rc = launch_steps<T, 32, 1>(p, B, slices, st);
    else
      rc = launch_steps<T, 64, 1>(p, B, slices, st);
  }
  if (rc != LRI_OK || slices == 1) return rc;
  return head_norm<T>(p, static_cast<int64_t>(B) * p.S, st);
}

constexpr int kMaxChannels = 512;

}  // namespace
}  // namespace lri

using namespace lri;

extern "C" size_t lri_hgrn2_workspace_bytes(int dtype, int B, int S, int heads, int dim, int vdim) {
  (void)dtype;
  if (B <= 0 || S <= 0 || heads <= 0 || dim <= 0 || vdim <= 0) return 0;
  const size_t raw = static_cast<size_t>(B) * S * heads * vdim * sizeof(float);
  const size_t blocks = hgrn2_blocks_workspace_bytes(B, S, heads, dim, vdim);
  return raw > blocks ? raw : blocks;
}

extern "C" int lri_hgrn2(int dtype, const float* proj, int64_t ld, int64_t q_off, int64_t f_off, int64_t v_off,
                         const void* f_bias, const void* lower, const void* norm_weight, float eps, float* state,
                         const void* input_pos, int pos_is_i64, void* out, int B, int S, int heads, int dim, int vdim,
                         void* workspace, size_t workspace_bytes, lri_stream_t stream) {
  LRI_REQUIRE(dtype >= LRI_BF16 && dtype <= LRI_FP32, LRI_ERR_UNSUPPORTED, "hgrn2: dtype %d", dtype);
  LRI_REQUIRE(proj && f_bias && lower && norm_weight && state && input_pos && out, LRI_ERR_ARG, "hgrn2: NULL pointer");
  LRI_REQUIRE(B >= 0 && B <= 65535 && S >= 0 && heads > 0 && heads <= 65535 && dim > 0 && vdim > 0, LRI_ERR_ARG,
              "hgrn2: B=%d S=%d heads=%d dim=%d vdim=%d", B, S, heads, dim, vdim);
  LRI_REQUIRE(dim <= kMaxChannels, LRI_ERR_UNSUPPORTED, "hgrn2: dim=%d > %d", dim, kMaxChannels);
  LRI_REQUIRE(aligned16(state), LRI_ERR_ALIGN, "hgrn2: state must be 16-byte aligned");
  if (B == 0 || S == 0) return LRI_OK;
  LRI_REQUIRE(workspace && aligned16(workspace) && workspace_bytes >= lri_hgrn2_workspace_bytes(dtype, B, S, heads, dim, vdim),
              LRI_ERR_WORKSPACE, "hgrn2: workspace of %zu bytes (16-byte aligned) required",
              lri_hgrn2_workspace_bytes(dtype, B, S, heads, dim, vdim));
  Hgrn2Params p{};
  p.proj = proj, p.ld = ld, p.q_off = q_off, p.f_off = f_off, p.v_off = v_off;
  p.f_bias = f_bias, p.lower = lower, p.norm_w = norm_weight, p.eps = eps, p.state = state;
  p.input_pos = input_pos, p.pos_is_i64 = pos_is_i64, p.out = out, p.o_raw = static_cast<float*>(workspace);
  p.S = S, p.H = heads, p.C = dim, p.E = vdim;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (option(OPT_HGRN2_BLOCKS) && hgrn2_blocks_supports(dtype, p, B)) return hgrn2_blocks_launch(dtype, p, B, workspace, st);
  if (dtype == LRI_BF16) return steps<__nv_bfloat16>(p, B, st);
  if (dtype == LRI_FP16) return steps<__half>(p, B, st);
  return steps<float>(p, B, st);
}
