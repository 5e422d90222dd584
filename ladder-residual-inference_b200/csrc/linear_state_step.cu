// One token of a matrix-state recurrence (linear_state.cuh) with everything around it in one kernel: from the fp32 input
// projections to the rows that the output projection reads.
//
//   gated delta rule          convolutions with the ring, silu, unit vectors, both low-rank second projections, decay, step
//                             size, state update, readout, RMSNorm over the value channels, sigmoid gate
//   gated linear attention    low-rank decay, state update, readout, RMSNorm, silu gate
//
// A cluster serves one (sequence, head), each CTA 32 NC value channels.  A warp owns 4 NC of them, 8 lanes a column of the
// state.  What all columns need (queries, keys, decays) every CTA computes for itself; only the sums of squares of the
// results cross the cluster.  A small grid takes NC = 1 (shortest chain), a large one NC = 4 (least work, mostly no cluster).
// Weights are fetched, and the state is asked into the L2, before the preceding kernel is awaited.
#include <cooperative_groups.h>

#include "linear_state.cuh"

namespace cg = cooperative_groups;

namespace lri {
namespace {

constexpr int kThreads = 256, kMaxCluster = 8;
constexpr int kRegTaps = 4;  // convolution weights up to this many taps are held in registers
constexpr int kStageBytes = 96 * 1024;  // second projections up to this size are staged in shared memory

struct StepParams {
  const float* proj;  // [B, ld]
  int64_t ld, q_off, k_off, v_off, b_off, a_off, gate_off;  // a: input of the decay's projection; gate: of the gate's, or the gate
  const void *conv_q, *conv_k, *conv_v;
  int taps;
  float* ring;
  const void *a2, *g2;  // [H * C, a_rank], [H * E, g_rank]; ranks are multiples of 8
  int a_rank, g_rank;
  const void *a_log, *bias;  // bias: dt_bias, or the decay projection's
  float inv_tau;
  const void* norm_w;
  float eps;
  float* state;
  const void* input_pos;
  int pos_is_i64;
  void* out;  // out + b * out_ld + h * E
  int64_t out_ld;
  float factor;
  int H, G, C, E;
  int staged;
};

__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(dst))), "l"(src) : "memory");
}

// y[row] = w[row] . x for n rows: 8 lanes a row, 4 rows a warp
template <typename T>
__device__ __forceinline__ void rows_dot(const T* w, int rank, const float* x, int n, float* y) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, part = (lane & 7) * 8;
  for (int r0 = warp * 4; r0 < n; r0 += kThreads / 8) {
    const int r = r0 + (lane >> 3);
    float acc = 0.f;
    if (r < n)
      for (int i = part; i < rank; i += 64) {
        float f[8], xv[8];
        load8<T>(w + r * rank + i, f);
        load8<float>(x + i, xv);
#pragma unroll
        for (int e = 0; e < 8; ++e) acc = fmaf(f[e], xv[e], acc);
      }
#pragma unroll
    for (int o = 1; o < 8; o <<= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
    if ((lane & 7) == 0 && r < n) y[r] = acc;
  }
}

// Convolution of one channel at this position, silu taken; its input enters the ring.  The slots that are read are other ones
// than the one that is written.
template <typename T>
struct StepConv {
  float w[kRegTaps];  // w[j]: tap j tokens back
  const T* taps_w;
  __device__ __forceinline__ void load(const void* w_all, int64_t ch, int taps, bool live) {
    taps_w = static_cast<const T*>(w_all) + ch * taps;
#pragma unroll
    for (int j = 0; j < kRegTaps; ++j) w[j] = live && taps <= kRegTaps && j < taps ? Num<T>::to_f(taps_w[taps - 1 - j]) : 0.f;
  }
  // slot: pos % taps
  __device__ __forceinline__ float run(float x, float* ring, int64_t channels, int taps, int pos, int slot, bool keep) const {
    float y = w[0] * x;
    if (taps <= kRegTaps) {
      float old[kRegTaps];
#pragma unroll
      for (int j = 1; j < kRegTaps; ++j) {
        const int at = slot >= j ? slot - j : slot - j + taps;
        old[j] = j < taps && pos >= j ? ring[at * channels] : 0.f;
      }
#pragma unroll
      for (int j = 1; j < kRegTaps; ++j) y = fmaf(w[j], old[j], y);
    } else {
      y = Num<T>::to_f(taps_w[taps - 1]) * x;
      for (int j = 1; j < taps; ++j)
        if (pos >= j) y = fmaf(Num<T>::to_f(taps_w[taps - 1 - j]), ring[(slot >= j ? slot - j : slot - j + taps) * channels], y);
    }
    if (keep && pos >= 0) ring[slot * channels] = x;
    return silu_f(y);
  }
};

template <typename T, bool DELTA, int RV, int NC>
__global__ void __launch_bounds__(kThreads, RV <= 4 ? 2 : 1) state_step_kernel(const StepParams p) {
  constexpr int CP = 32 * RV, kCols = 32 * NC;
  extern __shared__ __align__(16) uint8_t step_smem[];
  static_assert(CP <= kThreads && kCols <= kThreads, "a thread takes one key channel and one value channel");
  __shared__ __align__(16) float sq[CP], sk[CP], sg[CP];
  __shared__ float sbias[CP];
  __shared__ float sv[kCols], sgate[kCols], part[8], part_qk[8][3], cluster_part[kMaxCluster];
  cg::cluster_group cluster = cg::this_cluster();
  const int ranks = static_cast<int>(cluster.num_blocks());
  if (ranks > 1) asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory");  // waited for before the first remote store
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, rg = lane & 7, cl = lane >> 3;
  const int h = blockIdx.y, H = p.H, G = p.G, C = p.C, E = p.E, hk = h / (H / G);
  const int64_t b = blockIdx.z;
  const int col0 = blockIdx.x * kCols, my = (warp * 4 + cl) * NC, e0 = col0 + my;
  const int cols = E - col0 < kCols ? E - col0 : kCols;
  float* x_a = reinterpret_cast<float*>(step_smem);  // input of the decay's second projection
  float* x_g = x_a + p.a_rank;
  T* w_smem = reinterpret_cast<T*>(x_g + (DELTA ? p.g_rank : 0));
  const T* a2 = static_cast<const T*>(p.a2) + static_cast<int64_t>(h) * C * p.a_rank;
  const T* g2 = DELTA ? static_cast<const T*>(p.g2) + (static_cast<int64_t>(h) * E + col0) * p.g_rank : nullptr;
  float* st_base = p.state + (b * H + h) * static_cast<int64_t>(C) * E;
  if (p.staged) {  // constants of the model
    constexpr int kPer = 16 / sizeof(T);
    const int na = C * p.a_rank / kPer, ng = DELTA ? cols * p.g_rank / kPer : 0;
    for (int i = tid; i < na; i += kThreads) cp_async16(w_smem + i * kPer, a2 + i * kPer);
    for (int i = tid; i < ng; i += kThreads) cp_async16(w_smem + (na + i) * kPer, g2 + i * kPer);
    a2 = w_smem;
    if (DELTA) g2 = w_smem + na * kPer;
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
  for (int i = tid; i < C * NC; i += kThreads)  // one request per 128-byte line
    if (i % NC * 32 < cols) asm volatile("prefetch.global.L2 [%0];" ::"l"(st_base + i / NC * E + col0 + i % NC * 32));
  // a thread takes key channel tid and, the last ones, a value channel
  const int64_t ch_k = static_cast<int64_t>(hk) * C + tid;
  const int e_mine = tid - (kThreads - kCols);
  const bool has_k = tid < C, has_v = e_mine >= 0 && e_mine < cols;
  const int64_t ch_v = static_cast<int64_t>(h) * E + col0 + e_mine;
  [[maybe_unused]] StepConv<T> conv_q, conv_k, conv_v;
  float a = 0.f;
  if constexpr (DELTA) {
    conv_q.load(p.conv_q, ch_k, p.taps, has_k);
    conv_k.load(p.conv_k, ch_k, p.taps, has_k);
    conv_v.load(p.conv_v, ch_v, p.taps, has_v);
    a = expf(Num<T>::to_f(static_cast<const T*>(p.a_log)[h]));
  }
  if (has_k) sbias[tid] = Num<T>::to_f(static_cast<const T*>(p.bias)[h * C + tid]);
  float norm_w[NC];
#pragma unroll
  for (int j = 0; j < NC; ++j) norm_w[j] = e0 + j < E ? Num<T>::to_f(static_cast<const T*>(p.norm_w)[e0 + j]) : 0.f;
  pdl_launch_dependents();
  pdl_wait();

  // ---- state, and what the columns share -------------------------------------------------------------------
  const int pos = static_cast<int>(load_pos(p.input_pos, p.pos_is_i64, 0));
  float st[RV][4][NC];
  float* st_mine = st_base + 4 * rg * E + e0;
#pragma unroll
  for (int i = 0; i < RV; ++i)
#pragma unroll
    for (int r = 0; r < 4; ++r) {
      const bool live = (C == CP || 32 * i + 4 * rg + r < C) && e0 < E;
      if constexpr (NC == 4) {  // E is a multiple of 4
        const float4 v = pos > 0 && live ? *reinterpret_cast<const float4*>(st_mine + (32 * i + r) * E) : make_float4(0.f, 0.f, 0.f, 0.f);
        st[i][r][0] = v.x, st[i][r][1] = v.y, st[i][r][2] = v.z, st[i][r][3] = v.w;
      } else {
        st[i][r][0] = pos > 0 && live ? st_mine[(32 * i + r) * E] : 0.f;
      }
    }
  const float* in = p.proj + b * p.ld;
  const int64_t channels = 2ll * G * C + static_cast<int64_t>(H) * E;
  float* ring = DELTA ? p.ring + b * p.taps * channels : nullptr;
  const float beta = DELTA ? sigmoid_f(in[p.b_off + h]) : 0.f;
  const int slot = DELTA ? (pos < 0 ? 0 : pos) % p.taps : 0;
  float q = 0.f, k = 0.f;
  if (tid < CP) {
    if (has_k) {
      q = in[p.q_off + ch_k], k = in[p.k_off + ch_k];
      if constexpr (DELTA) {
        const bool keep = blockIdx.x == 0 && h % (H / G) == 0;  // the first CTA of a group keeps the shared channels
        q = conv_q.run(q, ring + ch_k, channels, p.taps, pos, slot, keep);
        k = conv_k.run(k, ring + static_cast<int64_t>(G) * C + ch_k, channels, p.taps, pos, slot, keep);
      }
    } else {
      sg[tid] = 1.f;
    }
    sq[tid] = q, sk[tid] = k;
  }
  if (e_mine >= 0) {
    float v = 0.f;
    if (has_v) {
      v = in[p.v_off + ch_v];
      if constexpr (DELTA)
        v = conv_v.run(v, ring + 2ll * G * C + ch_v, channels, p.taps, pos, slot, true);
    }
    sv[e_mine] = v;
    if (!DELTA) sgate[e_mine] = has_v ? silu_f(in[p.gate_off + ch_v]) : 0.f;
  }
  for (int i = tid; i < p.a_rank; i += kThreads) x_a[i] = rnd<T>(in[p.a_off + i]);
  if (DELTA)
    for (int i = tid; i < p.g_rank; i += kThreads) x_g[i] = rnd<T>(in[p.gate_off + i]);
  if constexpr (DELTA) {
    const float qq = warp_sum(q * q), kk = warp_sum(k * k), kq = warp_sum(k * q);
    if (lane == 0) part_qk[warp][0] = qq, part_qk[warp][1] = kk, part_qk[warp][2] = kq;
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();

  rows_dot<T>(a2, p.a_rank, x_a, C, sg);
  if constexpr (DELTA) rows_dot<T>(g2, p.g_rank, x_g, cols, sgate);
  float qs = 1.0f / sqrtf(static_cast<float>(C)), ks = 1.f, kq = 0.f;
  if constexpr (DELTA) {
    float qq = 0.f, kk = 0.f;
#pragma unroll
    for (int w = 0; w < (CP < kThreads ? CP / 32 : 8); ++w) qq += part_qk[w][0], kk += part_qk[w][1], kq += part_qk[w][2];
    qs /= sqrtf(qq + kUnitEps);
    ks = 1.0f / sqrtf(kk + kUnitEps);
    kq *= ks * qs;
  }
  __syncthreads();
  if (has_k) {
    const float z = sg[tid] + sbias[tid];
    sg[tid] = DELTA ? delta_decay_f(z, a) : logistic_decay_f(z, p.inv_tau);
  }
  if (DELTA && has_v) sgate[e_mine] = sigmoid_f(sgate[e_mine]);
  __syncthreads();

  // ---- the recurrence ------------------------------------------------------------------------------------------
  float dk[NC], dq[NC], u[NC], o[NC];
#pragma unroll
  for (int j = 0; j < NC; ++j) dk[j] = dq[j] = 0.f, u[j] = sv[my + j];
#pragma unroll
  for (int i = 0; i < RV; ++i) {
    float g[4], q4[4], k4[4];
    *reinterpret_cast<float4*>(g) = *reinterpret_cast<const float4*>(&sg[32 * i + 4 * rg]);
    *reinterpret_cast<float4*>(q4) = *reinterpret_cast<const float4*>(&sq[32 * i + 4 * rg]);
    *reinterpret_cast<float4*>(k4) = *reinterpret_cast<const float4*>(&sk[32 * i + 4 * rg]);
#pragma unroll
    for (int r = 0; r < 4; ++r)
#pragma unroll
      for (int j = 0; j < NC; ++j) {
        float& x = st[i][r][j];
        x *= g[r];
        if (DELTA)
          dk[j] = fmaf(x, k4[r], dk[j]);
        else
          x = fmaf(k4[r], u[j], x);
        dq[j] = fmaf(x, q4[r], dq[j]);
      }
  }
#pragma unroll
  for (int w = 1; w < 8; w <<= 1)
#pragma unroll
    for (int j = 0; j < NC; ++j) {
      if (DELTA) dk[j] += __shfl_xor_sync(0xffffffffu, dk[j], w);
      dq[j] += __shfl_xor_sync(0xffffffffu, dq[j], w);
    }
  float squares = 0.f;
#pragma unroll
  for (int j = 0; j < NC; ++j) {
    o[j] = dq[j] * qs;
    if constexpr (DELTA) {
      u[j] = beta * (u[j] - dk[j] * ks);
      o[j] = fmaf(u[j], kq, o[j]);
      u[j] *= ks;
    }
    if (e0 + j < E) squares = fmaf(o[j], o[j], squares);
  }

  // ---- norm over the head's value channels, gate -----------------------------------------------------------------
  const float ss = warp_sum(rg == 0 ? squares : 0.f);
  if (lane == 0) part[warp] = ss;
  __syncthreads();
  float total = 0.f;
  if (ranks > 1) {
    asm volatile("barrier.cluster.wait.aligned;" ::: "memory");
    if (tid < ranks) {
      float s = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) s += part[w];
      *cluster.map_shared_rank(&cluster_part[cluster.block_rank()], tid) = s;
    }
    cluster.sync();
    for (int r = 0; r < ranks; ++r) total += cluster_part[r];
  } else {
#pragma unroll
    for (int w = 0; w < 8; ++w) total += part[w];
  }
  if (rg == 0) {
    const float inv = p.factor / sqrtf(total / static_cast<float>(E) + p.eps);
    T* dst = static_cast<T*>(p.out) + b * p.out_ld + static_cast<int64_t>(h) * E + e0;
#pragma unroll
    for (int j = 0; j < NC; ++j)
      if (e0 + j < E) dst[j] = Num<T>::from_f(o[j] * inv * norm_w[j] * sgate[my + j]);
  }

  // ---- the state, behind the barriers, which would wait for its stores ---------------------------------------------
#pragma unroll
  for (int i = 0; i < RV; ++i) {
    float k4[4];
    *reinterpret_cast<float4*>(k4) = *reinterpret_cast<const float4*>(&sk[32 * i + 4 * rg]);
#pragma unroll
    for (int r = 0; r < 4; ++r) {
      if (DELTA)
#pragma unroll
        for (int j = 0; j < NC; ++j) st[i][r][j] = fmaf(k4[r], u[j], st[i][r][j]);
      if ((C == CP || 32 * i + 4 * rg + r < C) && e0 < E) {
        if constexpr (NC == 4)
          *reinterpret_cast<float4*>(st_mine + (32 * i + r) * E) = make_float4(st[i][r][0], st[i][r][1], st[i][r][2], st[i][r][3]);
        else
          st_mine[(32 * i + r) * E] = st[i][r][0];
      }
    }
  }
}

template <typename T, bool DELTA, int RV, int NC>
int launch(const StepParams& p, int B, cudaStream_t st) {
  constexpr int kCols = 32 * NC;
  const size_t x_bytes = (static_cast<size_t>(p.a_rank) + (DELTA ? p.g_rank : 0)) * 4;
  const size_t w_bytes = (static_cast<size_t>(p.C) * p.a_rank + (DELTA ? static_cast<size_t>(kCols) * p.g_rank : 0)) * sizeof(T);
  const unsigned cs = (p.E + kCols - 1) / kCols;
  StepParams q = p;
  q.staged = w_bytes <= kStageBytes;
  auto kern = state_step_kernel<T, DELTA, RV, NC>;
  static std::atomic<unsigned long long> attr_set{0};
  LRI_ONCE_PER_DEVICE(attr_set, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 2 * kStageBytes));
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(cs, p.H, B);
  cfg.blockDim = dim3(kThreads);
  cfg.dynamicSmemBytes = x_bytes + (q.staged ? w_bytes : 0);
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = cs;
  attr[0].val.clusterDim.y = 1;
  attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = pdl_enabled() ? 2 : 1;
  LRI_CUDA(cudaLaunchKernelEx(&cfg, kern, q));
  LRI_LAUNCH_CHECK("state_step_kernel");
  return LRI_OK;
}
template <typename T, bool DELTA, int RV>
int by_grid(const StepParams& p, int B, cudaStream_t st) {
  if constexpr (RV <= 4) {
    const int64_t ctas = static_cast<int64_t>(B) * p.H * ((p.E + 31) / 32);
    if (ctas > 2ll * device_sm_count() && p.E % 4 == 0 && p.E > 32) return launch<T, DELTA, RV, 4>(p, B, st);
  }
  return launch<T, DELTA, RV, 1>(p, B, st);
}
template <typename T, bool DELTA>
int by_channels(const StepParams& p, int B, cudaStream_t st) {
  if (p.C <= 32) return by_grid<T, DELTA, 1>(p, B, st);
  if (p.C <= 64) return by_grid<T, DELTA, 2>(p, B, st);
  if (p.C <= 128) return by_grid<T, DELTA, 4>(p, B, st);
  return by_grid<T, DELTA, 8>(p, B, st);
}
template <bool DELTA>
int run(const char* who, int dtype, const StepParams& p, int B, cudaStream_t st) {
  LRI_REQUIRE(dtype >= LRI_BF16 && dtype <= LRI_FP32, LRI_ERR_UNSUPPORTED, "%s: dtype %d", who, dtype);
  LRI_REQUIRE(p.proj && p.a2 && p.bias && p.norm_w && p.state && p.input_pos && p.out, LRI_ERR_ARG, "%s: NULL pointer", who);
  LRI_REQUIRE(B >= 0 && B <= 65535 && p.H > 0 && p.H <= 65535 && p.G > 0 && p.H % p.G == 0, LRI_ERR_ARG, "%s: B=%d heads=%d kv_heads=%d", who,
              B, p.H, p.G);
  LRI_REQUIRE(lri_state_step_supports(p.C, p.E, p.a_rank, p.g_rank), LRI_ERR_UNSUPPORTED, "%s: dim=%d vdim=%d ranks %d, %d", who, p.C, p.E,
              p.a_rank, p.g_rank);
  LRI_REQUIRE(aligned16(p.a2) && aligned16(p.g2) && aligned16(p.state), LRI_ERR_ALIGN,
              "%s: second projections and state must be 16-byte aligned", who);
  if (B == 0) return LRI_OK;
  if (dtype == LRI_BF16) return by_channels<__nv_bfloat16, DELTA>(p, B, st);
  if (dtype == LRI_FP16) return by_channels<__half, DELTA>(p, B, st);
  return by_channels<float, DELTA>(p, B, st);
}

}  // namespace
}  // namespace lri

using namespace lri;

extern "C" int lri_state_step_supports(int dim, int vdim, int decay_rank, int gate_rank) {
  return dim >= 1 && dim <= 256 && vdim >= 1 && vdim <= 32 * kMaxCluster && decay_rank >= 8 && decay_rank % 8 == 0 && decay_rank <= 4096 &&
         gate_rank >= 0 && gate_rank % 8 == 0 && gate_rank <= 4096;
}

extern "C" int lri_delta_step(int dtype, const float* proj, int64_t ld, int64_t q_off, int64_t k_off, int64_t v_off, int64_t a_off,
                              int64_t g_off, int64_t b_off, const void* conv_q, const void* conv_k, const void* conv_v, int taps,
                              float* ring, const void* a2, int a_rank, const void* g2, int g_rank, const void* a_log,
                              const void* dt_bias, const void* norm_weight, float eps, float factor, float* state,
                              const void* input_pos, int pos_is_i64, void* out, int64_t out_ld, int B, int heads, int kv_heads, int dim,
                              int vdim, lri_stream_t stream) {
  LRI_REQUIRE(conv_q && conv_k && conv_v && ring && g2 && a_log && taps >= 1 && taps <= kMaxTaps && g_rank >= 8, LRI_ERR_ARG,
              "delta_step: NULL pointer, taps=%d or gate rank %d", taps, g_rank);
  StepParams p{};
  p.proj = proj, p.ld = ld, p.q_off = q_off, p.k_off = k_off, p.v_off = v_off, p.a_off = a_off, p.gate_off = g_off, p.b_off = b_off;
  p.conv_q = conv_q, p.conv_k = conv_k, p.conv_v = conv_v, p.taps = taps, p.ring = ring, p.a2 = a2, p.g2 = g2, p.a_rank = a_rank, p.g_rank = g_rank;
  p.a_log = a_log, p.bias = dt_bias, p.norm_w = norm_weight, p.eps = eps, p.factor = factor, p.state = state;
  p.input_pos = input_pos, p.pos_is_i64 = pos_is_i64, p.out = out, p.out_ld = out_ld, p.H = heads, p.G = kv_heads, p.C = dim, p.E = vdim;
  return run<true>("delta_step", dtype, p, B, static_cast<cudaStream_t>(stream));
}

extern "C" int lri_gla_step(int dtype, const float* proj, int64_t ld, int64_t q_off, int64_t k_off, int64_t v_off, int64_t a_off,
                            int64_t g_off, const void* a2, int a_rank, const void* bias, float tau, const void* norm_weight, float eps,
                            float factor, float* state, const void* input_pos, int pos_is_i64, void* out, int64_t out_ld, int B, int heads,
                            int dim, int vdim, lri_stream_t stream) {
  LRI_REQUIRE(tau > 0.f, LRI_ERR_ARG, "gla_step: tau=%g", tau);
  StepParams p{};
  p.proj = proj, p.ld = ld, p.q_off = q_off, p.k_off = k_off, p.v_off = v_off, p.a_off = a_off, p.gate_off = g_off;
  p.a2 = a2, p.a_rank = a_rank, p.bias = bias, p.inv_tau = 1.0f / tau, p.norm_w = norm_weight, p.eps = eps, p.factor = factor, p.state = state;
  p.input_pos = input_pos, p.pos_is_i64 = pos_is_i64, p.out = out, p.out_ld = out_ld, p.H = heads, p.G = heads, p.C = dim, p.E = vdim;
  return run<false>("gla_step", dtype, p, B, static_cast<cudaStream_t>(stream));
}
