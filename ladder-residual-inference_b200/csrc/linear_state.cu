// Matrix-state recurrences over the tokens of a call (see linear_state.cuh), and what surrounds them:
//
//   delta_prepare    short convolutions, activations, unit vectors, decays and step sizes of the gated delta rule
//   conv_ring        the last convolution inputs of the call become state
//   logistic_decay   decays of gated linear attention
//   state_scan       the recurrence itself, any number of tokens
//   head_norm_gate   RMSNorm of each head's result, elementwise gate, factor, rounding
//
// The columns of a state (value channels) do not depend on one another: u, o and the update of column e use only that
// column.  So the scan needs no barrier between tokens: a warp owns a few columns, its lanes split the rows of S (8 lanes
// a column), and the two sums over rows, S^T k and S^T q, are taken of the decayed state at once, since
//   o = (S + k u^T)^T q = S^T q + (k . q) u.
// Rows stay in registers over all tokens, as pairs for the packed fp32 instructions; the tokens' vectors arrive in shared
// memory 16 tokens ahead.
#include "linear_state.cuh"

#include <type_traits>

namespace lri {
namespace {

// ---- packed fp32 pairs -------------------------------------------------------------------------------
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
__device__ __forceinline__ float sum_f2(f2 v) {
  float a, b;
  unpack_f2(v, a, b);
  return a + b;
}

__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async4(uint32_t dst, const void* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(dst), "l"(src) : "memory");
}

// ---- gated delta rule: everything in front of the recurrence -----------------------------------------
struct DeltaPrepareParams {
  const float* proj;  // [rows, ld]
  int64_t ld, q_off, k_off, v_off, b_off;
  const void *conv_q, *conv_k, *conv_v;  // [channels, taps]
  int taps;
  const float* ring;  // [B, taps, 2 G C + H E]
  float* z;           // [rows, H * C] in: decay projection, out: decay
  const void *a_log, *dt_bias;
  const void* input_pos;
  int pos_is_i64;
  float *q, *k, *v;  // [rows, G, C], [rows, G, C], [rows, H, E]
  float* beta;       // [rows, H]
  float* kq;         // [rows, G]
  int S, H, G, C, E;
};

// One warp per (row, q/k head) or (row, value head)
template <typename T>
__global__ void __launch_bounds__(256) delta_prepare_kernel(const DeltaPrepareParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int unit = blockIdx.y * 8 + (threadIdx.x >> 5);
  if (unit >= p.G + p.H) return;
  const int64_t row = blockIdx.x, b = row / p.S;
  const int s = static_cast<int>(row - b * p.S);
  const int64_t pos = load_pos(p.input_pos, p.pos_is_i64, s);
  const int64_t channels = 2ll * p.G * p.C + static_cast<int64_t>(p.H) * p.E;
  const ConvInput ci{p.proj + b * p.S * p.ld, p.ld, p.ring + b * p.taps * channels, channels, p.taps};
  if (unit < p.G) {
    const int g = unit;
    float* qo = p.q + (row * p.G + g) * p.C;
    float* ko = p.k + (row * p.G + g) * p.C;
    float qq = 0.f, kk = 0.f, kq = 0.f;
    for (int c = lane; c < p.C; c += 32) {
      const int64_t ch = static_cast<int64_t>(g) * p.C + c;
      const float q = silu_f(short_conv<T>(ci, static_cast<const T*>(p.conv_q) + ch * p.taps, p.q_off + ch, ch, s, pos));
      const float k = silu_f(short_conv<T>(ci, static_cast<const T*>(p.conv_k) + ch * p.taps, p.k_off + ch,
                                           static_cast<int64_t>(p.G) * p.C + ch, s, pos));
      qo[c] = q, ko[c] = k;  // read back by the same lane
      qq = fmaf(q, q, qq), kk = fmaf(k, k, kk), kq = fmaf(k, q, kq);
    }
    const float iq = 1.0f / sqrtf(warp_sum(qq) + 1e-6f), ik = 1.0f / sqrtf(warp_sum(kk) + 1e-6f);
    kq = warp_sum(kq);
    for (int c = lane; c < p.C; c += 32) qo[c] *= iq, ko[c] *= ik;
    if (lane == 0) p.kq[row * p.G + g] = kq * iq * ik;
    return;
  }
  const int h = unit - p.G;
  for (int e = lane; e < p.E; e += 32) {
    const int64_t ch = static_cast<int64_t>(h) * p.E + e;
    p.v[row * p.H * p.E + ch] = silu_f(
        short_conv<T>(ci, static_cast<const T*>(p.conv_v) + ch * p.taps, p.v_off + ch, 2ll * p.G * p.C + ch, s, pos));
  }
  const float a = Num<T>::to_f(static_cast<const T*>(p.a_log)[h]);
  for (int c = lane; c < p.C; c += 32) {
    const int64_t ch = static_cast<int64_t>(h) * p.C + c;
    float* z = p.z + row * p.H * p.C + ch;
    *z = delta_decay_f(*z + Num<T>::to_f(static_cast<const T*>(p.dt_bias)[ch]), a);
  }
  if (lane == 0) p.beta[row * p.H + h] = sigmoid_f(p.proj[row * p.ld + p.b_off + h]);
}

// The inputs of the call's last `taps` tokens into the ring.  Runs behind delta_prepare, which reads older ones from it.
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

template <typename T>
__global__ void __launch_bounds__(256) logistic_decay_kernel(float* z, const T* bias, float inv_tau, int64_t n, int width) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t i = static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x;
  if (i >= n) return;
  z[i] = logistic_decay_f(z[i] + Num<T>::to_f(bias[i % width]), inv_tau);
}

// ---- the recurrence ------------------------------------------------------------------------------------
struct ScanParams {
  const float* q;  // q + row * q_row + (head / group) * C
  const float* k;
  const float* v;  // v + row * v_row + head * E
  const float* g;  // [rows, H, C]
  int64_t q_row, k_row, v_row;
  const float* beta;  // [rows, H] (delta rule)
  const float* kq;    // [rows, H / group]
  float* state;       // [B_max, H, C, E]
  const void* input_pos;
  int pos_is_i64;
  float* o;  // [rows, H, E]
  float o_scale;
  int S, H, group, C, E;
  int vec;  // rows are aligned for 16-byte copies
};

constexpr int kBlock = 16;  // tokens staged at a time

// RV: 4-row pieces of a column per lane (32 RV rows in all); NC: columns per lane (4 NC a warp).
template <bool DELTA, int RV, int NC>
__global__ void __launch_bounds__(128) state_scan_kernel(const ScanParams p) {
  constexpr int CP = 32 * RV;
  extern __shared__ __align__(16) float sc_smem[];
  const int warps = blockDim.x >> 5, cols = warps * 4 * NC;
  const int stage = kBlock * (3 * CP + cols + 4);  // q, k, g, v, (beta, kq)
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, rg = lane & 7, cl = lane >> 3;
  const int h = blockIdx.y, C = p.C, E = p.E, hk = h / p.group;
  const int64_t b = blockIdx.z;
  const int col0 = blockIdx.x * cols, my = warp * 4 * NC + cl * NC, e0 = col0 + my;
  float* st_base = p.state + (b * p.H + h) * static_cast<int64_t>(C) * E;
  for (int i = tid; i < 2 * stage; i += blockDim.x) sc_smem[i] = 0.f;  // rows and columns past the end stay zero
  pdl_launch_dependents();
  pdl_wait();
  __syncthreads();

  const int copy_cols = E - col0 < cols ? E - col0 : cols;
  auto fetch = [&](int s0, float* dst) {
    const int n = p.S - s0 < kBlock ? p.S - s0 : kBlock;
    const int64_t r0 = b * p.S + s0;
    const uint32_t base = static_cast<uint32_t>(__cvta_generic_to_shared(dst));
    if (p.vec) {
      const int nc = C >> 2, nv = copy_cols >> 2, per = 3 * nc + nv;
      for (int i = tid; i < n * per; i += blockDim.x) {
        const int t = i / per, x = i - t * per;
        const int64_t row = r0 + t;
        if (x < nc)
          cp_async16(base + (t * CP + 4 * x) * 4, p.q + row * p.q_row + hk * C + 4 * x);
        else if (x < 2 * nc)
          cp_async16(base + ((kBlock + t) * CP + 4 * (x - nc)) * 4, p.k + row * p.k_row + hk * C + 4 * (x - nc));
        else if (x < 3 * nc)
          cp_async16(base + ((2 * kBlock + t) * CP + 4 * (x - 2 * nc)) * 4, p.g + (row * p.H + h) * C + 4 * (x - 2 * nc));
        else
          cp_async16(base + (3 * kBlock * CP + t * cols + 4 * (x - 3 * nc)) * 4, p.v + row * p.v_row + h * E + col0 + 4 * (x - 3 * nc));
      }
    } else {
      const int per = 3 * C + copy_cols;
      for (int i = tid; i < n * per; i += blockDim.x) {
        const int t = i / per, x = i - t * per;
        const int64_t row = r0 + t;
        if (x < C)
          cp_async4(base + (t * CP + x) * 4, p.q + row * p.q_row + hk * C + x);
        else if (x < 2 * C)
          cp_async4(base + ((kBlock + t) * CP + x - C) * 4, p.k + row * p.k_row + hk * C + x - C);
        else if (x < 3 * C)
          cp_async4(base + ((2 * kBlock + t) * CP + x - 2 * C) * 4, p.g + (row * p.H + h) * C + x - 2 * C);
        else
          cp_async4(base + (3 * kBlock * CP + t * cols + x - 3 * C) * 4, p.v + row * p.v_row + h * E + col0 + x - 3 * C);
      }
    }
    if (DELTA)
      for (int t = tid; t < n; t += blockDim.x) {
        const uint32_t at = base + (kBlock * (3 * CP + cols) + 2 * t) * 4;
        cp_async4(at, p.beta + (r0 + t) * p.H + h);
        cp_async4(at + 4, p.kq + (r0 + t) * (p.H / p.group) + hk);
      }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(0, sc_smem);

  // rows of this lane: 32 i + 4 rg + 0 .. 3
  f2 st[NC][2 * RV];
  const bool fresh = load_pos(p.input_pos, p.pos_is_i64, 0) <= 0;
#pragma unroll
  for (int j = 0; j < NC; ++j)
#pragma unroll
    for (int i = 0; i < RV; ++i) {
      float x[4];
#pragma unroll
      for (int r = 0; r < 4; ++r) {
        const int c = 32 * i + 4 * rg + r;
        x[r] = !fresh && c < C && e0 + j < E ? st_base[static_cast<int64_t>(c) * E + e0 + j] : 0.f;
      }
      st[j][2 * i] = pack_f2(x[0], x[1]);
      st[j][2 * i + 1] = pack_f2(x[2], x[3]);
    }

  int buf = 0;
  for (int s0 = 0; s0 < p.S; s0 += kBlock, buf ^= 1) {
    const float* cur = sc_smem + buf * stage;
    if (s0 + kBlock < p.S) {
      fetch(s0 + kBlock, sc_smem + (buf ^ 1) * stage);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
#pragma unroll 1
    for (int t0 = 0; t0 < kBlock && s0 + t0 < p.S; t0 += 8) {
      const int n = p.S - s0 - t0;
      float keep[NC];
#pragma unroll
      for (int t = 0; t < 8; ++t) {
        if (t >= n) break;
        const float* tv = cur + (t0 + t) * CP + 4 * rg;
        f2 q2[2 * RV], k2[2 * RV], g2[2 * RV];
#pragma unroll
        for (int i = 0; i < RV; ++i) {
          const ulonglong2 a = *reinterpret_cast<const ulonglong2*>(tv + 32 * i);
          const ulonglong2 c = *reinterpret_cast<const ulonglong2*>(tv + kBlock * CP + 32 * i);
          const ulonglong2 d = *reinterpret_cast<const ulonglong2*>(tv + 2 * kBlock * CP + 32 * i);
          q2[2 * i] = a.x, q2[2 * i + 1] = a.y;
          k2[2 * i] = c.x, k2[2 * i + 1] = c.y;
          g2[2 * i] = d.x, g2[2 * i + 1] = d.y;
        }
        float v[NC];
#pragma unroll
        for (int j = 0; j < NC; ++j) v[j] = cur[3 * kBlock * CP + (t0 + t) * cols + my + j];
        if constexpr (DELTA) {
          const float2 bk = *reinterpret_cast<const float2*>(cur + kBlock * (3 * CP + cols) + 2 * (t0 + t));
          float dk[NC], dq[NC];
#pragma unroll
          for (int j = 0; j < NC; ++j) {
            f2 a0 = 0, a1 = 0, b0 = 0, b1 = 0;
#pragma unroll
            for (int i = 0; i < 2 * RV; i += 2) {
              st[j][i] = mul2(st[j][i], g2[i]);
              st[j][i + 1] = mul2(st[j][i + 1], g2[i + 1]);
              a0 = fma2(st[j][i], k2[i], a0);
              a1 = fma2(st[j][i + 1], k2[i + 1], a1);
              b0 = fma2(st[j][i], q2[i], b0);
              b1 = fma2(st[j][i + 1], q2[i + 1], b1);
            }
            dk[j] = sum_f2(a0) + sum_f2(a1);
            dq[j] = sum_f2(b0) + sum_f2(b1);
          }
#pragma unroll
          for (int o = 1; o < 8; o <<= 1)
#pragma unroll
            for (int j = 0; j < NC; ++j) dk[j] += __shfl_xor_sync(0xffffffffu, dk[j], o);
#pragma unroll
          for (int j = 0; j < NC; ++j) {
            const float u = bk.x * (v[j] - dk[j]);
            const f2 u2 = pack_f2(u, u);
#pragma unroll
            for (int i = 0; i < 2 * RV; ++i) st[j][i] = fma2(k2[i], u2, st[j][i]);
            dk[j] = u;
          }
#pragma unroll
          for (int o = 1; o < 8; o <<= 1)
#pragma unroll
            for (int j = 0; j < NC; ++j) dq[j] += __shfl_xor_sync(0xffffffffu, dq[j], o);
          if (rg == t)
#pragma unroll
            for (int j = 0; j < NC; ++j) keep[j] = fmaf(dk[j], bk.y, dq[j]);
        } else {
          float dq[NC];
#pragma unroll
          for (int j = 0; j < NC; ++j) {
            const f2 v2 = pack_f2(v[j], v[j]);
            f2 b0 = 0, b1 = 0;
#pragma unroll
            for (int i = 0; i < 2 * RV; i += 2) {
              st[j][i] = fma2(st[j][i], g2[i], mul2(k2[i], v2));
              st[j][i + 1] = fma2(st[j][i + 1], g2[i + 1], mul2(k2[i + 1], v2));
              b0 = fma2(st[j][i], q2[i], b0);
              b1 = fma2(st[j][i + 1], q2[i + 1], b1);
            }
            dq[j] = sum_f2(b0) + sum_f2(b1);
          }
#pragma unroll
          for (int o = 1; o < 8; o <<= 1)
#pragma unroll
            for (int j = 0; j < NC; ++j) dq[j] += __shfl_xor_sync(0xffffffffu, dq[j], o);
          if (rg == t)
#pragma unroll
            for (int j = 0; j < NC; ++j) keep[j] = dq[j];
        }
      }
      // lane rg holds the results of token t0 + rg
      if (rg < n) {
        float* dst = p.o + ((b * p.S + s0 + t0 + rg) * p.H + h) * E + e0;
#pragma unroll
        for (int j = 0; j < NC; ++j)
          if (e0 + j < E) dst[j] = keep[j] * p.o_scale;
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int j = 0; j < NC; ++j)
#pragma unroll
    for (int i = 0; i < RV; ++i) {
      float x[4];
      unpack_f2(st[j][2 * i], x[0], x[1]);
      unpack_f2(st[j][2 * i + 1], x[2], x[3]);
#pragma unroll
      for (int r = 0; r < 4; ++r) {
        const int c = 32 * i + 4 * rg + r;
        if (c < C && e0 + j < E) st_base[static_cast<int64_t>(c) * E + e0 + j] = x[r];
      }
    }
}

template <bool DELTA, int RV, int NC>
int launch_scan(const ScanParams& p, int B, int warps, cudaStream_t st) {
  const int cols = warps * 4 * NC;
  const size_t smem = 2ull * kBlock * (3 * 32 * RV + cols + 4) * sizeof(float);
  auto kern = state_scan_kernel<DELTA, RV, NC>;
  static std::atomic<unsigned long long> attr_set{0};
  LRI_ONCE_PER_DEVICE(attr_set, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
  LRI_CUDA(launch_pdl(kern, dim3((p.E + cols - 1) / cols, p.H, B), dim3(warps * 32), smem, st, p));
  LRI_LAUNCH_CHECK("state_scan_kernel");
  return LRI_OK;
}

// Columns per lane and warps per CTA: more columns share a token's vectors, fewer leave more warps to hide latency.
template <bool DELTA, int RV>
int scan_rows(const ScanParams& p, int B, cudaStream_t st) {
  const int64_t heads = static_cast<int64_t>(B) * p.H, sms = device_sm_count();
  const int forced = option(OPT_SCAN_COLUMNS);
  int nc = RV >= 16 ? 1 : 2;
  if (RV <= 4 && heads * ((p.E + 15) / 16) >= 8 * sms) nc = 4;
  if (heads * ((p.E + 7) / 8) < sms) nc = 1;
  if (forced) nc = forced;
  if (RV >= 16) nc = 1;
  if (RV >= 8 && nc > 2) nc = 2;
  // enough CTAs to reach every SM before a CTA gets a second warp
  const int64_t warps_all = heads * ((p.E + 4 * nc - 1) / (4 * nc));
  const int warps = warps_all >= 4 * sms ? 4 : (warps_all >= 2 * sms ? 2 : 1);
  if constexpr (RV <= 4) {
    if (nc == 4) return launch_scan<DELTA, RV, 4>(p, B, warps, st);
  }
  if constexpr (RV <= 8) {
    if (nc == 2) return launch_scan<DELTA, RV, 2>(p, B, warps, st);
  }
  return launch_scan<DELTA, RV, 1>(p, B, warps, st);
}
template <bool DELTA>
int scan(const ScanParams& p, int B, cudaStream_t st) {
  if (p.C <= 32) return scan_rows<DELTA, 1>(p, B, st);
  if (p.C <= 64) return scan_rows<DELTA, 2>(p, B, st);
  if (p.C <= 128) return scan_rows<DELTA, 4>(p, B, st);
  if (p.C <= 256) return scan_rows<DELTA, 8>(p, B, st);
  return scan_rows<DELTA, 16>(p, B, st);
}

// ---- norm and gate of the results: one warp per (row, head) --------------------------------------------
template <typename T, int ACT>
__global__ void __launch_bounds__(256)
head_norm_gate_kernel(const float* o, const T* w, float eps, const float* gate, int64_t gate_ld, float scale, T* out, int64_t out_ld,
                      int64_t items, int H, int E) {
  const int lane = threadIdx.x & 31;
  pdl_launch_dependents();
  pdl_wait();
  const int64_t item = static_cast<int64_t>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  if (item >= items) return;
  const int64_t row = item / H;
  const int h = static_cast<int>(item - row * H);
  const float* x = o + item * E;
  const float* gt = gate + row * gate_ld + static_cast<int64_t>(h) * E;
  T* dst = out + row * out_ld + static_cast<int64_t>(h) * E;
  float ss = 0.f;
  for (int e = lane; e < E; e += 32) ss = fmaf(x[e], x[e], ss);
  const float inv = scale / sqrtf(warp_sum(ss) / static_cast<float>(E) + eps);
  for (int e = lane; e < E; e += 32) {
    const float a = ACT == 0 ? sigmoid_f(gt[e]) : silu_f(gt[e]);
    dst[e] = Num<T>::from_f(x[e] * inv * Num<T>::to_f(w[e]) * a);
  }
}

template <typename T>
int head_norm_gate(const float* o, const void* w, float eps, const float* gate, int64_t gate_ld, int act, float scale, void* out,
                   int64_t out_ld, int64_t rows, int H, int E, cudaStream_t st) {
  const int64_t items = rows * H;
  auto kern = act == 0 ? head_norm_gate_kernel<T, 0> : head_norm_gate_kernel<T, 1>;
  LRI_CUDA(launch_pdl(kern, dim3(static_cast<unsigned>((items + 7) / 8)), dim3(256), 0, st, o, static_cast<const T*>(w), eps, gate, gate_ld,
                      scale, static_cast<T*>(out), out_ld, items, H, E));
  LRI_LAUNCH_CHECK("head_norm_gate_kernel");
  return LRI_OK;
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

bool dtype_ok(int dtype) { return dtype >= LRI_BF16 && dtype <= LRI_FP32; }

constexpr int kMaxChannels = 512;

}  // namespace
}  // namespace lri

using namespace lri;

#define LRI_BY_TYPE(dtype, call) ((dtype) == LRI_BF16 ? call<__nv_bfloat16> : (dtype) == LRI_FP16 ? call<__half> : call<float>)

extern "C" int lri_delta_prepare(int dtype, const float* proj, int64_t ld, int64_t q_off, int64_t k_off, int64_t v_off, int64_t b_off,
                                 const void* conv_q, const void* conv_k, const void* conv_v, int taps, float* ring, float* z,
                                 const void* a_log, const void* dt_bias, const void* input_pos, int pos_is_i64, float* q, float* k,
                                 float* v, float* beta, float* kq, int B, int S, int heads, int kv_heads, int dim, int vdim,
                                 lri_stream_t stream) {
  LRI_REQUIRE(dtype_ok(dtype), LRI_ERR_UNSUPPORTED, "delta_prepare: dtype %d", dtype);
  LRI_REQUIRE(proj && conv_q && conv_k && conv_v && ring && z && a_log && dt_bias && input_pos && q && k && v && beta && kq, LRI_ERR_ARG,
              "delta_prepare: NULL pointer");
  LRI_REQUIRE(B >= 0 && B <= 65535 && S >= 0 && heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && dim > 0 && vdim > 0, LRI_ERR_ARG,
              "delta_prepare: B=%d S=%d heads=%d kv_heads=%d dim=%d vdim=%d", B, S, heads, kv_heads, dim, vdim);
  LRI_REQUIRE(taps >= 1 && taps <= kMaxTaps, LRI_ERR_UNSUPPORTED, "delta_prepare: taps=%d outside 1..%d", taps, kMaxTaps);
  const int64_t rows = static_cast<int64_t>(B) * S;
  if (rows == 0) return LRI_OK;
  DeltaPrepareParams p{};
  p.proj = proj, p.ld = ld, p.q_off = q_off, p.k_off = k_off, p.v_off = v_off, p.b_off = b_off;
  p.conv_q = conv_q, p.conv_k = conv_k, p.conv_v = conv_v, p.taps = taps, p.ring = ring, p.z = z, p.a_log = a_log, p.dt_bias = dt_bias;
  p.input_pos = input_pos, p.pos_is_i64 = pos_is_i64, p.q = q, p.k = k, p.v = v, p.beta = beta, p.kq = kq;
  p.S = S, p.H = heads, p.G = kv_heads, p.C = dim, p.E = vdim;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  LRI_CUDA(launch_pdl(LRI_BY_TYPE(dtype, delta_prepare_kernel), dim3(static_cast<unsigned>(rows), (heads + kv_heads + 7) / 8), dim3(256), 0,
                      st, p));
  LRI_LAUNCH_CHECK("delta_prepare_kernel");
  const int nqk = kv_heads * dim, nv = heads * vdim;
  LRI_CUDA(launch_pdl(conv_ring_kernel, dim3((2 * nqk + nv + 255) / 256, taps < S ? taps : S, B), dim3(256), 0, st, proj, ld, q_off, k_off,
                      v_off, nqk, nv, ring, taps, input_pos, pos_is_i64, S));
  LRI_LAUNCH_CHECK("conv_ring_kernel");
  return LRI_OK;
}

extern "C" int lri_logistic_decay(int dtype, float* z, const void* bias, float tau, int64_t rows, int width, lri_stream_t stream) {
  LRI_REQUIRE(dtype_ok(dtype), LRI_ERR_UNSUPPORTED, "logistic_decay: dtype %d", dtype);
  LRI_REQUIRE(z && bias && tau > 0.f && rows >= 0 && width > 0, LRI_ERR_ARG, "logistic_decay: rows=%lld width=%d tau=%g", (long long)rows,
              width, tau);
  const int64_t n = rows * width;
  if (n == 0) return LRI_OK;
  const unsigned grid = static_cast<unsigned>((n + 255) / 256);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
#define LRI_CALL(T) \
  LRI_CUDA(launch_pdl(logistic_decay_kernel<T>, dim3(grid), dim3(256), 0, st, z, static_cast<const T*>(bias), 1.0f / tau, n, width))
  if (dtype == LRI_BF16)
    LRI_CALL(__nv_bfloat16);
  else if (dtype == LRI_FP16)
    LRI_CALL(__half);
  else
    LRI_CALL(float);
#undef LRI_CALL
  LRI_LAUNCH_CHECK("logistic_decay_kernel");
  return LRI_OK;
}

extern "C" int lri_state_scan(const float* q, int64_t q_row, const float* k, int64_t k_row, const float* v, int64_t v_row,
                              const float* decay, const float* beta, const float* kq, float* state, const void* input_pos,
                              int pos_is_i64, float* o, float o_scale, int B, int S, int heads, int kv_heads, int dim, int vdim,
                              lri_stream_t stream) {
  LRI_REQUIRE(q && k && v && decay && state && input_pos && o, LRI_ERR_ARG, "state_scan: NULL pointer");
  LRI_REQUIRE((beta == nullptr) == (kq == nullptr), LRI_ERR_ARG, "state_scan: beta and kq go together");
  LRI_REQUIRE(B >= 0 && B <= 65535 && S >= 0 && heads > 0 && heads <= 65535 && kv_heads > 0 && heads % kv_heads == 0 && dim > 0 && vdim > 0,
              LRI_ERR_ARG, "state_scan: B=%d S=%d heads=%d kv_heads=%d dim=%d vdim=%d", B, S, heads, kv_heads, dim, vdim);
  LRI_REQUIRE(dim <= kMaxChannels, LRI_ERR_UNSUPPORTED, "state_scan: dim=%d > %d", dim, kMaxChannels);
  if (B == 0 || S == 0) return LRI_OK;
  ScanParams p{};
  p.q = q, p.k = k, p.v = v, p.g = decay, p.q_row = q_row, p.k_row = k_row, p.v_row = v_row, p.beta = beta, p.kq = kq;
  p.state = state, p.input_pos = input_pos, p.pos_is_i64 = pos_is_i64, p.o = o, p.o_scale = o_scale;
  p.S = S, p.H = heads, p.group = heads / kv_heads, p.C = dim, p.E = vdim;
  p.vec = dim % 4 == 0 && vdim % 4 == 0 && q_row % 4 == 0 && k_row % 4 == 0 && v_row % 4 == 0 && aligned16(q) && aligned16(k) &&
          aligned16(v) && aligned16(decay);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return beta ? scan<true>(p, B, st) : scan<false>(p, B, st);
}

extern "C" int lri_head_norm_gate(int dtype, const float* o, const void* norm_weight, float eps, const float* gate, int64_t gate_ld,
                                  int activation, float scale, void* out, int64_t out_ld, int64_t rows, int heads, int vdim,
                                  lri_stream_t stream) {
  LRI_REQUIRE(dtype_ok(dtype), LRI_ERR_UNSUPPORTED, "head_norm_gate: dtype %d", dtype);
  LRI_REQUIRE(o && norm_weight && gate && out, LRI_ERR_ARG, "head_norm_gate: NULL pointer");
  LRI_REQUIRE(activation == LRI_GATE_SIGMOID || activation == LRI_GATE_SILU, LRI_ERR_ARG, "head_norm_gate: activation %d", activation);
  LRI_REQUIRE(rows >= 0 && heads > 0 && vdim > 0, LRI_ERR_ARG, "head_norm_gate: rows=%lld heads=%d vdim=%d", (long long)rows, heads, vdim);
  if (rows == 0) return LRI_OK;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return LRI_BY_TYPE(dtype, head_norm_gate)(o, norm_weight, eps, gate, gate_ld, activation, scale, out, out_ld, rows, heads, vdim, st);
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
