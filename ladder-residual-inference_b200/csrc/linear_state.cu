// Matrix-state recurrences over the tokens of a call, in blocks of four (linear_state.cuh), and the norm and gate of
// their results.
//
// The columns of a state (value channels) do not depend on one another: u, o and the update of column e use only that
// column.  So the scan needs no barrier between tokens: a warp owns a few columns, its lanes split the rows of S (8 or 16 lanes
// a column).  Rows stay in registers over the whole call, as pairs for the packed fp32 instructions; block vectors and
// coefficients arrive in shared memory by TMA, 16 tokens a stage.  Waits for copies are bounded; on expiry a status word is
// set and the kernel returns.
#include "linear_state.cuh"
#include "tcgen05.cuh"

namespace lri {
namespace {

struct ScanParams {
  const float *qd, *kd, *ku;  // [B * blocks * 4, H, C]; kd NULL: gated linear attention
  const float* decay;         // [B * blocks, H, C]
  const float* coef;          // [B * blocks, H, 32]
  const float* v;             // v + row * v_row + head * E
  int64_t v_row;
  float* state;  // [B_max, H, C, E]
  const void* input_pos;
  int pos_is_i64;
  float* o;  // [rows, H, E]
  int S, H, C, E;
  int tma;  // the tensor maps below are valid
};
// [rows, heads, width] views
struct ScanMaps {
  CUtensorMap qd, kd, ku, decay, coef, v;
};

constexpr int kT = kStateBlock;
constexpr int kBlock = 16;  // tokens of a stage
constexpr int kSub = kBlock / kT;
// LN: lanes that share a column; RV: 4-row pieces of it per lane (4 LN RV rows in all)
template <bool DELTA, int LN, int RV>
struct ScanLayout {
  static constexpr int CP = 4 * LN * RV;
  static constexpr int kStages = CP > 256 ? 2 : 3;
  static constexpr int kQd = 0, kKu = kBlock * CP, kKd = 2 * kBlock * CP;
  static constexpr int kDecay = (DELTA ? 3 : 2) * kBlock * CP;
  static constexpr int kCf = kDecay + kSub * CP;
  static constexpr int kV = kCf + kSub * kCoef;  // [kBlock][columns of the CTA]
  static int floats(int cols) { return kStages * (kV + kBlock * cols); }
};

__device__ int g_scan_status = 0;

// NC: columns per lane (32 / LN * NC a warp)
template <bool DELTA, int LN, int RV, int NC>
__global__ void __launch_bounds__(128, 1) state_scan_kernel(const __grid_constant__ ScanMaps maps, const ScanParams p) {
  using L = ScanLayout<DELTA, LN, RV>;
  constexpr int CP = L::CP, kStages = L::kStages, kWarpCols = 32 / LN * NC;
  extern __shared__ __align__(1024) float sc_smem[];
  __shared__ uint64_t bars[kStages];
  __shared__ int abort_flag;
  const int warps = blockDim.x >> 5, cols = warps * kWarpCols;
  const int stage = L::kV + kBlock * cols;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, rg = lane % LN, cl = lane / LN;
  const int h = blockIdx.y, H = p.H, C = p.C, E = p.E;
  const int64_t b = blockIdx.z;
  const int col0 = blockIdx.x * cols, my = warp * kWarpCols + cl * NC, e0 = col0 + my;
  float* st_base = p.state + (b * H + h) * static_cast<int64_t>(C) * E;
  if (!p.tma)  // rows and columns past the end stay zero (the tensor maps fill them)
    for (int i = tid; i < kStages * stage; i += blockDim.x) sc_smem[i] = 0.f;
  if (tid == 0) {
    abort_flag = 0;
    for (int i = 0; i < kStages; ++i) tc::mbar_init(tc::smem_u32(&bars[i]), 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  }
  pdl_launch_dependents();
  __syncthreads();
  pdl_wait();

  const int seq_blocks = (p.S + kT - 1) / kT, stages = (p.S + kBlock - 1) / kBlock;
  const int64_t first_block = b * seq_blocks;
  auto fetch = [&](int i) {
    if (i >= stages) return;
    float* dst = sc_smem + (i % kStages) * stage;
    const int64_t blk = first_block + i * kSub, row = b * p.S + i * kBlock;
    if (p.tma) {
      if (tid != 0) return;
      // whole boxes: what lies past a vector's end reads as zero, blocks past the sequence's end are not used
      const uint32_t bar = tc::smem_u32(&bars[i % kStages]), base = tc::smem_u32(dst);
      const int y = static_cast<int>(blk);
      tc::mbar_expect_tx(bar, stage * 4);
      tc::tma_load_3d(base + L::kQd * 4, &maps.qd, bar, 0, h, y * kT);
      if (DELTA) tc::tma_load_3d(base + L::kKd * 4, &maps.kd, bar, 0, h, y * kT);
      tc::tma_load_3d(base + L::kKu * 4, &maps.ku, bar, 0, h, y * kT);
      tc::tma_load_3d(base + L::kDecay * 4, &maps.decay, bar, 0, h, y);
      tc::tma_load_3d(base + L::kCf * 4, &maps.coef, bar, 0, h, y);
      tc::tma_load_3d(base + L::kV * 4, &maps.v, bar, col0, h, static_cast<int>(row));
      return;
    }
    const int n = p.S - i * kBlock < kBlock ? p.S - i * kBlock : kBlock, nb = (n + kT - 1) / kT;
    for (int t = warp; t < nb * kT; t += warps) {
      const int64_t at = ((blk * kT + t) * H + h) * C;
      for (int c = lane; c < C; c += 32) {
        dst[L::kQd + t * CP + c] = p.qd[at + c];
        dst[L::kKu + t * CP + c] = p.ku[at + c];
        if (DELTA) dst[L::kKd + t * CP + c] = p.kd[at + c];
      }
      for (int e = lane; e < cols; e += 32)
        dst[L::kV + t * cols + e] = t < n && col0 + e < E ? p.v[(row + t) * p.v_row + h * E + col0 + e] : 0.f;
    }
    for (int j = warp; j < nb; j += warps) {
      for (int c = lane; c < C; c += 32) dst[L::kDecay + j * CP + c] = p.decay[((blk + j) * H + h) * C + c];
      dst[L::kCf + j * kCoef + lane] = p.coef[((blk + j) * H + h) * kCoef + lane];
    }
  };
  for (int i = 0; i < kStages - 1; ++i) fetch(i);

  // rows of this lane: 4 LN i + 4 rg + 0 .. 3
  f2 st[NC][2 * RV];
  const bool fresh = load_pos(p.input_pos, p.pos_is_i64, 0) <= 0;
#pragma unroll
  for (int j = 0; j < NC; ++j)
#pragma unroll
    for (int i = 0; i < RV; ++i) {
      float x[4];
#pragma unroll
      for (int r = 0; r < 4; ++r) {
        const int c = 4 * LN * i + 4 * rg + r;
        x[r] = !fresh && c < C && e0 + j < E ? st_base[static_cast<int64_t>(c) * E + e0 + j] : 0.f;
      }
      st[j][2 * i] = pack_f2(x[0], x[1]);
      st[j][2 * i + 1] = pack_f2(x[2], x[3]);
    }

  auto load_rows = [&](const float* v, f2 (&x)[2 * RV]) {
#pragma unroll
    for (int i = 0; i < RV; ++i) {
      const ulonglong2 a = *reinterpret_cast<const ulonglong2*>(v + 4 * LN * i + 4 * rg);
      x[2 * i] = a.x, x[2 * i + 1] = a.y;
    }
  };
  // column j of the state times a vector: this lane's share
  auto dot = [&](const f2 (&s)[2 * RV], const f2 (&x)[2 * RV]) {
    f2 a0 = mul2(s[0], x[0]), a1 = mul2(s[1], x[1]);
#pragma unroll
    for (int i = 2; i < 2 * RV; i += 2) a0 = fma2(s[i], x[i], a0), a1 = fma2(s[i + 1], x[i + 1], a1);
    return sum_f2(add2(a0, a1));
  };
  // results: lane rg keeps token rg / kPerToken of the block number rg % kPerToken of a pair
  constexpr int kPerToken = LN / kT;
  const int my_t = rg / kPerToken, my_block = rg % kPerToken;
  float keep[NC];
  auto block = [&](const float* cur, int sub, int nth) {
    const float* cf = cur + L::kCf + sub * kCoef;
    float d[kT][NC], dq[kT][NC], u[kT][NC];
#pragma unroll
    for (int t = 0; t < kT; ++t) {
      f2 x[2 * RV];
      if constexpr (DELTA) {
        load_rows(cur + L::kKd + (sub * kT + t) * CP, x);
#pragma unroll
        for (int j = 0; j < NC; ++j) d[t][j] = dot(st[j], x);
      }
      load_rows(cur + L::kQd + (sub * kT + t) * CP, x);
#pragma unroll
      for (int j = 0; j < NC; ++j) dq[t][j] = dot(st[j], x);
#pragma unroll
      for (int j = 0; j < NC; ++j) u[t][j] = cur[L::kV + (sub * kT + t) * cols + my + j];
    }
    if constexpr (DELTA) {
#pragma unroll
      for (int o = 1; o < LN; o <<= 1)
#pragma unroll
        for (int t = 0; t < kT; ++t)
#pragma unroll
          for (int j = 0; j < NC; ++j) d[t][j] += __shfl_xor_sync(0xffffffffu, d[t][j], o);
#pragma unroll
      for (int t = 0; t < kT; ++t)
#pragma unroll
        for (int j = 0; j < NC; ++j) {
          float x = u[t][j] - d[t][j];
#pragma unroll
          for (int s = 0; s < t; ++s) x = fmaf(-cf[kCoefA + t * (t - 1) / 2 + s], u[s][j], x);
          u[t][j] = cf[t] * x;
        }
    }
    {
      f2 x[2 * RV];
      load_rows(cur + L::kDecay + sub * CP, x);
#pragma unroll
      for (int j = 0; j < NC; ++j)
#pragma unroll
        for (int i = 0; i < 2 * RV; ++i) st[j][i] = mul2(st[j][i], x[i]);
    }
#pragma unroll
    for (int t = 0; t < kT; ++t) {
      f2 x[2 * RV];
      load_rows(cur + L::kKu + (sub * kT + t) * CP, x);
#pragma unroll
      for (int j = 0; j < NC; ++j) {
        const f2 u2 = pack_f2(u[t][j], u[t][j]);
#pragma unroll
        for (int i = 0; i < 2 * RV; ++i) st[j][i] = fma2(x[i], u2, st[j][i]);
      }
    }
    // sums of dq: each of the first two exchanges halves the tokens a lane holds
    const float4 bt = *reinterpret_cast<const float4*>(cf + kCoefB + kT * my_t);
#pragma unroll
    for (int j = 0; j < NC; ++j) {
      const bool up = rg & (LN / 2), up2 = rg & (LN / 4);
      const float x0 = (up ? dq[2][j] : dq[0][j]) + __shfl_xor_sync(0xffffffffu, up ? dq[0][j] : dq[2][j], LN / 2);
      const float x1 = (up ? dq[3][j] : dq[1][j]) + __shfl_xor_sync(0xffffffffu, up ? dq[1][j] : dq[3][j], LN / 2);
      float x = (up2 ? x1 : x0) + __shfl_xor_sync(0xffffffffu, up2 ? x0 : x1, LN / 4);
#pragma unroll
      for (int o = LN / 8; o >= 1; o >>= 1) x += __shfl_xor_sync(0xffffffffu, x, o);
      x = fmaf(bt.x, u[0][j], x), x = fmaf(bt.y, u[1][j], x), x = fmaf(bt.z, u[2][j], x), x = fmaf(bt.w, u[3][j], x);
      keep[j] = my_block == nth ? x : keep[j];
    }
  };

  bool ok = true;
  for (int i = 0; i < stages; ++i) {
    const float* cur = sc_smem + (i % kStages) * stage;
    if (p.tma) ok = tc::mbar_wait(tc::smem_u32(&bars[i % kStages]), (i / kStages) & 1, &abort_flag, 1, &g_scan_status);
    // every warp is done with the stage before this one, which the next copies overwrite
    if (!__syncthreads_and(ok)) {
      ok = false;
      break;
    }
    fetch(i + kStages - 1);
#pragma unroll 1
    for (int t0 = 0; t0 < kBlock && i * kBlock + t0 < p.S; t0 += 2 * kT) {
      const int n = p.S - i * kBlock - t0;
#pragma unroll
      for (int j = 0; j < NC; ++j) keep[j] = 0.f;
      if (n > kT) {  // straight on: the second block's sums start while the first one's results are reduced
        block(cur, t0 / kT, 0);
        block(cur, t0 / kT + 1, 1);
      } else {
        block(cur, t0 / kT, 0);
      }
      const int mine = my_block * kT + my_t;  // token whose results this lane holds
      if (my_block < 2 && mine < n) {
        float* dst = p.o + ((b * p.S + i * kBlock + t0 + mine) * H + h) * E + e0;
#pragma unroll
        for (int j = 0; j < NC; ++j)
          if (e0 + j < E) dst[j] = keep[j];
      }
    }
  }
  if (!ok) {  // a bounded wait gave up: let copies that were issued land before the shared memory is released
    for (int i = 0; i < 2000; ++i) __nanosleep(100);
    return;
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
        const int c = 4 * LN * i + 4 * rg + r;
        if (c < C && e0 + j < E) st_base[static_cast<int64_t>(c) * E + e0 + j] = x[r];
      }
    }
}

template <bool DELTA, int LN, int RV, int NC>
int launch_scan(const ScanParams& p, int B, int warps, cudaStream_t st) {
  using L = ScanLayout<DELTA, LN, RV>;
  const int cols = warps * (32 / LN) * NC;
  const size_t smem = static_cast<size_t>(L::floats(cols)) * sizeof(float);
  auto kern = state_scan_kernel<DELTA, LN, RV, NC>;
  static std::atomic<unsigned long long> attr_set{0};
  LRI_ONCE_PER_DEVICE(attr_set, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 222 * 1024));
  ScanParams sp = p;
  ScanMaps maps{};
  sp.tma = p.tma && L::CP <= 256;
  if (sp.tma) {
    const int64_t blocks = static_cast<int64_t>(B) * ((p.S + kT - 1) / kT), hc = static_cast<int64_t>(p.H) * p.C;
    int rc = make_tmap_f32(&maps.qd, p.qd, blocks * kT, hc, p.H, p.C, p.C, L::CP, kBlock);
    if (rc == LRI_OK && DELTA) rc = make_tmap_f32(&maps.kd, p.kd, blocks * kT, hc, p.H, p.C, p.C, L::CP, kBlock);
    if (rc == LRI_OK) rc = make_tmap_f32(&maps.ku, p.ku, blocks * kT, hc, p.H, p.C, p.C, L::CP, kBlock);
    if (rc == LRI_OK) rc = make_tmap_f32(&maps.decay, p.decay, blocks, hc, p.H, p.C, p.C, L::CP, kSub);
    if (rc == LRI_OK) rc = make_tmap_f32(&maps.coef, p.coef, blocks, static_cast<int64_t>(p.H) * kCoef, p.H, kCoef, kCoef, kCoef, kSub);
    if (rc == LRI_OK) rc = make_tmap_f32(&maps.v, p.v, static_cast<int64_t>(B) * p.S, p.v_row, p.H, p.E, p.E, cols, kBlock);
    if (rc != LRI_OK) return rc;
  }
  LRI_CUDA(launch_pdl(kern, dim3((p.E + cols - 1) / cols, p.H, B), dim3(warps * 32), smem, st, maps, sp));
  LRI_LAUNCH_CHECK("state_scan_kernel");
  return LRI_OK;
}

// Columns per lane and warps per CTA: more columns share a block's vectors, fewer leave more warps to hide latency.
template <bool DELTA, int LN, int RV>
int scan_shape(const ScanParams& p, int B, cudaStream_t st) {
  constexpr int kMaxCols = RV * LN > 64 ? 1 : (RV * LN > 32 ? 2 : 4);  // state registers of a lane
  const int64_t heads = static_cast<int64_t>(B) * p.H, sms = device_sm_count();
  auto warps_of = [&](int nc) { return heads * ((p.E + 32 / LN * nc - 1) / (32 / LN * nc)); };
  int nc = 2;
  if (warps_of(4) >= 4 * sms) nc = 4;
  if (warps_of(1) < 2 * sms) nc = 1;
  if (option(OPT_SCAN_COLUMNS)) nc = option(OPT_SCAN_COLUMNS);
  nc = nc > kMaxCols ? kMaxCols : nc;
  // enough CTAs to reach every SM before a CTA gets a second warp
  int warps = warps_of(nc) >= 4 * sms ? 4 : (warps_of(nc) >= 2 * sms ? 2 : 1);
  if (option(OPT_SCAN_WARPS)) warps = option(OPT_SCAN_WARPS);
  if (32 / LN * nc * warps < 4) warps = 2;  // a box of values is at least 16 bytes wide
  if constexpr (kMaxCols >= 4) {
    if (nc == 4) return launch_scan<DELTA, LN, RV, 4>(p, B, warps, st);
  }
  if constexpr (kMaxCols >= 2) {
    if (nc == 2) return launch_scan<DELTA, LN, RV, 2>(p, B, warps, st);
  }
  return launch_scan<DELTA, LN, RV, 1>(p, B, LN * RV > 64 ? 2 : warps, st);  // (long columns leave room for few)
}
template <bool DELTA>
int scan(const ScanParams& p, int B, cudaStream_t st) {
  // few columns: more lanes a column
  const bool wide = option(OPT_SCAN_LANES) ? option(OPT_SCAN_LANES) == 16
                                           : DELTA && p.C > 64 && static_cast<int64_t>(B) * p.H * p.E <= 14ll * device_sm_count();
  if (p.C <= 32) return scan_shape<DELTA, 8, 1>(p, B, st);
  if (p.C <= 64) return wide ? scan_shape<DELTA, 16, 1>(p, B, st) : scan_shape<DELTA, 8, 2>(p, B, st);
  if (p.C <= 128) return wide ? scan_shape<DELTA, 16, 2>(p, B, st) : scan_shape<DELTA, 8, 4>(p, B, st);
  if (p.C <= 256) return scan_shape<DELTA, 16, 4>(p, B, st);
  return scan_shape<DELTA, 16, 8>(p, B, st);
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

bool dtype_ok(int dtype) { return dtype >= LRI_BF16 && dtype <= LRI_FP32; }

constexpr int kMaxChannels = 512;

}  // namespace

int state_scan_status_read_and_clear(int* status_out) {
  int v = 0;
  LRI_CUDA(cudaMemcpyFromSymbol(&v, g_scan_status, sizeof(int)));
  if (v != 0) {
    int zero = 0;
    LRI_CUDA(cudaMemcpyToSymbol(g_scan_status, &zero, sizeof(int)));
  }
  *status_out = v;
  return LRI_OK;
}

}  // namespace lri

using namespace lri;

#define LRI_BY_TYPE(dtype, call) ((dtype) == LRI_BF16 ? call<__nv_bfloat16> : (dtype) == LRI_FP16 ? call<__half> : call<float>)

extern "C" int lri_state_scan(const float* qd, const float* kd, const float* ku, const float* decay, const float* coef, const float* v,
                              int64_t v_row, float* state, const void* input_pos, int pos_is_i64, float* o, int B, int S, int heads,
                              int dim, int vdim, lri_stream_t stream) {
  LRI_REQUIRE(qd && ku && decay && coef && v && state && input_pos && o, LRI_ERR_ARG, "state_scan: NULL pointer");
  LRI_REQUIRE(B >= 0 && B <= 65535 && S >= 0 && heads > 0 && heads <= 65535 && dim > 0 && vdim > 0, LRI_ERR_ARG,
              "state_scan: B=%d S=%d heads=%d dim=%d vdim=%d", B, S, heads, dim, vdim);
  LRI_REQUIRE(dim <= kMaxChannels, LRI_ERR_UNSUPPORTED, "state_scan: dim=%d > %d", dim, kMaxChannels);
  if (B == 0 || S == 0) return LRI_OK;
  ScanParams p{};
  p.qd = qd, p.kd = kd, p.ku = ku, p.decay = decay, p.coef = coef, p.v = v, p.v_row = v_row;
  p.state = state, p.input_pos = input_pos, p.pos_is_i64 = pos_is_i64, p.o = o;
  p.S = S, p.H = heads, p.C = dim, p.E = vdim;
  p.tma = static_cast<int64_t>(B) * (S + 2 * kBlock) < (1ll << 31) && dim % 4 == 0 && vdim % 4 == 0 && v_row % 4 == 0 && aligned16(qd) &&
          aligned16(kd) && aligned16(ku) && aligned16(decay) && aligned16(coef) && aligned16(v);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return kd ? scan<true>(p, B, st) : scan<false>(p, B, st);
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

