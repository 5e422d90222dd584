// Masked prompt attention (sliding window, chunks) with keys in two parts (per key head, and one shared by the heads) on
// tcgen05.
//
// A CTA owns 256 consecutive queries of one (sequence, head) as two groups of 128, and walks the key tiles of 64 that
// any of them sees; both groups use a tile while it is in shared memory.  Per group and tile:
//   S = Q1 K1^T + Q2 K2^T   tcgen05.mma 128 x 64, one accumulation over the chunks of both parts, S in one of the group's
//                           two TMEM buffers
//   softmax                 4 warps, thread i owns query row i (one TMEM lane): scale, window mask, exp2 against the
//                           running reference maximum, P written over S in the storage type
//   O += P V                P from TMEM as the A operand, V MN-major from shared memory, O in TMEM
// O is rescaled only when a row's maximum grows by more than 2^8.  Widths are cut in chunks of 64 elements; a tail
// chunk is filled with zeros by the tensor maps, which view every operand as [rows, heads, width].  A row of a group
// may see nothing of the group's first tiles (short windows): its maximum is then still -inf and P is zero.
// Keys are rows gathered for the call (row j = position pos0 - history + j) or rows of a cache (row = position; C2 = 0,
// key heads shared by groups of query heads).  A sink adds exp(sink) to a row's sum at the end.
// Every mbarrier wait is bounded; on expiry a status word is set, TMEM is freed and the kernel returns.
#include "latent_attention.cuh"
#include "tcgen05.cuh"

namespace lri {
namespace {

using namespace tc;

constexpr int kRows = 128;  // queries of a group
constexpr int kKeys = 64;   // keys of a tile
constexpr int kGroups = 2;
constexpr int kThreads = 64 + kGroups * 128;
constexpr float kRescaleLog2 = 8.0f;

__device__ int g_window_tc_status = 0;

struct TcParams {
  void* out;
  const void* input_pos;
  int pos_is_i64;
  int S, H, dv, group;
  int history, k_rows, window, chunk;
  int64_t batch_rows, batch_heads;  // offsets of a sequence's keys in rows and in heads of the tensor maps
  const void* sink;
  int64_t out_ld;
  float scale_log2, out_scale;
};

struct Tiles {
  int lo, n;  // first key tile and number of tiles
};

// First key row seen from key row j (rows below j_min do not exist; chunks need row = position)
__device__ __forceinline__ int first_row(const TcParams& p, int j, int j_min) {
  int lo = j - p.window + 1;
  lo = lo > j_min ? lo : j_min;
  if (p.chunk > 0) {
    const int c = j / p.chunk * p.chunk;
    lo = lo > c ? lo : c;
  }
  return lo;
}
// Tiles seen by queries q0 .. q_end - 1 (key row of query i is history + i)
__device__ __forceinline__ Tiles tiles_of_queries(const TcParams& p, int history, int q0, int q_end, int j_min) {
  Tiles t;
  t.lo = first_row(p, history + q0, j_min) / kKeys;
  t.n = (history + q_end - 1) / kKeys - t.lo + 1;
  return t;
}

// C1, C2, CV: 64-element chunks of the per-head key part, the shared key part and the value
template <typename T, int C1, int C2, int CV>
struct Sizes {
  static constexpr int kQk = C1 + C2;
  static constexpr uint32_t kQBytes = kQk * kRows * 128;  // one group
  static constexpr uint32_t kStage = (kQk + CV) * kKeys * 128;
  static constexpr int kFit = static_cast<int>((226u * 1024u - 1024u - kGroups * kQBytes) / kStage);
  static constexpr int kStages = kFit > 4 ? 4 : kFit;
  static constexpr int kSmem = kGroups * kQBytes + kStages * kStage + 1024;
  static_assert(kStages >= 2, "two key tiles must fit");
};

template <typename T, int C1, int C2, int CV>
__global__ void __launch_bounds__(kThreads, 1)
window_attention_tc_kernel(const __grid_constant__ CUtensorMap tq1, const __grid_constant__ CUtensorMap tq2,
                           const __grid_constant__ CUtensorMap tk1, const __grid_constant__ CUtensorMap tk2,
                           const __grid_constant__ CUtensorMap tv, const TcParams p) {
  using Z = Sizes<T, C1, C2, CV>;
  constexpr int kQk = Z::kQk, kStages = Z::kStages;
  constexpr uint32_t kQChunk = kRows * 128, kKvChunk = kKeys * 128;
  constexpr uint32_t kGroupCols = 2 * kKeys + CV * 64;  // two S buffers and O
  constexpr uint32_t kTmemCols = 512;

  extern __shared__ uint8_t wtc_smem[];
  const uint32_t base = (smem_u32(wtc_smem) + 1023u) & ~1023u;
  const uint32_t kv_smem = base + kGroups * Z::kQBytes;
  __shared__ uint64_t bars[1 + 2 * kStages + 6 * kGroups];
  __shared__ uint32_t tmem_base_slot;
  __shared__ int abort_flag;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int q_tile = gridDim.x - 1 - blockIdx.x;  // long (late) tiles first
  const int q0 = q_tile * kRows * kGroups;
  const int head = blockIdx.y, b = blockIdx.z;

  const uint32_t q_full = smem_u32(&bars[0]);
  const uint32_t kv_full0 = smem_u32(&bars[1]);
  const uint32_t kv_empty0 = smem_u32(&bars[1 + kStages]);
  auto s_full = [&](int g, int i) { return smem_u32(&bars[1 + 2 * kStages + g * 6 + i]); };      // S ready
  auto p_full = [&](int g, int i) { return smem_u32(&bars[1 + 2 * kStages + g * 6 + 2 + i]); };  // P ready
  auto o_done = [&](int g, int i) { return smem_u32(&bars[1 + 2 * kStages + g * 6 + 4 + i]); };  // O holds the tile

  if (threadIdx.x == 0) {
    abort_flag = 0;
    mbar_init(q_full, 1);
    for (int s = 0; s < kStages; ++s) {
      mbar_init(kv_full0 + 8 * s, 1);
      mbar_init(kv_empty0 + 8 * s, 1);
    }
    for (int g = 0; g < kGroups; ++g)
      for (int i = 0; i < 2; ++i) {
        mbar_init(s_full(g, i), 1);
        mbar_init(p_full(g, i), 128);
        mbar_init(o_done(g, i), 1);
      }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_base_slot)),
                 "r"(kTmemCols)
                 : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
  const uint32_t tmem_base = tmem_base_slot;
  pdl_wait();
  pdl_launch_dependents();

  int64_t pos0 = load_pos(p.input_pos, p.pos_is_i64, 0);
  pos0 = pos0 < 0 ? 0 : pos0;
  const int history = p.history < 0 ? static_cast<int>(pos0) : p.history;  // key row of the first query
  const int j_min = pos0 < history ? history - static_cast<int>(pos0) : 0;  // key row of position 0
  Tiles gt[kGroups], all;
  int groups = 0;
#pragma unroll
  for (int g = 0; g < kGroups; ++g) {
    const int a = q0 + g * kRows;
    const int e = a + kRows < p.S ? a + kRows : p.S;
    gt[g] = Tiles{0, 0};
    if (a < p.S) {
      gt[g] = tiles_of_queries(p, history, a, e, j_min);
      groups = g + 1;
    }
  }
  all.lo = gt[0].lo;
  all.n = gt[groups - 1].lo + gt[groups - 1].n - all.lo;  // the groups' ranges overlap or follow one another
  auto active = [&](int g, int t) { return t >= gt[g].lo && t < gt[g].lo + gt[g].n; };

  if (warp == 0) {
    if (lane == 0) {
      mbar_expect_tx(q_full, kGroups * Z::kQBytes);
#pragma unroll
      for (int g = 0; g < kGroups; ++g) {
        // rows past the end of the tensor read as zero; the second group's box may start there
        const int row = b * p.S + q0 + g * kRows;
#pragma unroll
        for (int c = 0; c < C1; ++c) tma_load_3d(base + g * Z::kQBytes + c * kQChunk, &tq1, q_full, c * 64, head, row);
#pragma unroll
        for (int c = 0; c < C2; ++c)
          tma_load_3d(base + g * Z::kQBytes + (C1 + c) * kQChunk, &tq2, q_full, c * 64, head, row);
      }
      for (int j = 0; j < all.n; ++j) {
        const uint32_t s = j % kStages, round = j / kStages;
        if (!mbar_wait(kv_empty0 + 8 * s, (round & 1u) ^ 1u, &abort_flag, 1, &g_window_tc_status)) break;
        mbar_expect_tx(kv_full0 + 8 * s, Z::kStage);
        const uint32_t dst = kv_smem + s * Z::kStage;
        const int row = static_cast<int>(b * p.batch_rows) + (all.lo + j) * kKeys;
        const int kv_head = static_cast<int>(b * p.batch_heads) + head / p.group;
#pragma unroll
        for (int c = 0; c < C1; ++c) tma_load_3d(dst + c * kKvChunk, &tk1, kv_full0 + 8 * s, c * 64, kv_head, row);
#pragma unroll
        for (int c = 0; c < C2; ++c) tma_load_3d(dst + (C1 + c) * kKvChunk, &tk2, kv_full0 + 8 * s, c * 64, 0, row);
#pragma unroll
        for (int c = 0; c < CV; ++c) tma_load_3d(dst + (kQk + c) * kKvChunk, &tv, kv_full0 + 8 * s, c * 64, kv_head, row);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t kFmt = std::is_same<T, __nv_bfloat16>::value ? 1u : 0u;
      constexpr uint32_t idesc_qk = umma_idesc<T>(kKeys);
      // A from TMEM (K-major), B MN-major (bit 16), N = value columns
      constexpr uint32_t idesc_pv = (1u << 4) | (kFmt << 7) | (kFmt << 10) | (1u << 16) |
                                    (static_cast<uint32_t>(CV * 64 >> 3) << 17) | (static_cast<uint32_t>(kRows >> 4) << 24);
      bool ok = mbar_wait(q_full, 0, &abort_flag, 2, &g_window_tc_status);
      auto issue_qk = [&](int g, int t) {
        const uint32_t k_smem = kv_smem + ((t - all.lo) % kStages) * Z::kStage;
        const uint32_t d = tmem_base + g * kGroupCols + ((t - gt[g].lo) & 1) * kKeys;
#pragma unroll
        for (int kk = 0; kk < kQk * 4; ++kk) {
          const uint64_t qd = smem_desc_sw128(base + g * Z::kQBytes + (kk / 4) * kQChunk) + 2 * (kk % 4);
          const uint64_t kd = smem_desc_sw128(k_smem + (kk / 4) * kKvChunk) + 2 * (kk % 4);
          umma_f16(d, qd, kd, idesc_qk, kk > 0 ? 1u : 0u);
        }
        umma_commit(s_full(g, (t - gt[g].lo) & 1));
      };
      auto issue_pv = [&](int g, int t) {
        const int jg = t - gt[g].lo;
        if (!mbar_wait(p_full(g, jg & 1), (static_cast<uint32_t>(jg) >> 1) & 1u, &abort_flag, 4, &g_window_tc_status)) return false;
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        const uint32_t v_smem = kv_smem + ((t - all.lo) % kStages) * Z::kStage + kQk * kKvChunk;
        const uint32_t pa = tmem_base + g * kGroupCols + (jg & 1) * kKeys;
#pragma unroll
        for (int kk = 0; kk < kKeys / kUmmaK; ++kk)
          umma_ts_f16(tmem_base + g * kGroupCols + 2 * kKeys, pa + kk * 8,
                      smem_desc_mn_sw128(v_smem + kk * 2048u, kKvChunk, 1024u), idesc_pv, (jg > 0 || kk > 0) ? 1u : 0u);
        umma_commit(o_done(g, jg & 1));
        return true;
      };
      // S of tile t is issued before P of tile t - 1 is awaited, so the tensor pipe works while the softmax warps do
      for (int j = 0; j <= all.n && ok; ++j) {
        const int t = all.lo + j;
        if (j < all.n) {
          ok = mbar_wait(kv_full0 + 8 * (j % kStages), (j / kStages) & 1u, &abort_flag, 3, &g_window_tc_status);
          if (!ok) break;
          asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
#pragma unroll
          for (int g = 0; g < kGroups; ++g)
            if (active(g, t)) issue_qk(g, t);
        }
        if (j > 0) {
#pragma unroll
          for (int g = 0; g < kGroups; ++g)
            if (ok && active(g, t - 1)) ok = issue_pv(g, t - 1);
          if (ok) umma_commit(kv_empty0 + 8 * ((j - 1) % kStages));
        }
      }
    }
  } else {
    const int g = (warp - 2) >> 2;
    const int quarter = warp & 3;  // TMEM lanes a warp may touch: 32 * (warp id mod 4)
    const int i = quarter * 32 + lane;
    const uint32_t lane_off = static_cast<uint32_t>(quarter * 32) << 16;
    const uint32_t tm = tmem_base + lane_off + g * kGroupCols;
    const int qa = q0 + g * kRows;
    const int jq = history + qa + i;  // key row of this thread's query
    const int lo_i = first_row(p, jq, j_min);
    const int full_lo = first_row(p, history + qa + kRows - 1, j_min);  // from this key row on every query's window has begun
    const int full_hi = history + qa;                                   // up to here no query is behind its key
    const int lo_tile = g == 0 ? gt[0].lo : gt[1].lo, n_tiles = g == 0 ? gt[0].n : gt[1].n;
    float m_ref = -INFINITY, l = 0.f;
    bool alive = n_tiles > 0;
    for (int j = 0; j < n_tiles; ++j) {
      const uint32_t sb = static_cast<uint32_t>(j & 1);
      const bool ready = mbar_wait(s_full(g, sb), (static_cast<uint32_t>(j) >> 1) & 1u, &abort_flag, 5, &g_window_tc_status);
      if (!__all_sync(0xffffffffu, ready)) {
        alive = false;
        break;
      }
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      const uint32_t s_addr = tm + sb * kKeys;
      uint32_t r0[32], r1[32];
      tmem_ld32_issue(s_addr, r0);
      tmem_ld32_issue(s_addr + 32, r1);
      tmem_wait_ld();
      float sv[kKeys];
#pragma unroll
      for (int e = 0; e < 32; ++e) {
        sv[e] = __uint_as_float(r0[e]);
        sv[32 + e] = __uint_as_float(r1[e]);
      }
      const int key0 = (lo_tile + j) * kKeys;
      if (key0 < full_lo || key0 < j_min || key0 + kKeys - 1 > full_hi) {
#pragma unroll
        for (int e = 0; e < kKeys; ++e)
          if (key0 + e < lo_i || key0 + e > jq) sv[e] = -INFINITY;
      }
      float mx4[4] = {sv[0], sv[1], sv[2], sv[3]};
#pragma unroll
      for (int e = 4; e < kKeys; ++e) mx4[e & 3] = fmaxf(mx4[e & 3], sv[e]);
      const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])) * p.scale_log2;
      if (j == 0) {
        m_ref = mx;
      } else {
        const bool need = mx > m_ref + kRescaleLog2;
        if (__any_sync(0xffffffffu, need)) {
          const uint32_t ob = static_cast<uint32_t>((j - 1) & 1);
          const bool done = mbar_wait(o_done(g, ob), (static_cast<uint32_t>(j - 1) >> 1) & 1u, &abort_flag, 6, &g_window_tc_status);
          if (!__all_sync(0xffffffffu, done)) {
            alive = false;
            break;
          }
          asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
          const float corr = need ? exp2f(m_ref - mx) : 1.0f;
#pragma unroll 1
          for (int cc = 0; cc < CV * 64; cc += 32) {
            uint32_t o[32];
            tmem_ld32(tm + 2 * kKeys + cc, o);
#pragma unroll
            for (int e = 0; e < 32; ++e) o[e] = __float_as_uint(__uint_as_float(o[e]) * corr);
            tmem_st32(tm + 2 * kKeys + cc, o);
          }
          tmem_wait_st();
          l *= corr;
          if (need) m_ref = mx;
        }
      }
      const float neg_m = m_ref == -INFINITY ? 0.f : -m_ref;
      uint32_t pk[32];
      float sum4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int e = 0; e < 32; ++e) {
        const float p0 = exp2_approx(fmaf(sv[2 * e], p.scale_log2, neg_m));
        const float p1 = exp2_approx(fmaf(sv[2 * e + 1], p.scale_log2, neg_m));
        sum4[e & 3] += p0 + p1;
        pk[e] = pack2<T>(p0, p1);
      }
      l += (sum4[0] + sum4[1]) + (sum4[2] + sum4[3]);
      tmem_st32(s_addr, pk);  // P over the first 32 columns of this S buffer
      tmem_wait_st();
      asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
      mbar_arrive(p_full(g, sb));
    }
    if (alive) {
      const uint32_t ob = static_cast<uint32_t>((n_tiles - 1) & 1);
      const bool done = mbar_wait(o_done(g, ob), (static_cast<uint32_t>(n_tiles - 1) >> 1) & 1u, &abort_flag, 7, &g_window_tc_status);
      if (__all_sync(0xffffffffu, done)) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        if (p.sink) l += exp2f(fmaf(Num<T>::to_f(static_cast<const T*>(p.sink)[head]), 1.4426950408889634f, m_ref == -INFINITY ? 0.f : -m_ref));
        const float inv = l > 0.f ? p.out_scale / l : 0.f;
        const int s_idx = qa + i;
        T* dst = static_cast<T*>(p.out) + (static_cast<int64_t>(b) * p.S + s_idx) * p.out_ld + static_cast<int64_t>(head) * p.dv;
#pragma unroll 1
        for (int cc = 0; cc < CV * 64; cc += 32) {
          uint32_t o[32];
          tmem_ld32(tm + 2 * kKeys + cc, o);
          if (s_idx < p.S) {
#pragma unroll
            for (int v = 0; v < 4; ++v) {
              if (cc + v * 8 >= p.dv) break;  // dv is a multiple of 8
              float f[8];
#pragma unroll
              for (int e = 0; e < 8; ++e) f[e] = __uint_as_float(o[v * 8 + e]) * inv;
              reinterpret_cast<uint4*>(dst + cc)[v] = pack8<T>(f);
            }
          }
        }
      }
    }
  }

  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  if (abort_flag && threadIdx.x == 0) {
    // give copies that were already issued time to land before the CTA's shared memory is released
    for (int w = 0; w < 2000; ++w) __nanosleep(100);
  }
  __syncthreads();
  if (warp == 1) {
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(kTmemCols) : "memory");
  }
}

template <typename T, int C1, int C2, int CV>
int launch(int dtype, const WindowParams& w, int B, cudaStream_t st) {
  using Z = Sizes<T, C1, C2, CV>;
  CUtensorMap tq1, tq2, tk1, tk2, tv;
  const T* q = static_cast<const T*>(w.q);
  const bool cached = w.history < 0;
  const int kv_heads = w.H / w.group;
  const int64_t q_rows = static_cast<int64_t>(B) * w.S, k_rows = cached ? w.k_rows : B * w.k_rows;
  const int64_t all_heads = cached ? static_cast<int64_t>(B) * kv_heads : kv_heads;
  int rc = make_tmap_heads(&tq1, dtype, q, q_rows, w.q_row, w.H, w.q_head, w.d1, kRows);
  if (rc == LRI_OK) rc = make_tmap_heads(&tk1, dtype, w.k, k_rows, w.k_row, all_heads, w.k_head, w.d1, kKeys);
  if (rc == LRI_OK) rc = make_tmap_heads(&tv, dtype, w.v, k_rows, w.v_row, all_heads, w.v_head, w.dv, kKeys);
  if (C2 > 0) {
    if (rc == LRI_OK) rc = make_tmap_heads(&tq2, dtype, q + w.d1, q_rows, w.q_row, w.H, w.q_head, w.d2, kRows);
    if (rc == LRI_OK) rc = make_tmap_heads(&tk2, dtype, w.k2, k_rows, w.k2_row, 1, w.k2_row, w.d2, kKeys);
  } else {
    tq2 = tq1, tk2 = tk1;  // not read
  }
  if (rc != LRI_OK) return rc;
  TcParams p{};
  p.out = w.out, p.input_pos = w.input_pos, p.pos_is_i64 = w.pos_is_i64;
  p.S = w.S, p.H = w.H, p.dv = w.dv, p.history = w.history, p.k_rows = static_cast<int>(w.k_rows);
  p.group = w.group, p.batch_rows = cached ? 0 : w.k_rows, p.batch_heads = cached ? kv_heads : 0;
  p.chunk = static_cast<int>(w.chunk < (1 << 30) ? w.chunk : 0);
  p.sink = w.sink, p.out_ld = w.out_ld, p.out_scale = w.out_scale;
  p.window = static_cast<int>(w.window < (1 << 30) ? w.window : (1 << 30));
  p.scale_log2 = w.scale * 1.4426950408889634f;
  auto kern = window_attention_tc_kernel<T, C1, C2, CV>;
  static std::atomic<unsigned long long> attr_set{0};
  LRI_ONCE_PER_DEVICE(attr_set, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, Z::kSmem));
  const int per = kRows * kGroups;
  LRI_CUDA(launch_pdl(kern, dim3((w.S + per - 1) / per, w.H, B), dim3(kThreads), static_cast<size_t>(Z::kSmem), st, tq1, tq2, tk1,
                      tk2, tv, p));
  LRI_LAUNCH_CHECK("window_attention_tc_kernel");
  return LRI_OK;
}

template <typename T>
int dispatch(int dtype, const WindowParams& w, int B, cudaStream_t st) {
  if (w.d2 == 0) {
    if (w.d1 <= 64) return w.dv <= 64 ? launch<T, 1, 0, 1>(dtype, w, B, st) : launch<T, 1, 0, 2>(dtype, w, B, st);
    return w.dv <= 64 ? launch<T, 2, 0, 1>(dtype, w, B, st) : launch<T, 2, 0, 2>(dtype, w, B, st);
  }
  if (w.d1 <= 64) return w.dv <= 64 ? launch<T, 1, 1, 1>(dtype, w, B, st) : launch<T, 1, 1, 2>(dtype, w, B, st);
  return w.dv <= 64 ? launch<T, 2, 1, 1>(dtype, w, B, st) : launch<T, 2, 1, 2>(dtype, w, B, st);
}

}  // namespace

bool window_attention_tc_supports(int dtype, const WindowParams& w, int B) {
  if (dtype != LRI_BF16 && dtype != LRI_FP16) return false;
  if (w.S < 16 || !(w.scale > 0.f)) return false;
  if (w.d1 < 8 || w.d1 > 128 || w.d1 % 8 || w.d2 > 64 || w.d2 % 8 || w.dv < 8 || w.dv > 128 || w.dv % 8) return false;
  if (w.q_row % 8 || w.q_head % 8 || w.k_row % 8 || w.k_head % 8 || w.v_row % 8 || w.v_head % 8 || w.out_ld % 8) return false;
  if (w.q_head < 8 || w.k_head < 8 || w.v_head < 8) return false;
  if (w.history < 0) {
    // rows of a cache [sequence, key head, position]: the sequences' heads follow one another
    const int64_t g = w.H / w.group;
    if (w.d2 != 0 || w.k_batch != g * w.k_head || w.v_batch != g * w.v_head) return false;
    if (!aligned16(w.q) || !aligned16(w.k) || !aligned16(w.v) || !aligned16(w.out)) return false;
    return B <= 65535 && w.H <= 65535 && w.k_rows < (1ll << 30) && B * g < (1ll << 31) &&
           static_cast<int64_t>(B) * w.S + 2 * kRows < (1ll << 31);
  }
  if (w.d2 < 8 || w.k2_row % 8 || w.group != 1 || w.chunk > 0) return false;
  // the rows of the sequences follow one another
  if (w.k_batch != w.k_rows * w.k_row || w.k2_batch != w.k_rows * w.k2_row || w.v_batch != w.k_rows * w.v_row) return false;
  if (w.k_rows < w.history + w.S) return false;
  if (!aligned16(w.q) || !aligned16(w.k) || !aligned16(w.k2) || !aligned16(w.v) || !aligned16(w.out)) return false;
  return B <= 65535 && w.H <= 65535 && B * w.k_rows + kKeys < (1ll << 31) && static_cast<int64_t>(B) * w.S + 2 * kRows < (1ll << 31);
}

int window_attention_tc_launch(int dtype, const WindowParams& w, int B, cudaStream_t st) {
  return dtype == LRI_BF16 ? dispatch<__nv_bfloat16>(dtype, w, B, st) : dispatch<__half>(dtype, w, B, st);
}

int window_attention_tc_status_read_and_clear(int* status_out) {
  int v = 0;
  LRI_CUDA(cudaMemcpyFromSymbol(&v, g_window_tc_status, sizeof(int)));
  if (v != 0) {
    int zero = 0;
    LRI_CUDA(cudaMemcpyToSymbol(g_window_tc_status, &zero, sizeof(int)));
  }
  *status_out = v;
  return LRI_OK;
}

}  // namespace lri
