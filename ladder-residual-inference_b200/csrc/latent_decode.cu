// Single-token attention on cached latents (flash-decoding over the window): every head's query has the width of a cache
// row [latent (r) | rotated key (dr)], and the values are the rows' latents, so a row read once serves as key and value of
// all heads.
//
// CTA (split, tile of 16 heads, sequence): walks its share of the visible 64-row tiles.  A tile is copied to shared
// memory once (cp.async); S = Q K^T and O += P V run on mma.sync m16n8k16 with the 16 heads as rows: in the score phase a
// warp owns 8 keys, in the value phase a share of the latent columns.  Softmax state is fp32.  Partial results of the
// splits are merged by a second kernel.
#include "latent_attention.cuh"
#include "mma.cuh"

namespace lri {
namespace {

constexpr int kKeys = 64, kHeads = 16, kWarps = 8, kThreads = kWarps * 32;
constexpr int kMaxSplits = 128;
constexpr int kMaxUnits = 4;  // 16-column units of the latent per warp: r <= 512
constexpr int kPadP = 72, kPadS = 68;

struct DecodeParams {
  const void* q;  // [B, H, row_len]
  int64_t q_row, q_head;
  const void* cache;  // [B, smax, row_len]
  int64_t batch_pitch, smax;
  const void* input_pos;
  int pos_is_i64;
  int64_t window;
  float scale_log2;
  int H, r, row_len, splits;
  void* out;      // [B, H, r]
  float* part_o;  // [B, H, splits, r]
  float* part_ml;  // [B, H, splits, 2]
};

__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(dst))), "l"(src)
               : "memory");
}
__device__ __forceinline__ void cp_async_wait_all() { asm volatile("cp.async.wait_all;" ::: "memory"); }

// Visible rows lo .. hi and the tiles t0 .. t1 - 1 of a split
struct TileRange {
  int64_t lo, hi, t0, t1;
};
__device__ __forceinline__ TileRange tile_range(const DecodeParams& p, int split) {
  const int64_t pos = *reinterpret_cast<const volatile int*>(p.input_pos);  // the low word of a 64-bit position too
  TileRange r;
  r.hi = pos < p.smax ? pos : p.smax - 1;
  r.lo = pos - p.window + 1;
  r.lo = r.lo < 0 ? 0 : r.lo;
  const int64_t first = r.lo / kKeys, n = r.hi / kKeys - first + 1;
  const int64_t per = (n + p.splits - 1) / p.splits;
  r.t0 = first + split * per;
  r.t1 = r.t0 + per < first + n ? r.t0 + per : first + n;
  return r;
}

template <typename T>
__global__ void __launch_bounds__(kThreads) latent_decode_kernel(const DecodeParams p) {
  extern __shared__ __align__(16) uint8_t ld_smem[];
  const int pitch = p.row_len + 8;  // an odd number of 16-byte units: ldmatrix rows fall into different banks
  T* ks = reinterpret_cast<T*>(ld_smem);
  T* qs = ks + kKeys * pitch;
  T* ps = qs + kHeads * pitch;
  float* sc = reinterpret_cast<float*>(ps + kHeads * kPadP);
  __shared__ float m_s[kHeads], l_s[kHeads], corr_s[kHeads];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int split = blockIdx.x, h0 = blockIdx.y * kHeads, b = blockIdx.z;
  const int vecs = p.row_len / 8;
  const T* kg = static_cast<const T*>(p.cache) + b * p.batch_pitch;
  pdl_launch_dependents();
  // Rows of earlier steps do not depend on the preceding kernel: ask the L2 for the first tile while it drains.  (Only a
  // hint, from a position that may not be final, kept inside the cache.)
  {
    const TileRange g = tile_range(p, split);
    const int64_t row = g.t0 * kKeys + (threadIdx.x >> 2);
    if (g.t0 < g.t1 && row >= 0 && row < p.smax)
      for (int e = (threadIdx.x & 3) * 64; e < p.row_len; e += 256)
        asm volatile("prefetch.global.L2 [%0];" ::"l"(kg + row * p.row_len + e));
  }
  pdl_wait();
  const TileRange range = tile_range(p, split);
  const int64_t lo = range.lo, hi = range.hi, t0 = range.t0, t1 = range.t1;
  const T* qg = static_cast<const T*>(p.q) + b * p.q_row;
  // (a warp copies whole rows; the wait for the first tile of keys covers the queries too)
  for (int h = warp; h < kHeads; h += kWarps)
    for (int v = lane; v < vecs; v += 32) {
      T* dst = qs + h * pitch + v * 8;
      if (h0 + h < p.H)
        cp_async16(dst, qg + (h0 + h) * p.q_head + v * 8);
      else
        *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
    }
  if (threadIdx.x < kHeads) m_s[threadIdx.x] = -INFINITY, l_s[threadIdx.x] = 0.f;
  float acc[kMaxUnits][2][4];
#pragma unroll
  for (int u = 0; u < kMaxUnits; ++u)
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[u][n][e] = 0.f;
  const int units = p.r / 16;

  for (int64_t t = t0; t < t1; ++t) {
    __syncthreads();  // the previous tile has been consumed (first pass: nothing)
#pragma unroll
    for (int i = 0; i < kKeys / kWarps; ++i) {
      const int j = warp * (kKeys / kWarps) + i;
      const int64_t row = t * kKeys + j;
      T* dst = ks + j * pitch;
      const T* src = kg + row * p.row_len;
      for (int v = lane; v < vecs; v += 32) {
        if (row <= hi)
          cp_async16(dst + v * 8, src + v * 8);
        else
          *reinterpret_cast<uint4*>(dst + v * 8) = make_uint4(0, 0, 0, 0);
      }
    }
    cp_async_wait_all();
    __syncthreads();
    // scores of 16 heads x this warp's 8 keys
    {
      float c[4] = {0.f, 0.f, 0.f, 0.f}, c2[4] = {0.f, 0.f, 0.f, 0.f};  // two chains of products
      const T* qa = qs + (lane & 15) * pitch + (lane >> 4) * 8;
      const T* kb = ks + (warp * 8 + (lane & 7)) * pitch + (lane >> 3) * 8;
      int k = 0;
#pragma unroll 4
      for (; k + 32 <= p.row_len; k += 32) {
        uint32_t a[8], bb[4];
        ldmatrix_x4(qa + k, a[0], a[1], a[2], a[3]);
        ldmatrix_x4(qa + k + 16, a[4], a[5], a[6], a[7]);
        ldmatrix_x4(kb + k, bb[0], bb[1], bb[2], bb[3]);
        mma16816<T>(c, a[0], a[1], a[2], a[3], bb[0], bb[1]);
        mma16816<T>(c2, a[4], a[5], a[6], a[7], bb[2], bb[3]);
      }
      if (k < p.row_len) {
        uint32_t a0, a1, a2, a3, b0, b1;
        ldmatrix_x4(qa + k, a0, a1, a2, a3);
        ldmatrix_x2(ks + (warp * 8 + (lane & 7)) * pitch + ((lane >> 3) & 1) * 8 + k, b0, b1);
        mma16816<T>(c, a0, a1, a2, a3, b0, b1);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) c[e] += c2[e];
      const int row = lane >> 2, col = warp * 8 + 2 * (lane & 3);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int64_t key = t * kKeys + col + (e & 1);
        sc[(row + (e >> 1) * 8) * kPadS + col + (e & 1)] = key >= lo && key <= hi ? c[e] * p.scale_log2 : -INFINITY;
      }
    }
    __syncthreads();
    // softmax of two heads per warp
#pragma unroll
    for (int i = 0; i < kHeads / kWarps; ++i) {
      const int h = warp * (kHeads / kWarps) + i;
      const float s0 = sc[h * kPadS + 2 * lane], s1 = sc[h * kPadS + 2 * lane + 1];
      const float m_old = m_s[h];
      const float m = fmaxf(m_old, warp_max(fmaxf(s0, s1)));
      const float ref = m == -INFINITY ? 0.f : m;
      const float p0 = exp2f(s0 - ref), p1 = exp2f(s1 - ref);
      const float sum = warp_sum(p0 + p1);
      *reinterpret_cast<uint32_t*>(ps + h * kPadP + 2 * lane) = pack2<T>(p0, p1);
      if (lane == 0) {
        const float corr = exp2f(m_old - ref);  // exp2(-inf) = 0
        m_s[h] = m;
        l_s[h] = l_s[h] * corr + sum;
        corr_s[h] = corr;
      }
    }
    __syncthreads();
    // O += P V on this warp's columns
    const float c0 = corr_s[lane >> 2], c1 = corr_s[(lane >> 2) + 8];
    uint32_t pa[4][4];
#pragma unroll
    for (int k = 0; k < 4; ++k)
      ldmatrix_x4(ps + (lane & 15) * kPadP + k * 16 + (lane >> 4) * 8, pa[k][0], pa[k][1], pa[k][2], pa[k][3]);
#pragma unroll
    for (int u = 0; u < kMaxUnits; ++u) {
      const int unit = warp + u * kWarps;
      if (unit >= units) break;
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        acc[u][n][0] *= c0, acc[u][n][1] *= c0;
        acc[u][n][2] *= c1, acc[u][n][3] *= c1;
      }
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4_trans(ks + (k * 16 + (lane & 15)) * pitch + unit * 16 + (lane >> 4) * 8, b0, b1, b2, b3);
        mma16816<T>(acc[u][0], pa[k][0], pa[k][1], pa[k][2], pa[k][3], b0, b1);
        mma16816<T>(acc[u][1], pa[k][0], pa[k][1], pa[k][2], pa[k][3], b2, b3);
      }
    }
  }
  __syncthreads();
  const int row = lane >> 2;
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int h = h0 + row + half * 8;
    if (h >= p.H) continue;
    const int64_t bh = static_cast<int64_t>(b) * p.H + h;
    const float l = l_s[row + half * 8];
    if (p.splits > 1) {
      if (warp == 0 && (lane & 3) == 0) {
        float* ml = p.part_ml + (bh * p.splits + split) * 2;
        ml[0] = m_s[row + half * 8];
        ml[1] = l;
      }
      if (t0 >= t1) continue;  // no keys: the merge skips this split
    }
    const float inv = l > 0.f ? 1.0f / l : 0.f;
#pragma unroll
    for (int u = 0; u < kMaxUnits; ++u) {
      const int unit = warp + u * kWarps;
      if (unit >= units) break;
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        const int col = unit * 16 + n * 8 + 2 * (lane & 3);
        const float v0 = acc[u][n][2 * half], v1 = acc[u][n][2 * half + 1];
        if (p.splits > 1)
          *reinterpret_cast<float2*>(p.part_o + (bh * p.splits + split) * p.r + col) = make_float2(v0, v1);
        else
          *reinterpret_cast<uint32_t*>(static_cast<T*>(p.out) + bh * p.r + col) = pack2<T>(v0 * inv, v1 * inv);
      }
    }
  }
}

// Grid (heads, sequences, column groups of 128)
template <typename T>
__global__ void __launch_bounds__(128) latent_decode_merge_kernel(const DecodeParams p) {
  __shared__ float w_s[kMaxSplits];
  __shared__ float part[33];
  __shared__ float4 sums[4][32];
  pdl_launch_dependents();
  pdl_wait();
  const int64_t bh = static_cast<int64_t>(blockIdx.y) * p.H + blockIdx.x;
  static_assert(kMaxSplits == 128, "one thread per split");
  const int s = threadIdx.x;
  float2 ml = make_float2(-INFINITY, 0.f);
  if (s < p.splits) ml = *reinterpret_cast<const float2*>(p.part_ml + (bh * p.splits + s) * 2);
  const bool used = ml.y > 0.f;  // every tile of a window holds a visible key: the splits in use come first
  const float wm = warp_max(ml.x);
  if ((s & 31) == 0) part[s >> 5] = wm;
  const int n = __syncthreads_count(used);
  const float m = fmaxf(fmaxf(part[0], part[1]), fmaxf(part[2], part[3]));
  const float w = used ? exp2f(ml.x - m) : 0.f;
  w_s[s] = w;
  __syncthreads();  // part is used again
  const float l = block_sum(w * ml.y, part);  // also orders w_s
  // 4 warps take every fourth split, a lane 4 columns: the loads of a thread are in flight together
  const int warp = s >> 5, lane = s & 31;
  const int col = blockIdx.z * 128 + lane * 4;
  float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
  if (col < p.r) {
    const float* o = p.part_o + bh * p.splits * p.r + col;
#pragma unroll 8
    for (int i = warp; i < n; i += 4) {
      const float4 v = *reinterpret_cast<const float4*>(o + static_cast<int64_t>(i) * p.r);
      const float wi = w_s[i];
      acc.x = fmaf(wi, v.x, acc.x), acc.y = fmaf(wi, v.y, acc.y), acc.z = fmaf(wi, v.z, acc.z), acc.w = fmaf(wi, v.w, acc.w);
    }
  }
  sums[warp][lane] = acc;
  __syncthreads();
  const int c = blockIdx.z * 128 + s;
  if (c >= p.r) return;
  float v = 0.f;
#pragma unroll
  for (int i = 0; i < 4; ++i) v += reinterpret_cast<const float*>(&sums[i][0])[s];
  static_cast<T*>(p.out)[bh * p.r + c] = Num<T>::from_f(l > 0.f ? v / l : 0.f);
}

int head_tiles(int H) { return (H + kHeads - 1) / kHeads; }

int plan_splits(int B, int H, int64_t keys) {
  const int64_t tiles = keys / kKeys + 2;  // a window may begin and end inside a tile
  int64_t s = 2 * device_sm_count() / (static_cast<int64_t>(B) * head_tiles(H));
  s = s > tiles ? tiles : s;
  s = s > kMaxSplits ? kMaxSplits : s;
  return s < 1 ? 1 : static_cast<int>(s);
}

template <typename T>
int launch(const DecodeParams& p, int B, cudaStream_t st) {
  const size_t pitch = p.row_len + 8;
  const size_t smem = ((kKeys + kHeads) * pitch + kHeads * kPadP) * sizeof(T) + kHeads * kPadS * sizeof(float);
  auto kern = latent_decode_kernel<T>;
  static std::atomic<unsigned long long> attr_set{0};
  LRI_ONCE_PER_DEVICE(attr_set, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 112 * 1024));
  LRI_CUDA(launch_pdl(kern, dim3(p.splits, head_tiles(p.H), B), dim3(kThreads), smem, st, p));
  LRI_LAUNCH_CHECK("latent_decode_kernel");
  if (p.splits > 1) {
    LRI_CUDA(launch_pdl(latent_decode_merge_kernel<T>, dim3(p.H, B, (p.r + 127) / 128), dim3(128), 0, st, p));
    LRI_LAUNCH_CHECK("latent_decode_merge_kernel");
  }
  return LRI_OK;
}

}  // namespace

bool latent_decode_supports(int dtype, const WindowParams& w) {
  if (dtype != LRI_BF16 && dtype != LRI_FP16) return false;
  if (w.S != 1 || w.history >= 0 || w.k_head != 0 || w.v_head != 0 || w.k != w.v || w.dv != w.d1) return false;
  const int row_len = w.d1 + w.d2;
  if (w.d1 % 16 || w.d2 % 16 || w.d1 > 16 * kMaxUnits * kWarps || row_len > 640) return false;
  if (w.k_row != row_len || w.k2_row != row_len || w.v_row != row_len || w.k_batch != w.v_batch || w.k_batch != w.k2_batch) return false;
  if (static_cast<const uint16_t*>(w.k2) != static_cast<const uint16_t*>(w.k) + w.d1) return false;
  return w.q_row % 8 == 0 && w.q_head % 8 == 0 && w.k_batch % 8 == 0 && aligned16(w.q) && aligned16(w.k) && aligned16(w.out) &&
         w.H <= 16 * 65535;
}

// keys: the most keys a query can see
size_t latent_decode_scratch_bytes(int B, int H, int dv, int64_t keys) {
  const size_t s = plan_splits(B, H, keys);
  return s > 1 ? static_cast<size_t>(B) * H * s * (dv + 2) * sizeof(float) : 0;
}

int latent_decode_launch(int dtype, const WindowParams& w, int B, void* scratch, size_t scratch_bytes, cudaStream_t st) {
  DecodeParams p{};
  p.q = w.q, p.q_row = w.q_row, p.q_head = w.q_head, p.cache = w.k, p.batch_pitch = w.k_batch, p.smax = w.k_rows;
  p.input_pos = w.input_pos, p.pos_is_i64 = w.pos_is_i64, p.window = w.window;
  p.scale_log2 = w.scale * 1.4426950408889634f;
  p.H = w.H, p.r = w.d1, p.row_len = w.d1 + w.d2, p.out = w.out;
  const int64_t keys = w.window < w.k_rows ? w.window : w.k_rows;
  p.splits = plan_splits(B, w.H, keys);
  const size_t need = latent_decode_scratch_bytes(B, w.H, w.dv, keys);
  LRI_REQUIRE(need == 0 || (scratch && aligned16(scratch) && scratch_bytes >= need), LRI_ERR_WORKSPACE,
              "window_attention: scratch of %zu bytes (16-byte aligned) required", need);
  p.part_o = static_cast<float*>(scratch);
  p.part_ml = p.part_o + static_cast<size_t>(B) * w.H * p.splits * w.dv;
  return dtype == LRI_BF16 ? launch<__nv_bfloat16>(p, B, st) : launch<__half>(p, B, st);
}

}  // namespace lri
