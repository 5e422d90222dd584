// Mixture-of-experts feed-forward: routing, the grouping of tokens by expert, and the expert projections.
//
//   route    per token: logistic scores of the router logits, the `top` largest (lowest index on ties)
//   plan     per expert: the tokens that chose it are packed into tiles of 128 rows; the tile list names the expert
//   gather   copies each token's row to its packed places
//   gate/up  hidden = glu(score * (W_gate x), score * (W_up x)); the score multiplies the expert's INPUT, which is the
//            same as scaling the fp32 sums of the two projections
//   down     y = W_down hidden
//
// Few (token, choice) pairs run unpacked: the weight-streaming kernel takes one pair per grid slice and picks the
// expert's matrix on the device.  Many pairs run as tcgen05 tiles of 128 packed rows, each tile with its expert's matrix.
// fp32 and shapes that are not multiples of 8 run a plain SIMT kernel, one pair per grid slice.
#include "linear.cuh"

namespace lri {
namespace {

// (No __restrict__ on what a preceding kernel writes: loads of read-only pointers may be moved above the wait for it.)
constexpr int kTileRows = 128;
constexpr int kRouteWarps = 4;
constexpr int kMaxExperts = 1024;

// One warp per token.  scratch (when given): counts[e] becomes the number of tokens of expert e and rank[pair] the
// place of the pair among them.
__global__ void __launch_bounds__(kRouteWarps * 32)
moe_route_kernel(const float* logits, int64_t ld, int experts, int top, int64_t rows, int32_t* ids,
                 float* scores, int32_t* counts, int32_t* rank) {
  extern __shared__ float route_smem[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* s = route_smem + warp * experts;
  const int64_t row = static_cast<int64_t>(blockIdx.x) * kRouteWarps + warp;
  pdl_launch_dependents();
  pdl_wait();
  if (row >= rows) return;
  for (int e = lane; e < experts; e += 32) s[e] = logits[row * ld + e];
  __syncwarp();
  for (int k = 0; k < top; ++k) {
    // the logistic function is monotonic: the largest logits are the largest scores
    float best = -INFINITY;
    int arg = experts;
    for (int e = lane; e < experts; e += 32)
      if (s[e] > best || arg == experts) best = s[e], arg = e;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, o);
      const int oa = __shfl_xor_sync(0xffffffffu, arg, o);
      if (oa < experts && (arg >= experts || ob > best || (ob == best && oa < arg))) best = ob, arg = oa;
    }
    if (lane == 0) {
      const int64_t pair = row * top + k;
      ids[pair] = arg;
      scores[pair] = sigmoid_f(best);
      if (counts) rank[pair] = atomicAdd(counts + arg, 1);
      s[arg] = -INFINITY;
    }
    __syncwarp();
  }
}

// One CTA: tile list and first packed row of every expert from the counts, which are left at zero.
__global__ void __launch_bounds__(1024)
moe_plan_kernel(int experts, int max_tiles, int32_t* counts, int32_t* first_row, int32_t* tiles) {
  __shared__ int scan[kMaxExperts];
  pdl_launch_dependents();
  pdl_wait();
  const int e = threadIdx.x;
  const int mine = e < experts ? (counts[e] + kTileRows - 1) / kTileRows : 0;
  scan[e] = mine;
  __syncthreads();
  for (int o = 1; o < kMaxExperts; o <<= 1) {
    const int add = e >= o ? scan[e - o] : 0;
    __syncthreads();
    scan[e] += add;
    __syncthreads();
  }
  const int t0 = scan[e] - mine;
  if (e < experts) {
    counts[e] = 0;
    first_row[e] = t0 * kTileRows;
    for (int t = 0; t < mine && t0 + t < max_tiles; ++t) tiles[1 + t0 + t] = e;
  }
  if (e == kMaxExperts - 1) tiles[0] = scan[e] < max_tiles ? scan[e] : max_tiles;
}

// One CTA per pair: packed row, its scale, and where the combine step finds the pair's result.
__global__ void __launch_bounds__(128)
moe_gather_kernel(const uint4* x, int vecs, int top, const int32_t* ids,
                  const float* scores, const int32_t* rank, const int32_t* first_row,
                  int64_t packed_rows, uint4* packed, float* row_scale, int32_t* slots) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t pair = blockIdx.x;
  const int64_t dst = first_row[ids[pair]] + rank[pair];
  if (dst < 0 || dst >= packed_rows) return;  // ranks of another call: nothing is written outside the buffers
  const uint4* src = x + (pair / top) * vecs;
  for (int v = threadIdx.x; v < vecs; v += 128) packed[dst * vecs + v] = src[v];
  if (threadIdx.x == 0) {
    row_scale[dst] = scores[pair];
    slots[pair] = static_cast<int32_t>(dst);
  }
}

// Plain form for any shape and type: grid (output groups of 8, pairs), one warp per output.
template <typename T, bool GLU>
__global__ void __launch_bounds__(256)
moe_generic_kernel(const T* __restrict__ x, const T* __restrict__ w, T* __restrict__ y, const ExpertArgs ex, int n, int k) {
  const int64_t pair = blockIdx.y;
  const int j = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (j >= n) return;
  const T* xr = x + (pair / ex.rows_per_input) * k;
  const T* wr = w + (static_cast<int64_t>(ex.experts[pair]) * ex.matrix_rows + j) * k;
  float a = 0.f, b = 0.f;
  for (int i = lane; i < k; i += 32) {
    const float xv = Num<T>::to_f(xr[i]);
    a = fmaf(Num<T>::to_f(wr[i]), xv, a);
    if (GLU) b = fmaf(Num<T>::to_f(wr[static_cast<int64_t>(n) * k + i]), xv, b);
  }
  a = warp_sum(a);
  if (GLU) b = warp_sum(b);
  if (lane == 0) {
    if (GLU) {
      const float sc = ex.row_scale[pair];
      a = clamped_glu(sc * b, sc * a, ex.glu);
    }
    y[pair * n + j] = Num<T>::from_f(a);
  }
}

template <typename T>
int generic(bool glu, const void* x, const void* w, void* y, const ExpertArgs& ex, int64_t pairs, int n, int k, cudaStream_t st) {
  for (int64_t p0 = 0; p0 < pairs; p0 += 65532 / ex.rows_per_input * ex.rows_per_input) {
    // (a grid dimension holds 65535 slices; slices start at a multiple of rows_per_input)
    const int64_t step = 65532 / ex.rows_per_input * ex.rows_per_input;
    const unsigned here = static_cast<unsigned>(pairs - p0 < step ? pairs - p0 : step);
    ExpertArgs a = ex;
    a.experts += p0;
    if (a.row_scale) a.row_scale += p0;
    const T* xp = static_cast<const T*>(x) + p0 / ex.rows_per_input * k;
    T* yp = static_cast<T*>(y) + p0 * n;
    const dim3 grid((n + 7) / 8, here);
    if (glu)
      moe_generic_kernel<T, true><<<grid, 256, 0, st>>>(xp, static_cast<const T*>(w), yp, a, n, k);
    else
      moe_generic_kernel<T, false><<<grid, 256, 0, st>>>(xp, static_cast<const T*>(w), yp, a, n, k);
    LRI_LAUNCH_CHECK("moe_generic_kernel");
  }
  return LRI_OK;
}

}  // namespace
}  // namespace lri

using namespace lri;

// Pairs up to which the unpacked streaming kernel runs (measured at 8 experts of 4096 x 7168, top 2: 8 pairs 147 against
// 178 us for both projections with packing, 16 pairs 286 against 231 us).
static int streaming_pairs() { return option(OPT_MOE_STREAM_PAIRS); }

extern "C" int lri_moe_packs(int dtype, int64_t rows, int top, int dim, int ff) {
  return dtype != LRI_FP32 && rows * top > streaming_pairs() && dim % 8 == 0 && ff % 8 == 0 ? 1 : 0;
}
extern "C" int64_t lri_moe_max_tiles(int64_t rows, int top, int experts) {
  const int64_t pairs = rows * top;
  return pairs / kTileRows + (pairs < experts ? pairs : experts);
}

extern "C" int lri_moe_route(const float* logits, int64_t ld, int experts, int top, int64_t rows, int32_t* ids, float* scores,
                             int32_t* counts, int32_t* rank, lri_stream_t stream) {
  LRI_REQUIRE(logits && ids && scores && (counts == nullptr) == (rank == nullptr), LRI_ERR_ARG, "moe_route: NULL pointer");
  LRI_REQUIRE(experts >= 1 && experts <= kMaxExperts && top >= 1 && top <= experts, LRI_ERR_UNSUPPORTED,
              "moe_route: %d of %d experts (at most %d)", top, experts, kMaxExperts);
  LRI_REQUIRE(rows >= 0 && rows * top < (1ll << 31), LRI_ERR_ARG, "moe_route: rows=%lld", (long long)rows);
  if (rows == 0) return LRI_OK;
  const unsigned grid = static_cast<unsigned>((rows + kRouteWarps - 1) / kRouteWarps);
  LRI_CUDA(launch_pdl(moe_route_kernel, dim3(grid), dim3(kRouteWarps * 32), static_cast<size_t>(experts) * kRouteWarps * sizeof(float),
                      static_cast<cudaStream_t>(stream), logits, ld, experts, top, rows, ids, scores, counts, rank));
  LRI_LAUNCH_CHECK("moe_route_kernel");
  return LRI_OK;
}

extern "C" int lri_moe_pack(int dtype, const void* x, int64_t rows, int dim, int top, int experts, const int32_t* ids,
                            const float* scores, const int32_t* rank, int32_t* counts, int32_t* first_row, int32_t* tiles,
                            int64_t max_tiles, void* packed, float* row_scale, int32_t* slots, lri_stream_t stream) {
  LRI_REQUIRE(dtype == LRI_BF16 || dtype == LRI_FP16, LRI_ERR_UNSUPPORTED, "moe_pack: dtype %d", dtype);
  LRI_REQUIRE(x && ids && scores && rank && counts && first_row && tiles && packed && row_scale && slots, LRI_ERR_ARG,
              "moe_pack: NULL pointer");
  LRI_REQUIRE(dim > 0 && dim % 8 == 0 && aligned16(x) && aligned16(packed), LRI_ERR_ALIGN,
              "moe_pack: dim=%d must be a multiple of 8 and the rows 16-byte aligned", dim);
  LRI_REQUIRE(experts >= 1 && experts <= kMaxExperts, LRI_ERR_UNSUPPORTED, "moe_pack: %d experts", experts);
  LRI_REQUIRE(rows > 0 && rows * top < (1ll << 31), LRI_ERR_ARG, "moe_pack: rows=%lld", (long long)rows);
  LRI_REQUIRE(max_tiles >= lri_moe_max_tiles(rows, top, experts), LRI_ERR_ARG, "moe_pack: room for %lld tiles, %lld needed",
              (long long)max_tiles, (long long)lri_moe_max_tiles(rows, top, experts));
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  LRI_CUDA(launch_pdl(moe_plan_kernel, dim3(1), dim3(kMaxExperts), 0, st, experts,
                      static_cast<int>(max_tiles), counts, first_row, tiles));
  LRI_LAUNCH_CHECK("moe_plan_kernel");
  LRI_CUDA(launch_pdl(moe_gather_kernel, dim3(static_cast<unsigned>(rows * top)), dim3(128), 0, st,
                      static_cast<const uint4*>(x), dim / 8, top, ids, scores, rank, first_row, max_tiles * kTileRows, static_cast<uint4*>(packed),
                      row_scale, slots));
  LRI_LAUNCH_CHECK("moe_gather_kernel");
  return LRI_OK;
}

static int check_experts(const char* who, int dtype, const void* x, const void* w, const void* y, int n, int k) {
  LRI_REQUIRE(dtype >= LRI_BF16 && dtype <= LRI_FP32, LRI_ERR_UNSUPPORTED, "%s: dtype %d", who, dtype);
  LRI_REQUIRE(x && w && y, LRI_ERR_ARG, "%s: NULL pointer", who);
  LRI_REQUIRE(n > 0 && k > 0, LRI_ERR_ARG, "%s: N=%d K=%d", who, n, k);
  return LRI_OK;
}

static int experts_unpacked(const char* who, int epi, int dtype, const void* x, const void* w, void* y, const ExpertArgs& ex,
                            int64_t pairs, int n, int k, cudaStream_t st) {
  LRI_REQUIRE(ex.experts && pairs > 0 && pairs < (1ll << 31) && ex.rows_per_input > 0, LRI_ERR_ARG, "%s: pairs=%lld", who,
              (long long)pairs);
  const bool glu = epi == EPI_GLU;
  if (dtype != LRI_FP32 && k % 8 == 0 && aligned16(x) && aligned16(w) && n <= 2 * 65535) {
    LinearParams p{};
    p.x = x, p.w = w, p.y = y, p.m = 1, p.n = n, p.k = k;
    p.ex = ex;
    p.ex.pairs = static_cast<int>(pairs);
    return gemv_launch(dtype, epi, p, st);
  }
  if (dtype == LRI_BF16) return generic<__nv_bfloat16>(glu, x, w, y, ex, pairs, n, k, st);
  if (dtype == LRI_FP16) return generic<__half>(glu, x, w, y, ex, pairs, n, k, st);
  return generic<float>(glu, x, w, y, ex, pairs, n, k, st);
}

static int experts_packed(const char* who, int epi, int dtype, const void* x, const void* w, void* y, const ExpertArgs& ex,
                          int experts, int64_t max_tiles, int n, int k, cudaStream_t st) {
  LRI_REQUIRE(dtype != LRI_FP32 && max_tiles > 0 && max_tiles * kTileRows < (1ll << 31), LRI_ERR_ARG, "%s: max_tiles=%lld", who,
              (long long)max_tiles);
  LinearParams p{};
  p.x = x, p.w = w, p.y = y, p.m = static_cast<int>(max_tiles * kTileRows), p.n = n, p.k = k;
  p.ex = ex;
  p.ex.pairs = experts;
  return gemm_tcgen05_experts_launch(dtype, epi, p, static_cast<int>(max_tiles), st);
}

extern "C" int lri_moe_gateup(int dtype, const void* x, const void* w1, void* hidden, const int32_t* ids, const float* scores,
                              int64_t pairs, int top, const int32_t* tiles, const float* row_scale, int64_t max_tiles,
                              int experts, int ff, int dim, float alpha, float limit, float offset, lri_stream_t stream) {
  int rc = check_experts("moe_gateup", dtype, x, w1, hidden, ff, dim);
  if (rc != LRI_OK) return rc;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  ExpertArgs ex{};
  ex.matrix_rows = 2ll * ff;
  ex.glu = GluParams{alpha, limit, offset};
  if (tiles) {
    LRI_REQUIRE(row_scale, LRI_ERR_ARG, "moe_gateup: row_scale is NULL");
    ex.tiles = tiles, ex.row_scale = row_scale;
    return experts_packed("moe_gateup", EPI_GLU, dtype, x, w1, hidden, ex, experts, max_tiles, ff, dim, st);
  }
  LRI_REQUIRE(ids && scores, LRI_ERR_ARG, "moe_gateup: ids or scores is NULL");
  ex.experts = ids, ex.row_scale = scores, ex.rows_per_input = top;
  return experts_unpacked("moe_gateup", EPI_GLU, dtype, x, w1, hidden, ex, pairs, ff, dim, st);
}

extern "C" int lri_moe_down(int dtype, const void* hidden, const void* w2, void* y, const int32_t* ids, int64_t pairs,
                            const int32_t* tiles, int64_t max_tiles, int experts, int dim, int ff, lri_stream_t stream) {
  int rc = check_experts("moe_down", dtype, hidden, w2, y, dim, ff);
  if (rc != LRI_OK) return rc;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  ExpertArgs ex{};
  ex.matrix_rows = dim;
  if (tiles) {
    ex.tiles = tiles;
    return experts_packed("moe_down", EPI_PLAIN, dtype, hidden, w2, y, ex, experts, max_tiles, dim, ff, st);
  }
  ex.experts = ids, ex.rows_per_input = 1;
  return experts_unpacked("moe_down", EPI_PLAIN, dtype, hidden, w2, y, ex, pairs, dim, ff, st);
}
