// HGRN2 over prompt portions: 16 tokens at a time on tensor cores, segments of a sequence in parallel.
//
// With f the forget gates of a block of 16 tokens (per head and channel c), k = 1 - f, and S the state before the block:
//   q"_t = q_t prod_{1..t} f        k"_s = k_s prod_{s+1..16} f        F = prod_{1..16} f
//   A[t, s] = sum_c q_t k_s prod_{s+1..t} f   (s <= t)
//   o_t = q"_t S + sum_s A[t, s] v_s          S <- F S + sum_s k"_s v_s
// Every product of gates is a running product, never a quotient or a difference of logarithms, so small gates
// are harmless.  A is summed in fp32; the other sums are mma.sync products.
//
// Precision: gates, running products, A and the state are fp32.  A tensor-core operand that holds them is the sum of three
// bf16 terms (24 mantissa bits, an fp32 value), and a product keeps the term pairs that reach beyond 2^-24; sums are
// fp32.  The values v are a projection and enter in the storage type (one bf16 term, two for fp16).
//
// The state is held transposed, S^T [E, C], in the accumulators of the warps (16 rows of E and half of the channels
// each): those fragments are the A operand of o^T = S^T q"^T as they stand, and the result of the update
// S^T <- S^T F + V^T K".
//
// A CTA runs one segment of one (sequence, head).  With P > 1 segments a first pass leaves every segment's own
// contribution and decay in the workspace (the first segment's contribution starts from the sequence's state), and the second
// pass starts segment p from R_0, decayed and joined with the contributions of segments 1 .. p - 1.
#include "hgrn2.cuh"
#include "mma.cuh"

#include <type_traits>

namespace lri {
namespace {

constexpr int kBlock = 16;
constexpr int kThreads = 512, kWarps = 16;
constexpr int kTerms = 3;
constexpr int kMaxSegments = 8;
constexpr int kMinSegment = 64;  // tokens
constexpr int kMaxE = 128;

using bf16 = __nv_bfloat16;

struct Segments {
  int count, tokens;  // segments per sequence and tokens of each but the last
  float* init;        // [B, H, C, E] state before the call
  float* part;        // [count - 1][B, H, C, E]
  float* decay;       // [count - 1][B, H, C]
};

// x = t[0] + t[1] + t[2] up to 2^-24 |x|; two values at a time, packed low half first
__device__ __forceinline__ void split2(float x, float y, uint32_t (&t)[kTerms]) {
#pragma unroll
  for (int i = 0; i < kTerms; ++i) {
    t[i] = pack2<bf16>(x, y);
    float hx, hy;
    Num<bf16>::unpack2(t[i], hx, hy);
    x -= hx;
    y -= hy;
  }
}
template <int N = kTerms>
__device__ __forceinline__ void split_store(bf16* dst, int term_pitch, float x) {
#pragma unroll
  for (int i = 0; i < N; ++i) {
    const bf16 h = __float2bfloat16_rn(x);
    dst[i * term_pitch] = h;
    x -= __bfloat162float(h);
  }
}
// d += a b over term pairs (i, j) with i + j < kTerms, small products first
template <int NA>
__device__ __forceinline__ void mma_terms(float (&d)[4], const uint32_t (&a)[NA][4], const uint32_t (&b0)[kTerms],
                                          const uint32_t (&b1)[kTerms]) {
#pragma unroll
  for (int sum = kTerms - 1; sum >= 0; --sum)
#pragma unroll
    for (int i = 0; i <= sum && i < NA; ++i)
      mma16816<bf16>(d, a[i][0], a[i][1], a[i][2], a[i][3], b0[sum - i], b1[sum - i]);
}

__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(dst))), "l"(src)
               : "memory");
}

// Gates by the special-function unit: a few units in the last place of fp32.
__device__ __forceinline__ float gate(float raw, float bias, float low) {
  return low + (1.0f - low) * __fdividef(1.0f, 1.0f + __expf(-(raw + bias)));
}
__device__ __forceinline__ float silu(float x) { return x * __fdividef(1.0f, 1.0f + __expf(-x)); }

template <int CP>
struct Smem {
  static constexpr int kPitchC = CP + 8;      // bf16 rows of q", k"
  static constexpr int kPitchE = kMaxE + 8;   // bf16 rows of v
  static constexpr int kPitchA = kBlock + 8;  // bf16 rows of A
  alignas(16) float raw[2][kBlock * (2 * CP + kMaxE)];    // q, f, v of a block as they arrive
  alignas(16) float q[kBlock][CP];
  alignas(16) float f[kBlock][CP];
  alignas(16) float bias[CP];
  alignas(16) float low[CP];
  alignas(16) float F[2][CP];
  alignas(16) float w[kMaxE];
  float o[2][kBlock][kMaxE + 4];  // per half of the channels
  alignas(16) bf16 qd[2][kTerms][kBlock * kPitchC];
  alignas(16) bf16 kd[2][kTerms][kBlock * kPitchC];
  alignas(16) bf16 v[2][2][kBlock * kPitchE];
  alignas(16) bf16 a[2][kTerms][kBlock * kPitchA];
};

// Grid (segments, heads, sequences).  FULL: outputs and the sequence's final state; otherwise the segment's contribution.
template <typename T, int CP, bool FULL>
__global__ void __launch_bounds__(kThreads, 1) hgrn2_blocks_kernel(const Hgrn2Params p, const Segments sg) {
  constexpr int kTiles = CP / 16;  // 8-column tiles of S^T of a warp
  constexpr int kVTerms = sizeof(T) == 2 && std::is_same<T, bf16>::value ? 1 : 2;
  extern __shared__ __align__(16) uint8_t hb_smem[];
  Smem<CP>& sm = *reinterpret_cast<Smem<CP>*>(hb_smem);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int seg = blockIdx.x, h = blockIdx.y, b = blockIdx.z, H = p.H, C = p.C, E = p.E;
  const int64_t bh = static_cast<int64_t>(b) * H + h, all_bh = static_cast<int64_t>(gridDim.z) * H;
  const int s_begin = seg * sg.tokens;
  const int s_end = seg == sg.count - 1 ? p.S : s_begin + sg.tokens;
  const int e0 = (warp & 7) * 16, half = warp >> 3, c0 = half * (CP / 2);
  const bool live = e0 < E;
  const int er = e0 + (lane >> 2), cc = 2 * (lane & 3);  // this thread's first row and column in a tile of S^T

  for (int c = tid; c < CP; c += kThreads) {
    sm.bias[c] = c < C ? Num<T>::to_f(static_cast<const T*>(p.f_bias)[h * C + c]) : 0.f;
    sm.low[c] = c < C ? Num<T>::to_f(static_cast<const T*>(p.lower)[h * C + c]) : 0.f;
  }
  for (int e = tid; e < E; e += kThreads) sm.w[e] = Num<T>::to_f(static_cast<const T*>(p.norm_w)[e]);
  static_assert(kWarps == kBlock && kThreads == 4 * 128, "work is dealt to warps by token and to threads by channel");
  // channels past C stay zero in the arrays that the products read
  if (C < CP)
    for (int i = tid; i < 2 * kTerms * kBlock * Smem<CP>::kPitchC; i += kThreads) {
      (&sm.qd[0][0][0])[i] = __float2bfloat16_rn(0.f);
      (&sm.kd[0][0][0])[i] = __float2bfloat16_rn(0.f);
    }
  pdl_launch_dependents();
  pdl_wait();

  // warp t works on token t of a block, a lane on 4 consecutive channels (or values)
  const int x4 = lane * 4;
  auto fetch = [&](int s0, int buf) {
    if (s0 + warp < s_end) {
      const float* row = p.proj + (static_cast<int64_t>(b) * p.S + s0 + warp) * p.ld + x4;
      float* dst = sm.raw[buf] + warp * (2 * CP + kMaxE) + x4;
      if (x4 < C) {
        if (FULL) cp_async16(dst, row + p.q_off + h * C);
        cp_async16(dst + CP, row + p.f_off + h * C);
      }
      if (x4 < E) cp_async16(dst + 2 * CP, row + p.v_off + h * E);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };

  // ---- state before the segment ----
  float st[kTiles][4];
#pragma unroll
  for (int n = 0; n < kTiles; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) st[n][e] = 0.f;
  const bool fresh = load_pos(p.input_pos, p.pos_is_i64, 0) <= 0;
  auto each = [&](auto fn) {  // fn(register, channel, row of E)
#pragma unroll
    for (int n = 0; n < kTiles; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int c = c0 + n * 8 + cc + (e & 1), row = er + (e >> 1) * 8;
        if (live && c < C) fn(st[n][e], c, row);
      }
  };
  const int64_t mat = static_cast<int64_t>(C) * E;
  if (seg == 0) {
    const float* src = FULL && sg.count > 1 ? sg.init + bh * mat : p.state + bh * mat;
    const bool zero = fresh && !(FULL && sg.count > 1);
    each([&](float& x, int c, int row) { x = zero ? 0.f : src[static_cast<int64_t>(c) * E + row]; });
    if (!FULL) each([&](float& x, int c, int row) { sg.init[bh * mat + static_cast<int64_t>(c) * E + row] = x; });
  } else if (FULL) {
    for (int i = 0; i < seg; ++i) {
      const float* src = sg.part + (i * all_bh + bh) * mat;
      const float* dec = sg.decay + (i * all_bh + bh) * C;
      if (i == 0)
        each([&](float& x, int c, int row) { x = src[static_cast<int64_t>(c) * E + row]; });
      else
        each([&](float& x, int c, int row) { x = fmaf(dec[c], x, src[static_cast<int64_t>(c) * E + row]); });
    }
  }
  float decay = 1.f;  // thread c: product of all gates of the segment (first pass)

  // ---- steps of a block; buf = parity of the block ----
  // gates, activations, v terms (each thread reads what it fetched itself)
  auto gates = [&](int s0, int buf) {
    const bool in = s0 + warp < s_end;
    const float* rw = sm.raw[buf] + warp * (2 * CP + kMaxE) + x4;
    if (x4 < CP) {
      float4 f = make_float4(1.f, 1.f, 1.f, 1.f), q = make_float4(0.f, 0.f, 0.f, 0.f);
      if (in && x4 < C) {
        const float4 fr = *reinterpret_cast<const float4*>(rw + CP);
        const float4 bi = *reinterpret_cast<const float4*>(&sm.bias[x4]), lo = *reinterpret_cast<const float4*>(&sm.low[x4]);
        f.x = gate(fr.x, bi.x, lo.x), f.y = gate(fr.y, bi.y, lo.y), f.z = gate(fr.z, bi.z, lo.z), f.w = gate(fr.w, bi.w, lo.w);
        if (FULL) {
          const float4 qr = *reinterpret_cast<const float4*>(rw);
          q = make_float4(silu(qr.x), silu(qr.y), silu(qr.z), silu(qr.w));
        }
      }
      *reinterpret_cast<float4*>(&sm.f[warp][x4]) = f;
      if (FULL) *reinterpret_cast<float4*>(&sm.q[warp][x4]) = q;
    }
    if (x4 < E) {
      const float4 x = in ? *reinterpret_cast<const float4*>(rw + 2 * CP) : make_float4(0.f, 0.f, 0.f, 0.f);
      uint32_t lo[kTerms], hi[kTerms];
      split2(rnd<T>(x.x), rnd<T>(x.y), lo);
      split2(rnd<T>(x.z), rnd<T>(x.w), hi);
#pragma unroll
      for (int i = 0; i < kVTerms; ++i)
        *reinterpret_cast<uint2*>(&sm.v[buf][i][warp * Smem<CP>::kPitchE + x4]) = make_uint2(lo[i], hi[i]);
    }
  };
  auto products = [&](int buf) {
    // running products: thread (channel, k" or q", first or last 8 tokens)
    {
      constexpr int kH = kBlock / 2;
      const int c = tid & 127, part = tid >> 7, t0 = (part & 1) * kH;
      if (part < 2) {
        if (c < C) {
          float r = 1.f;
          if (t0 == 0)
#pragma unroll
            for (int t = kH; t < kBlock; ++t) r *= sm.f[t][c];
#pragma unroll
          for (int i = kH - 1; i >= 0; --i) {
            const float f = sm.f[t0 + i][c];
            split_store(&sm.kd[buf][0][(t0 + i) * Smem<CP>::kPitchC + c], kBlock * Smem<CP>::kPitchC, (1.f - f) * r);
            r *= f;
          }
          if (t0 == 0) {
            sm.F[buf][c] = r;
            decay *= r;
          }
        } else if (c < CP) {
          sm.F[buf][c] = 1.f;
        }
      } else if (FULL && c < C) {
        float r = 1.f;
        if (t0 > 0)
#pragma unroll
          for (int t = 0; t < kH; ++t) r *= sm.f[t][c];
#pragma unroll
        for (int i = 0; i < kH; ++i) {
          r *= sm.f[t0 + i][c];
          split_store(&sm.qd[buf][0][(t0 + i) * Smem<CP>::kPitchC + c], kBlock * Smem<CP>::kPitchC, sm.q[t0 + i][c] * r);
        }
      }
    }
    if (!FULL) return;
    // A[t, s]: warp s, lanes over channels
    constexpr int kPer = CP / 32;
    const int s = warp;
    float d[kPer] = {}, a[kBlock];
#pragma unroll
    for (int t = 0; t < kBlock; ++t) {
      float x = 0.f;
      if (t >= s) {
#pragma unroll
        for (int j = 0; j < kPer; j += 2) {
          const float2 f = *reinterpret_cast<const float2*>(&sm.f[t][lane * kPer + j]);
          const float2 q = *reinterpret_cast<const float2*>(&sm.q[t][lane * kPer + j]);
          d[j] = t == s ? 1.f - f.x : d[j] * f.x;
          d[j + 1] = t == s ? 1.f - f.y : d[j + 1] * f.y;
          x = fmaf(q.x, d[j], x);
          x = fmaf(q.y, d[j + 1], x);
        }
      }
      a[t] = x;
    }
    // sums over the lanes: each exchange halves the values a lane holds
    int t_mine = 0;
#pragma unroll
    for (int n = kBlock / 2, o = 16; n >= 1; n >>= 1, o >>= 1) {
      const bool up = lane & o;
#pragma unroll
      for (int i = 0; i < n; ++i) {
        const float give = up ? a[i] : a[i + n];
        a[i] = (up ? a[i + n] : a[i]) + __shfl_xor_sync(0xffffffffu, give, o);
      }
      t_mine = t_mine * 2 + (up ? 1 : 0);
    }
    a[0] += __shfl_xor_sync(0xffffffffu, a[0], 1);
    if ((lane & 1) == 0) split_store(&sm.a[buf][0][t_mine * Smem<CP>::kPitchA + s], kBlock * Smem<CP>::kPitchA, a[0]);
  };
  auto tensor = [&](int buf) {
    if (live) {
      // V^T: rows of E, 16 tokens deep
      uint32_t va[kVTerms][4];
#pragma unroll
      for (int i = 0; i < kVTerms; ++i)
        ldmatrix_x4_trans(&sm.v[buf][i][((lane & 7) + ((lane >> 4) & 1) * 8) * Smem<CP>::kPitchE + e0 + ((lane >> 3) & 1) * 8], va[i][0],
                          va[i][1], va[i][2], va[i][3]);
      if (FULL) {
        float o[2][4] = {};
#pragma unroll
        for (int k = 0; k < CP / 32; ++k) {
          uint32_t sa[kTerms][4];
#pragma unroll
          for (int r = 0; r < 4; ++r) {
            uint32_t t3[kTerms];
            split2(st[2 * k + (r >> 1)][(r & 1) * 2], st[2 * k + (r >> 1)][(r & 1) * 2 + 1], t3);
#pragma unroll
            for (int i = 0; i < kTerms; ++i) sa[i][r] = t3[i];
          }
          uint32_t b[kTerms][4];  // tokens 0-7: [0], [1]; tokens 8-15: [2], [3]
#pragma unroll
          for (int i = 0; i < kTerms; ++i)
            ldmatrix_x4(&sm.qd[buf][i][((lane & 7) + (lane >> 4) * 8) * Smem<CP>::kPitchC + c0 + k * 16 + ((lane >> 3) & 1) * 8], b[i][0], b[i][1],
                        b[i][2], b[i][3]);
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            uint32_t b0[kTerms], b1[kTerms];
#pragma unroll
            for (int i = 0; i < kTerms; ++i) b0[i] = b[i][2 * n], b1[i] = b[i][2 * n + 1];
            mma_terms(o[n], sa, b0, b1);
          }
        }
        {
          uint32_t b[kTerms][4];
#pragma unroll
          for (int i = 0; i < kTerms; ++i)
            ldmatrix_x4(&sm.a[buf][i][((lane & 7) + (lane >> 4) * 8) * Smem<CP>::kPitchA + ((lane >> 3) & 1) * 8], b[i][0], b[i][1], b[i][2],
                        b[i][3]);
          // each half of the channels adds this product for half of the tokens
          uint32_t b0[kTerms], b1[kTerms];
#pragma unroll
          for (int i = 0; i < kTerms; ++i) b0[i] = half ? b[i][2] : b[i][0], b1[i] = half ? b[i][3] : b[i][1];
          if (half)
            mma_terms(o[1], va, b0, b1);
          else
            mma_terms(o[0], va, b0, b1);
        }
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) sm.o[half][n * 8 + cc + (e & 1)][er + (e >> 1) * 8] = o[n][e];
      }
      // ---- state update ----
#pragma unroll
      for (int k = 0; k < CP / 32; ++k) {
        uint32_t b[kTerms][4];  // channels c0 + 16 k .. + 7: [0], [1]; + 8 ..: [2], [3]
#pragma unroll
        for (int i = 0; i < kTerms; ++i)
          ldmatrix_x4_trans(&sm.kd[buf][i][(lane & 15) * Smem<CP>::kPitchC + c0 + k * 16 + (lane >> 4) * 8], b[i][0], b[i][1], b[i][2], b[i][3]);
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          const float2 F = *reinterpret_cast<const float2*>(&sm.F[buf][c0 + k * 16 + n * 8 + cc]);
          float(&s)[4] = st[2 * k + n];
          s[0] *= F.x, s[1] *= F.y, s[2] *= F.x, s[3] *= F.y;
          uint32_t b0[kTerms], b1[kTerms];
#pragma unroll
          for (int i = 0; i < kTerms; ++i) b0[i] = b[i][2 * n], b1[i] = b[i][2 * n + 1];
          mma_terms(s, va, b0, b1);
        }
      }
    }
  };
  // RMSNorm over E, one token per warp
  auto norm = [&](int s0) {
        const int t = warp;
    if (s0 + t < s_end) {
      float x[4], ss = 0.f;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int e = lane * 4 + j;
        x[j] = e < E ? sm.o[0][t][e] + sm.o[1][t][e] : 0.f;
        ss += x[j] * x[j];
      }
      const float inv = 1.0f / sqrtf(warp_sum(ss) / static_cast<float>(E) + p.eps);
      if (lane * 4 < E) {
        T* dst = static_cast<T*>(p.out) + ((static_cast<int64_t>(b) * p.S + s0 + t) * H + h) * E + lane * 4;
        uint2 v;
        v.x = pack2<T>(x[0] * inv * sm.w[x4], x[1] * inv * sm.w[x4 + 1]);
        v.y = pack2<T>(x[2] * inv * sm.w[x4 + 2], x[3] * inv * sm.w[x4 + 3]);
        *reinterpret_cast<uint2*>(dst) = v;
      }
    }
  };

  // Two barriers a block: while the tensor products of block i run, the gates of block i + 1 are taken (half of the warps
  // begin with the one, half with the other); then the running products of block i + 1 beside the norm of block i.
  auto wait_fetched = [] { asm volatile("cp.async.wait_group 1;" ::: "memory"); };
  fetch(s_begin, 0);
  fetch(s_begin + kBlock, 1);
  wait_fetched();
  __syncthreads();  // bias, low
  gates(s_begin, 0);
  __syncthreads();
  products(0);
  __syncthreads();
  int buf = 0;
  for (int s0 = s_begin; s0 < s_end; s0 += kBlock, buf ^= 1) {
    const bool more = s0 + kBlock < s_end;
    fetch(s0 + 2 * kBlock, buf);
    wait_fetched();
#pragma unroll 1
    for (int turn = 0; turn < 2; ++turn) {
      if ((turn ^ (warp & 1)) == 0) {
        if (more) gates(s0 + kBlock, buf ^ 1);
      } else {
        tensor(buf);
      }
    }
    __syncthreads();
    if (more) products(buf ^ 1);
    if (FULL) norm(s0);
    __syncthreads();
  }
  if (FULL) {
    if (seg == sg.count - 1)
      each([&](float& x, int c, int row) { p.state[bh * mat + static_cast<int64_t>(c) * E + row] = x; });
  } else {
    each([&](float& x, int c, int row) { sg.part[(seg * all_bh + bh) * mat + static_cast<int64_t>(c) * E + row] = x; });
    if (tid < C) sg.decay[(seg * all_bh + bh) * C + tid] = decay;  // (part 0: threads of the first 8 tokens)
  }
}

// Segments wanted: as many CTAs as SMs.  Grows with S, so that the workspace of a longer call serves a shorter one.
int64_t wanted_segments(int B, int S, int H) {
  int64_t n = device_sm_count() / (static_cast<int64_t>(B) * H);
  n = n > kMaxSegments ? kMaxSegments : n;
  n = n > S / kMinSegment ? S / kMinSegment : n;
  return n < 1 ? 1 : n;
}

Segments plan(int B, int S, int H) {
  Segments s{};
  const int64_t n = wanted_segments(B, S, H);
  int tokens = static_cast<int>((S + n - 1) / n);
  tokens = (tokens + kBlock - 1) / kBlock * kBlock;
  s.tokens = tokens;
  s.count = (S + tokens - 1) / tokens;
  return s;
}

template <typename T, int CP>
int launch(const Hgrn2Params& p, const Segments& sg, int B, cudaStream_t st) {
  constexpr int smem = static_cast<int>(sizeof(Smem<CP>));
  auto full = hgrn2_blocks_kernel<T, CP, true>;
  auto part = hgrn2_blocks_kernel<T, CP, false>;
  static std::atomic<unsigned long long> full_set{0}, part_set{0};
  LRI_ONCE_PER_DEVICE(full_set, cudaFuncSetAttribute(full, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
  LRI_ONCE_PER_DEVICE(part_set, cudaFuncSetAttribute(part, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
  if (sg.count > 1) {
    LRI_CUDA(launch_pdl(part, dim3(sg.count - 1, p.H, B), dim3(kThreads), static_cast<size_t>(smem), st, p, sg));
    LRI_LAUNCH_CHECK("hgrn2_blocks_kernel<part>");
  }
  LRI_CUDA(launch_pdl(full, dim3(sg.count, p.H, B), dim3(kThreads), static_cast<size_t>(smem), st, p, sg));
  LRI_LAUNCH_CHECK("hgrn2_blocks_kernel");
  return LRI_OK;
}

}  // namespace

bool hgrn2_blocks_supports(int dtype, const Hgrn2Params& p, int B) {
  if (dtype != LRI_BF16 && dtype != LRI_FP16) return false;
  if (p.S < kBlock || p.C > 128 || p.C % 4 || p.E > kMaxE || p.E % 16) return false;
  return p.ld % 4 == 0 && p.q_off % 4 == 0 && p.f_off % 4 == 0 && p.v_off % 4 == 0 && aligned16(p.proj) && aligned16(p.out) && B <= 65535;
}

size_t hgrn2_blocks_workspace_bytes(int B, int S, int H, int C, int E) {
  const int64_t n = wanted_segments(B, S, H);
  if (n < 2) return 0;
  return static_cast<size_t>(B) * H * C * (static_cast<size_t>(n) * E + n - 1) * sizeof(float);
}

int hgrn2_blocks_launch(int dtype, const Hgrn2Params& p, int B, void* workspace, cudaStream_t st) {
  Segments sg = plan(B, p.S, p.H);
  const size_t mat = static_cast<size_t>(B) * p.H * p.C * p.E;
  sg.init = static_cast<float*>(workspace);
  sg.part = sg.init + mat;
  sg.decay = sg.part + mat * (sg.count - 1);
  const bool bf = dtype == LRI_BF16;
  if (p.C <= 64) return bf ? launch<bf16, 64>(p, sg, B, st) : launch<__half, 64>(p, sg, B, st);
  return bf ? launch<bf16, 128>(p, sg, B, st) : launch<__half, 128>(p, sg, B, st);
}

}  // namespace lri
