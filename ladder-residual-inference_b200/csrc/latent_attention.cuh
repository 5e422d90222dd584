// Parameters shared by the forms of masked softmax attention: sliding windows and chunks, keys per head or shared by a
// group of query heads, keys gathered for the call or read from a cache, an optional sink in the denominator.
#pragma once

#include "common.cuh"

namespace lri {

struct WindowParams {
  const void* q;  // [d1 | d2] at q + row * q_row + head * q_head
  int64_t q_row, q_head;
  const void* k;  // d1 elements at k + b * k_batch + j * k_row + (head / group) * k_head
  int64_t k_batch, k_row, k_head;
  const void* k2;  // d2 elements at k2 + b * k2_batch + j * k2_row, shared by the heads (d2 = 0: none)
  int64_t k2_batch, k2_row;
  const void* v;  // dv elements
  int64_t v_batch, v_row, v_head;
  int group;  // query heads per key head
  void* out;  // row pitch out_ld, heads of dv
  int64_t out_ld;
  float out_scale;
  const void* input_pos;
  int pos_is_i64;
  int history;  // key row j holds position pos0 - history + j; history < 0: position j
  int64_t k_rows;
  int64_t window;
  int64_t chunk;     // > 0: a query sees only keys of its own chunk of positions
  const void* sink;  // [H] or NULL: exp(sink) joins the denominator
  float scale;
  int S, H, d1, d2, dv;
};

// First position that a query at position pos sees
__host__ __device__ __forceinline__ int64_t first_visible(int64_t pos, int64_t window, int64_t chunk) {
  int64_t lo = pos - window + 1;
  if (chunk > 0) {
    const int64_t c = pos / chunk * chunk;
    lo = lo > c ? lo : c;
  }
  return lo > 0 ? lo : 0;
}

// Prompt form on the fifth-generation tensor cores (latent_attention_tc.cu).
bool window_attention_tc_supports(int dtype, const WindowParams& p, int B);
int window_attention_tc_launch(int dtype, const WindowParams& p, int B, cudaStream_t st);
int window_attention_tc_status_read_and_clear(int* status_out);

// Single-token form on keys and values shared by the heads (latent_decode.cu); scratch holds split partial results.
bool latent_decode_supports(int dtype, const WindowParams& p);
size_t latent_decode_scratch_bytes(int B, int H, int dv, int64_t keys);
int latent_decode_launch(int dtype, const WindowParams& p, int B, void* scratch, size_t scratch_bytes, cudaStream_t st);

// Single-token form on a cache of grouped keys (attention_cluster.cu).
bool attn_decode_masked_supports(int dtype, const WindowParams& p);
int attn_decode_masked_launch(int dtype, const WindowParams& p, int B, cudaStream_t st);

// Any size and type, one warp per (token, head) (latent_attention.cu).
int window_attention_plain_launch(int dtype, const WindowParams& p, int64_t rows, cudaStream_t st);

}  // namespace lri
