// Parameters shared by the forms of sliding-window attention.
#pragma once

#include "common.cuh"

namespace lri {

struct WindowParams {
  const void* q;  // [d1 | d2] at q + row * q_row + head * q_head
  int64_t q_row, q_head;
  const void* k;  // d1 elements at k + b * k_batch + j * k_row + head * k_head
  int64_t k_batch, k_row, k_head;
  const void* k2;  // d2 elements at k2 + b * k2_batch + j * k2_row, shared by the heads
  int64_t k2_batch, k2_row;
  const void* v;  // dv elements
  int64_t v_batch, v_row, v_head;
  void* out;  // [rows, H * dv]
  const void* input_pos;
  int pos_is_i64;
  int history;  // key row j holds position pos0 - history + j; history < 0: position j
  int64_t k_rows;
  int64_t window;
  float scale;
  int S, H, d1, d2, dv;
};

// Prompt form on the fifth-generation tensor cores (latent_attention_tc.cu).
bool window_attention_tc_supports(int dtype, const WindowParams& p, int B);
int window_attention_tc_launch(int dtype, const WindowParams& p, int B, cudaStream_t st);
int window_attention_tc_status_read_and_clear(int* status_out);

// Single-token form on keys and values shared by the heads (latent_decode.cu); scratch holds split partial results.
bool latent_decode_supports(int dtype, const WindowParams& p);
size_t latent_decode_scratch_bytes(int B, int H, int dv, int64_t keys);
int latent_decode_launch(int dtype, const WindowParams& p, int B, void* scratch, size_t scratch_bytes, cudaStream_t st);

}  // namespace lri
