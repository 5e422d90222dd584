// Parameters shared by the two forms of the HGRN2 mixer.
#pragma once

#include "common.cuh"

namespace lri {

struct Hgrn2Params {
  const float* proj;  // [B * S, ld]: q_raw at q_off, f_raw at f_off, v at v_off
  int64_t ld, q_off, f_off, v_off;
  const void* f_bias;  // [H * C]
  const void* lower;   // [H * C]
  const void* norm_w;  // [E]
  float eps;
  float* state;        // [B_max, H, C, E]
  const void* input_pos;
  int pos_is_i64;
  void* out;     // [B * S, H * E]
  float* o_raw;  // [B * S, H * E] when the columns of a head are cut over CTAs, else NULL
  int S, H, C, E;
};

__device__ __forceinline__ float forget_gate(float raw, float bias, float low) {
  return low + (1.0f - low) * sigmoid_f(raw + bias);
}

// Prompt form: blocks of tokens on tensor cores (hgrn2_blocks.cu)
bool hgrn2_blocks_supports(int dtype, const Hgrn2Params& p, int B);
size_t hgrn2_blocks_workspace_bytes(int B, int S, int H, int C, int E);
int hgrn2_blocks_launch(int dtype, const Hgrn2Params& p, int B, void* workspace, cudaStream_t st);

}  // namespace lri
