// What the forms of the Mamba-2 recurrence share: their parameters and a token's step and decay.
#pragma once
#include "common.cuh"

namespace leone {

struct SsdParams {
  const void* act;             // [n_tokens, lda]: x, B and C after their convolution
  int lda, x_off, b_off, c_off;
  const void* raw;             // [n_tokens, ldr], run dtype: one dt per head at dt_off
  int ldr, dt_off;
  const float* a_log;          // [heads]
  const float* dt_bias;        // [heads]
  const float* d_skip;         // [heads]
  float* out;                  // [n_tokens, ldo], head h at columns h * vdim
  int ldo;
  float* state;                // [n_slots, heads, n_state, vdim]
  const int* q_start;
  const int* slot_ids;
  int n_seqs, heads, groups, n_state, vdim, n_slots;
  int* status;
  int chunk;                   // 0: sequences are not cut
  float* chunk_state;          // [chunks, heads, n_state, vdim]
  float* chunk_decay;          // [chunks, heads, n_state], equal along n_state
};

// softplus(dt + bias), no clamp
__device__ __forceinline__ float ssd_step(float raw, float bias) {
  const float z = raw + bias;
  return z > 20.f ? z : log1pf(expf(z));
}

}  // namespace leone
