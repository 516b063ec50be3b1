// What the forms of gated linear attention share: their parameters, the token range a block works on, and
// the decay of a key channel.
#pragma once
#include "common.cuh"

namespace leone {

struct GlaParams {
  const float* proj;           // [n_tokens, ld]
  int ld, q_off, k_off, v_off, u_off;
  const float* w2;             // [rank, heads * dim]: W_2 transposed
  const float* w2_bias;        // [heads * dim]
  int rank;
  float inv_tau, q_scale;
  float* state;                // [n_slots, heads, dim, vdim]
  const int* q_start;
  const int* slot_ids;
  int heads, dim, vdim, chunk, n_seqs, n_slots;
  float* chunk_state;          // [chunks, heads, dim, vdim]
  float* chunk_decay;          // [chunks, heads, dim]
  float* out;                  // fp32 [n_tokens, ldo], or null with `gated`
  int ldo;
  void* gated;                 // run dtype [n_tokens, ldg]: the finished heads
  int ldg;
  const float* norm_w;         // [vdim]
  int gate_off, gate_act;      // columns of proj; 0 sigmoid, 1 silu
  float eps;
  int* status;
};

// The (sequence, chunk) pair a block works on, its token range, and whether it is the sequence's last (P: parameters with
// chunk, n_seqs and q_start).
struct GlaSpan { int seq, t0, t1, last; };

template <typename P> __device__ __forceinline__ bool gla_span(const P& p, int z, GlaSpan& sp) {
  if (p.chunk <= 0) {
    sp.seq = z;
    sp.t0 = p.q_start[z];
    sp.t1 = p.q_start[z + 1];
    sp.last = 1;
    return sp.t0 < sp.t1;
  }
  for (int b = 0; b < p.n_seqs; ++b) {
    const int first = p.q_start[b], end = p.q_start[b + 1];
    const int nc = (end - first + p.chunk - 1) / p.chunk;
    if (z < nc) {
      sp.seq = b;
      sp.t0 = first + z * p.chunk;
      sp.t1 = min(end, sp.t0 + p.chunk);
      sp.last = sp.t1 == end;
      return true;
    }
    z -= nc;
  }
  return false;
}

// sigmoid(z)^(1/tau) = exp(-softplus(-z) / tau)
__device__ __forceinline__ float channel_decay(float z, float inv_tau) {
  const float sp = z < -20.f ? -z : log1pf(expf(-z));
  return expf(-sp * inv_tau);
}

// The pass over a sequence's chunks (gated_linear_attention.cu): chunk_state from contributions to start states.
int launch_gla_prefix(const GlaParams& p, cudaStream_t stream);

}  // namespace leone
