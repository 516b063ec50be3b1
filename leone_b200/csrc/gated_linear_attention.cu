// Gated linear attention: a recurrence whose state rows decay each at its own rate, token by token.
//
//   per head, S: [dim, vdim] fp32, per request:
//     S_t = diag(alpha_t) S_(t-1) + k_t v_t^T          alpha_t: [dim], one factor per key channel
//     o_t = S_t^T q_t
//     alpha_t = sigmoid(z_t)^(1/tau),  z_t = W_2 u_t + b   (u: a low-rank projection of the token)
//
// q (times `q_scale`), k, v and u arrive as columns of one fp32 projection.  Everything here is fp32.  The
// state is read from and written back to the request's state slot, so a sequence may be cut into steps
// anywhere; a step of one token per sequence (decode) is the same walk.
//
// The walk: a block owns (a slice of value columns, head, sequence); a thread keeps DPT rows x VPT value
// columns of the state in registers, 16 tokens are staged in shared memory at a time (their decay factors
// are formed there), and the partial read-outs of the row groups are summed through shared memory.  Long
// prompt portions run chunk-parallel: every chunk but the last sums its own contributions from a zero state
// and the product of its decays, a pass over the chunks turns those into the state at each chunk's start,
// then every chunk walks its tokens from there.
//
// Where one block holds all of a head's value columns, it also finishes the head: RMS norm over vdim,
// weight, times act(gate), stored in the run dtype.
#include "common.cuh"
#include "gla_parts.cuh"

namespace leone {

constexpr int kGlaTokens = 16;
constexpr int kGlaLanes = 32;

// OUT: outputs written, the walk starts from the chunk's (or the slot's) state; else the chunk's own
// contribution from a zero state.  T: dtype of the finished heads.
template <typename T, int DPT, int VPT, bool OUT>
__global__ void __launch_bounds__(256)
gla_walk_kernel(const GlaParams p) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ __align__(16) float smem[];
  constexpr int VW = kGlaLanes * VPT;
  const int dim = p.dim, vdim = p.vdim, heads = p.heads;
  const int DP = blockDim.y;
  float* q_s = smem;                               // [tokens][dim]
  float* k_s = q_s + kGlaTokens * dim;             // [tokens][dim]
  float* a_s = k_s + kGlaTokens * dim;             // [tokens][dim]
  float* v_s = a_s + kGlaTokens * dim;             // [tokens][VW]
  float* part = v_s + kGlaTokens * VW;             // [DP][tokens][VW]
  float* u_s = part + DP * kGlaTokens * VW;        // [rank][tokens]
  const int tx = threadIdx.x, ty = threadIdx.y;
  const int tid = ty * kGlaLanes + tx, nthreads = kGlaLanes * DP;
  const int h = blockIdx.y, v0 = blockIdx.x * VW;
  GlaSpan sp;
  if (!gla_span(p, blockIdx.z, sp)) return;
  if (!OUT && sp.last) return;                     // the last chunk's contribution is never needed
  const int slot = p.slot_ids[sp.seq];
  if (slot < 0 || slot >= p.n_slots) {
    if (tid == 0) set_status(p.status, kBadSequence, sp.seq, slot);
    return;
  }
  const size_t per_head = (size_t)dim * vdim;
  float* slot_state = p.state + ((size_t)slot * heads + h) * per_head;
  float* mine = p.chunk > 0 ? p.chunk_state + ((size_t)blockIdx.z * heads + h) * per_head : slot_state;
  const float* s_in = OUT ? mine : nullptr;
  float* s_out = !OUT ? mine : (sp.last ? slot_state : nullptr);
  const int d_per = (dim + DP - 1) / DP, d0 = ty * d_per;
  const int c0 = v0 + tx * VPT;                    // this thread's first value column
  const bool vec = VPT == 4 && vdim % 4 == 0;
  float S[DPT][VPT];
#pragma unroll
  for (int i = 0; i < DPT; ++i) {
    const int d = d0 + i;
    const bool row = s_in != nullptr && i < d_per && d < dim;
    if (vec) {
      const float4 x = row && c0 < vdim ? *reinterpret_cast<const float4*>(s_in + (size_t)d * vdim + c0) : make_float4(0.f, 0.f, 0.f, 0.f);
      const float xs[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
      for (int j = 0; j < VPT; ++j) S[i][j] = xs[j & 3];
    } else {
#pragma unroll
      for (int j = 0; j < VPT; ++j) S[i][j] = row && c0 + j < vdim ? s_in[(size_t)d * vdim + c0 + j] : 0.f;
    }
  }
  float decay[2] = {1.f, 1.f};                     // product of the chunk's factors, channels tid and tid + nthreads
  const int hd = heads * dim;
  for (int tb = sp.t0; tb < sp.t1; tb += kGlaTokens) {
    const int nt = min(kGlaTokens, sp.t1 - tb);
    __syncthreads();
    for (int i = tid; i < nt * dim; i += nthreads) {
      const int tt = i / dim, d = i - tt * dim;
      const float* row = p.proj + (size_t)(tb + tt) * p.ld + (size_t)h * dim + d;
      if (OUT) q_s[i] = row[p.q_off] * p.q_scale;
      k_s[i] = row[p.k_off];
    }
    for (int i = tid; i < nt * VW; i += nthreads) {
      const int tt = i / VW, vv = i - tt * VW;
      v_s[i] = v0 + vv < vdim ? p.proj[(size_t)(tb + tt) * p.ld + p.v_off + (size_t)h * vdim + v0 + vv] : 0.f;
    }
    for (int i = tid; i < kGlaTokens * p.rank; i += nthreads) {
      const int tt = i / p.rank, r = i - tt * p.rank;
      u_s[r * kGlaTokens + tt] = tt < nt ? p.proj[(size_t)(tb + tt) * p.ld + p.u_off + r] : 0.f;
    }
    __syncthreads();
    // decay factors: a channel and eight tokens at a time
    for (int i = tid; i < dim * ((nt + 7) / 8); i += nthreads) {
      const int g = i / dim, c = i - g * dim;
      float z[8];
      const float b = p.w2_bias[(size_t)h * dim + c];
#pragma unroll
      for (int j = 0; j < 8; ++j) z[j] = b;
      const float* wr = p.w2 + (size_t)h * dim + c;
#pragma unroll 16
      for (int r = 0; r < p.rank; ++r) {
        const float w = wr[(size_t)r * hd];
        const float4 ua = *reinterpret_cast<const float4*>(u_s + r * kGlaTokens + g * 8);
        const float4 ub = *reinterpret_cast<const float4*>(u_s + r * kGlaTokens + g * 8 + 4);
        z[0] = fmaf(w, ua.x, z[0]); z[1] = fmaf(w, ua.y, z[1]); z[2] = fmaf(w, ua.z, z[2]); z[3] = fmaf(w, ua.w, z[3]);
        z[4] = fmaf(w, ub.x, z[4]); z[5] = fmaf(w, ub.y, z[5]); z[6] = fmaf(w, ub.z, z[6]); z[7] = fmaf(w, ub.w, z[7]);
      }
#pragma unroll
      for (int j = 0; j < 8; ++j)
        if (g * 8 + j < nt) a_s[(g * 8 + j) * dim + c] = channel_decay(z[j], p.inv_tau);
    }
    __syncthreads();
    if (!OUT) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int d = tid + e * nthreads;
        if (d < dim)
          for (int tt = 0; tt < nt; ++tt) decay[e] *= a_s[tt * dim + d];
      }
    }
    for (int tt = 0; tt < nt; ++tt) {
      float vt[VPT], acc[VPT];
#pragma unroll
      for (int j = 0; j < VPT; ++j) {
        vt[j] = v_s[tt * VW + tx * VPT + j];
        acc[j] = 0.f;
      }
      const float* kk = k_s + tt * dim + d0;
      const float* qq = q_s + tt * dim + d0;
      const float* aa = a_s + tt * dim + d0;
#pragma unroll
      for (int i = 0; i < DPT; ++i) {
        if (i < d_per && d0 + i < dim) {
          const float kv = kk[i], av = aa[i];
#pragma unroll
          for (int j = 0; j < VPT; ++j) S[i][j] = fmaf(av, S[i][j], kv * vt[j]);
          if (OUT) {
            const float qv = qq[i];
#pragma unroll
            for (int j = 0; j < VPT; ++j) acc[j] = fmaf(S[i][j], qv, acc[j]);
          }
        }
      }
      if (OUT) {
#pragma unroll
        for (int j = 0; j < VPT; ++j) part[(ty * kGlaTokens + tt) * VW + tx * VPT + j] = acc[j];
      }
    }
    if (OUT) {
      __syncthreads();
      // a row group's warp per token in turn: the sum over row groups, and the head's norm and gate
      for (int tt = ty; tt < nt; tt += DP) {
        const size_t t = tb + tt;
        float o[VPT], ss = 0.f;
#pragma unroll
        for (int j = 0; j < VPT; ++j) {
          const int vv = tx + j * kGlaLanes;
          float sum = 0.f;
          for (int g = 0; g < DP; ++g) sum += part[(g * kGlaTokens + tt) * VW + vv];
          o[j] = sum;
          ss = fmaf(sum, sum, ss);                 // columns past vdim hold zeros
          if (p.out != nullptr && v0 + vv < vdim) p.out[t * p.ldo + (size_t)h * vdim + v0 + vv] = sum;
        }
        if (p.gated != nullptr) {
          ss = warp_sum(ss);
          const float r = 1.f / sqrtf(ss / (float)vdim + p.eps);
#pragma unroll
          for (int j = 0; j < VPT; ++j) {
            const int vv = tx + j * kGlaLanes;
            if (vv < vdim) {
              const float z = p.proj[t * p.ld + p.gate_off + (size_t)h * vdim + vv];
              const float sg = 1.f / (1.f + expf(-z));
              reinterpret_cast<T*>(p.gated)[t * p.ldg + (size_t)h * vdim + vv] =
                  from_float<T>(o[j] * r * p.norm_w[vv] * (p.gate_act == 1 ? z * sg : sg));
            }
          }
        }
      }
    }
  }
  if (s_out != nullptr) {
#pragma unroll
    for (int i = 0; i < DPT; ++i) {
      const int d = d0 + i;
      if (i < d_per && d < dim) {
        if (vec) {
          if (c0 < vdim)
            *reinterpret_cast<float4*>(s_out + (size_t)d * vdim + c0) =
                make_float4(S[i][0], S[i][1 % VPT], S[i][2 % VPT], S[i][3 % VPT]);
        } else {
#pragma unroll
          for (int j = 0; j < VPT; ++j)
            if (c0 + j < vdim) s_out[(size_t)d * vdim + c0 + j] = S[i][j];
        }
      }
    }
  }
  if (!OUT && blockIdx.x == 0) {
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int d = tid + e * nthreads;
      if (d < dim) p.chunk_decay[((size_t)blockIdx.z * heads + h) * dim + d] = decay[e];
    }
  }
}

// The pass over a sequence's chunks: entry c of chunk_state holds chunk c's own contribution on entry and
// the state at chunk c's start on exit.  One thread per V state elements (V value columns of one row) walks
// the chunks in order, eight of them requested at a time.
template <int V>
__global__ void __launch_bounds__(128)
gla_prefix_kernel(const GlaParams p) {
  pdl_trigger();
  pdl_wait();
  constexpr int kAhead = 8;
  const int s = blockIdx.y;
  const size_t per_seq = (size_t)p.heads * p.dim * p.vdim;
  const size_t e = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * V;
  if (e >= per_seq) return;
  const int slot = p.slot_ids[s];
  if (slot < 0 || slot >= p.n_slots) return;
  int first = 0;
  for (int b = 0; b < s; ++b) first += (p.q_start[b + 1] - p.q_start[b] + p.chunk - 1) / p.chunk;
  const int nc = (p.q_start[s + 1] - p.q_start[s] + p.chunk - 1) / p.chunk;
  const size_t row = e / p.vdim;                   // head * dim + channel
  const size_t rows = (size_t)p.heads * p.dim;
  float run[V];
  const float* at0 = p.state + (size_t)slot * per_seq + e;
#pragma unroll
  for (int v = 0; v < V; ++v) run[v] = at0[v];
  for (int c0 = 0; c0 < nc; c0 += kAhead) {
    float own[kAhead][V], f[kAhead];
#pragma unroll
    for (int i = 0; i < kAhead; ++i) {             // (the last chunk's contribution is not there)
      const bool more = c0 + i + 1 < nc;
      const float* at = p.chunk_state + (size_t)(first + c0 + i) * per_seq + e;
      f[i] = more ? p.chunk_decay[(size_t)(first + c0 + i) * rows + row] : 0.f;
      if (V == 4) {
        const float4 x = more ? *reinterpret_cast<const float4*>(at) : make_float4(0.f, 0.f, 0.f, 0.f);
        own[i][0] = x.x; own[i][1 % V] = x.y; own[i][2 % V] = x.z; own[i][3 % V] = x.w;
      } else {
        own[i][0] = more ? at[0] : 0.f;
      }
    }
#pragma unroll
    for (int i = 0; i < kAhead; ++i) {
      if (c0 + i < nc) {
        float* at = p.chunk_state + (size_t)(first + c0 + i) * per_seq + e;
        if (V == 4) *reinterpret_cast<float4*>(at) = make_float4(run[0], run[1 % V], run[2 % V], run[3 % V]);
        else at[0] = run[0];
#pragma unroll
        for (int v = 0; v < V; ++v) run[v] = fmaf(f[i], run[v], own[i][v]);
      }
    }
  }
}

int launch_gla_prefix(const GlaParams& p, cudaStream_t stream) {
  const size_t per_seq = (size_t)p.heads * p.dim * p.vdim;
  if (p.vdim % 4 == 0)
    return launch_kernel(gla_prefix_kernel<4>, dim3((unsigned)((per_seq / 4 + 127) / 128), p.n_seqs), dim3(128), 0, stream, p);
  return launch_kernel(gla_prefix_kernel<1>, dim3((unsigned)((per_seq + 127) / 128), p.n_seqs), dim3(128), 0, stream, p);
}

}  // namespace leone

using namespace leone;

// proj: fp32 [n_tokens, ld] with q, k (heads x dim each), v (heads x vdim), u (rank) and the gate (heads x
// vdim) at their column offsets.  w2: fp32 [rank, heads * dim].  state: fp32 [n_slots, heads, dim, vdim].
// out: fp32 [n_tokens, ldo] or null; gated: `dtype` [n_tokens, ldg] or null (only with vdim <= 128: one block
// holds a head's columns): o / rms(o) * norm_w * act(gate), gate_act 0 sigmoid, 1 silu.  chunk == 0: one
// walk per sequence; chunk > 0: chunk-parallel with `n_chunks` = sum over sequences of ceil(len / chunk).
extern "C" int leone_gla(int dtype, const float* proj, int ld, int q_off, int k_off, int v_off, int u_off, int gate_off,
                         const float* w2, const float* w2_bias, int rank, float inv_tau, float q_scale, float* out,
                         int ldo, void* gated, int ldg, const float* norm_w, int gate_act, float eps, float* state,
                         const int* q_start, const int* slot_ids, int n_seqs, int heads, int dim, int vdim, int n_slots,
                         int chunk, int n_chunks, float* chunk_state, float* chunk_decay, int* status,
                         cudaStream_t stream) {
  if (n_seqs <= 0) return 0;
  if (heads <= 0 || dim <= 0 || vdim <= 0 || rank <= 0 || heads > 65535 || n_seqs > 65535 || dim > 512) return kRefusedSize;
  if (chunk < 0 || (chunk > 0 && (n_chunks <= 0 || n_chunks > 65535 || chunk_state == nullptr || chunk_decay == nullptr)))
    return kRefusedSize;
  if (dtype != 0 && dtype != 1) return kRefusedDtype;
  if (out == nullptr && gated == nullptr) return kRefusedSize;
  int dp = (dim + 15) / 16;                        // row groups of at most 16 rows each, up to 8 groups
  if (dp > 8) dp = 8;
  const int d_per = (dim + dp - 1) / dp;
  const int dpt = d_per <= 8 ? 8 : d_per <= 16 ? 16 : d_per <= 32 ? 32 : 64;
  const int vpt = dpt <= 16 ? (vdim > 64 ? 4 : vdim > 32 ? 2 : 1) : dpt == 32 ? (vdim > 32 ? 2 : 1) : 1;
  const int vw = kGlaLanes * vpt, slices = (vdim + vw - 1) / vw;
  if (gated != nullptr && (slices != 1 || norm_w == nullptr)) return kRefusedSize;
  const size_t smem = sizeof(float) * ((size_t)3 * kGlaTokens * dim + kGlaTokens * vw + (size_t)dp * kGlaTokens * vw +
                                       (size_t)kGlaTokens * rank);
  if (smem > 220 * 1024) return kRefusedSize;
  GlaParams p = {proj, ld, q_off, k_off, v_off, u_off, w2, w2_bias, rank, inv_tau, q_scale, state, q_start, slot_ids,
                 heads, dim, vdim, chunk, n_seqs, n_slots, chunk_state, chunk_decay, out, ldo, gated, ldg, norm_w,
                 gate_off, gate_act, eps, status};
  const dim3 block(kGlaLanes, dp);
  int code = 0;
#define WALK(T, D, V, GRIDZ, OUT)                                                                               \
  do {                                                                                                          \
    auto kern = gla_walk_kernel<T, D, V, OUT>;                                                                  \
    if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);   \
    code = launch_kernel(kern, dim3(slices, heads, GRIDZ), block, smem, stream, p);                             \
  } while (0)
#define WALK_D(T, GRIDZ, OUT)                          \
  do {                                                 \
    if (dpt == 8) {                                    \
      if (vpt == 4) WALK(T, 8, 4, GRIDZ, OUT);         \
      else if (vpt == 2) WALK(T, 8, 2, GRIDZ, OUT);    \
      else WALK(T, 8, 1, GRIDZ, OUT);                  \
    } else if (dpt == 16) {                            \
      if (vpt == 4) WALK(T, 16, 4, GRIDZ, OUT);        \
      else if (vpt == 2) WALK(T, 16, 2, GRIDZ, OUT);   \
      else WALK(T, 16, 1, GRIDZ, OUT);                 \
    } else if (dpt == 32) {                            \
      if (vpt == 2) WALK(T, 32, 2, GRIDZ, OUT);        \
      else WALK(T, 32, 1, GRIDZ, OUT);                 \
    } else {                                           \
      WALK(T, 64, 1, GRIDZ, OUT);                      \
    }                                                  \
  } while (0)
  const int grid_z = chunk > 0 ? n_chunks : n_seqs;
  if (chunk > 0) {
    WALK_D(float, grid_z, false);
    if (code != 0) return code;
    code = launch_gla_prefix(p, stream);
    if (code != 0) return code;
  }
  if (dtype == 0) WALK_D(float, grid_z, true);
  else WALK_D(__nv_bfloat16, grid_z, true);
#undef WALK_D
#undef WALK
  return code;
}
