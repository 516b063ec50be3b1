// The Mamba-2 recurrence (ssd.cu) for prompt portions in bfloat16 runs: 64 tokens at a time as matrix products on
// tensor cores (mma.sync m16n8k16).  x, B and C are bfloat16 and enter exactly; what is fp32 (the state, the weights with
// decays and steps in them) enters as two bfloat16 terms each (hi + lo, relative error 2^-17).
//
// With a_t the sum of the decays' logarithms from the 64 tokens' start through token t, d_t the steps, S the state
// before them:
//
//   y_t = exp(a_t) S^T C_t + sum_{s <= t} A_ts x_s        A_ts = (C_t . B_s) exp(a_t - a_s) d_s  (+ D where s = t)
//   S'  = exp(a_63) S + sum_s B_s (exp(a_63 - a_s) d_s x_s)^T
//
// All exponents are sums of logarithms of decays between two tokens, never positive, so nothing grows where decays are
// strong.
//
// A block owns (a slice of 64 value columns, head, a chunk of tokens or a whole sequence).  Warp w keeps rows
// 16 w .. 16 w + 15 of S^T (value columns) x all state rows as fp32 accumulator fragments, which are at the same time the A
// operand of the read-out; of A it forms tokens 16 w .. 16 w + 15.  Long portions run chunk-parallel: contributions per chunk
// (the same kernel without outputs, from a zero state), the pass over the chunks that gated linear attention has, outputs
// per chunk.
#include "gla_parts.cuh"
#include "mma_tile.cuh"
#include "ssd_parts.cuh"

namespace leone {

constexpr int kSmTokens = 64, kSmThreads = 128, kSmCols = 64;
constexpr int kSmPX = kSmCols + 8, kSmPA = kSmTokens + 8;               // bfloat16 per row of x and of A

template <int KD, bool OUT, int STAGES> struct SmLayout {
  static constexpr int NP = KD * 16, PD = NP + 8;                       // state rows with padding; bfloat16 per row of B and C
  static constexpr int kTile = kSmTokens * ((OUT ? 2 : 1) * PD + kSmPX);
  static constexpr size_t bytes = 2 * (size_t)(STAGES * kTile + (OUT ? 2 * kSmTokens * kSmPA : 0)) + sizeof(float) * (4 * kSmTokens + 1);
};

template <int KD, bool OUT, int STAGES>
__global__ void __launch_bounds__(kSmThreads, 2)
ssd_mma_kernel(const SsdParams p) {
  pdl_trigger();
  pdl_wait();
  using L = SmLayout<KD, OUT, STAGES>;
  constexpr int NP = L::NP, PD = L::PD, NT = 2 * KD;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  __nv_bfloat16* tiles = reinterpret_cast<__nv_bfloat16*>(smem_raw);    // per stage: B, x, C
  __nv_bfloat16* ah = tiles + STAGES * L::kTile;                        // A: hi, lo
  float* a_s = reinterpret_cast<float*>(ah + (OUT ? 2 * kSmTokens * kSmPA : 0));   // sums of logarithms (base 2)
  float* d_s = a_s + kSmTokens;                                         // steps
  float* w_s = d_s + kSmTokens;                                         // what a token's write keeps until the tile's end
  float* e_s = w_s + kSmTokens;                                         // what the state before keeps until the token
  float* keep_s = e_s + kSmTokens;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3, mi = lane >> 3;
  const int n_state = p.n_state, vdim = p.vdim, h = blockIdx.y, v0 = blockIdx.x * kSmCols;
  GlaSpan sp;
  if (!gla_span(p, blockIdx.z, sp)) return;
  if (!OUT && sp.last) return;                     // the last chunk's contribution is never needed
  const int slot = p.slot_ids[sp.seq];
  if (slot < 0 || slot >= p.n_slots) {
    if (tid == 0) set_status(p.status, kBadSequence, sp.seq, slot);
    return;
  }
  const size_t per_head = (size_t)n_state * vdim;
  float* slot_state = p.state + ((size_t)slot * p.heads + h) * per_head;
  float* mine = p.chunk > 0 ? p.chunk_state + ((size_t)blockIdx.z * p.heads + h) * per_head : slot_state;
  float* s_out = !OUT ? mine : (sp.last ? slot_state : nullptr);
  const int cols = min(kSmCols, vdim - v0);        // this block's value columns
  const bool owner = warp * 16 < cols;             // (warp-uniform) this warp holds rows of the state
  const int grp = h / (p.heads / p.groups);
  const __nv_bfloat16* act = reinterpret_cast<const __nv_bfloat16*>(p.act);
  const __nv_bfloat16* b_src = act + p.b_off + (size_t)grp * n_state;
  const __nv_bfloat16* c_src = act + p.c_off + (size_t)grp * n_state;
  const __nv_bfloat16* x_src = act + p.x_off + (size_t)h * vdim + v0;
  const __nv_bfloat16* dt_src = reinterpret_cast<const __nv_bfloat16*>(p.raw) + p.dt_off + h;

  auto request = [&](int tb, int stage) {
    const int nt = min(kSmTokens, sp.t1 - tb);
    const uint32_t b_at = (uint32_t)__cvta_generic_to_shared(tiles + stage * L::kTile);
    const uint32_t x_at = b_at + 2 * kSmTokens * PD, c_at = x_at + 2 * kSmTokens * kSmPX;
    for (int i = tid; i < kSmTokens * 2 * KD; i += kSmThreads) {
      const int tt = i / (2 * KD), d = (i - tt * 2 * KD) * 8;
      const bool ok = tt < nt && d < n_state;
      const size_t at = (size_t)(tb + (ok ? tt : 0)) * p.lda + (ok ? d : 0);
      cp_async16_zfill(b_at + (tt * PD + d) * 2, b_src + at, ok);
      if (OUT) cp_async16_zfill(c_at + (tt * PD + d) * 2, c_src + at, ok);
    }
#pragma unroll
    for (int i = tid; i < kSmTokens * (kSmCols / 8); i += kSmThreads) {
      const int tt = i >> 3, c = (i & 7) * 8;
      const bool ok = tt < nt && c < cols;
      cp_async16_zfill(x_at + (tt * kSmPX + c) * 2, x_src + (size_t)(tb + (ok ? tt : 0)) * p.lda + (ok ? c : 0), ok);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  // a lane of warp 0 has the steps of tokens 2 lane and 2 lane + 1 of the next 64
  float raw0 = 0.f, raw1 = 0.f;
  auto steps = [&](int tb) {
    const int t = tb + 2 * lane;
    if (warp == 0 && t < sp.t1) raw0 = __bfloat162float(dt_src[(size_t)t * p.ldr]);
    if (warp == 0 && t + 1 < sp.t1) raw1 = __bfloat162float(dt_src[(size_t)(t + 1) * p.ldr]);
  };
  request(sp.t0, 0);
  steps(sp.t0);

  // S^T fragments: value row warp * 16 + g (+ 8), state rows n * 8 + 2 tq (+ 1)
  float S[NT][4];
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int v = warp * 16 + g + (i >> 1) * 8, d = n * 8 + 2 * tq + (i & 1);
      S[n][i] = OUT && v < cols && d < n_state ? mine[(size_t)d * vdim + v0 + v] : 0.f;
    }
  const float rate2 = expf(p.a_log[h]) * 1.4426950408889634f, bias = p.dt_bias[h], skip = p.d_skip[h];
  float log_kept = 0.f;                            // warp 0: the chunk's sum of logarithms
  const uint32_t a_addr = (uint32_t)__cvta_generic_to_shared(ah);
  constexpr uint32_t kLoA = kSmTokens * kSmPA * 2;

  int stage = 0;
  for (int tb = sp.t0; tb < sp.t1; tb += kSmTokens) {
    const int nt = min(kSmTokens, sp.t1 - tb);
    const bool more = tb + kSmTokens < sp.t1;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                               // the tokens are there; the last ones' operands are read
    if (STAGES == 2 && more) request(tb + kSmTokens, stage ^ 1);
    const uint32_t b_at = (uint32_t)__cvta_generic_to_shared(tiles + stage * L::kTile);
    const uint32_t x_at = b_at + 2 * kSmTokens * PD, c_at = x_at + 2 * kSmTokens * kSmPX;
    if (warp == 0) {
      const float d0 = 2 * lane < nt ? ssd_step(raw0, bias) : 0.f, d1 = 2 * lane + 1 < nt ? ssd_step(raw1, bias) : 0.f;
      const float l0 = -rate2 * d0, l1 = -rate2 * d1;
      float sum = l0 + l1;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float before = __shfl_up_sync(0xffffffffu, sum, o);
        if (lane >= o) sum += before;
      }
      float a0 = __shfl_up_sync(0xffffffffu, sum, 1);
      a0 = (lane == 0 ? 0.f : a0) + l0;
      const float total = __shfl_sync(0xffffffffu, sum, 31);
      *reinterpret_cast<float2*>(a_s + 2 * lane) = make_float2(a0, sum);
      *reinterpret_cast<float2*>(d_s + 2 * lane) = make_float2(d0, d1);
      *reinterpret_cast<float2*>(w_s + 2 * lane) = make_float2(d0 * exp2_fast(total - a0), d1 * exp2_fast(total - sum));
      *reinterpret_cast<float2*>(e_s + 2 * lane) = make_float2(exp2_fast(a0), exp2_fast(sum));
      if (lane == 0) *keep_s = exp2_fast(total);
      log_kept += total;
      steps(tb + kSmTokens);
    }
    float Y[8][4];
    if (OUT) {
      // C B^T for this warp's 16 tokens and the tokens up to them
      float G[8][4];
#pragma unroll
      for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) G[n][i] = 0.f;
#pragma unroll
      for (int k = 0; k < KD; ++k) {
        uint32_t c[4];
        ldsm4(c_at + ((warp * 16 + (lane & 15)) * PD + (lane >> 4) * 8 + k * 16) * 2, c[0], c[1], c[2], c[3]);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          if (j <= warp) {
            uint32_t b[4];
            ldsm4(b_at + ((j * 16 + (lane & 7) + (mi >> 1) * 8) * PD + (mi & 1) * 8 + k * 16) * 2, b[0], b[1], b[2], b[3]);
            mma16816(G[2 * j], c[0], c[1], c[2], c[3], b[0], b[1]);
            mma16816(G[2 * j + 1], c[0], c[1], c[2], c[3], b[2], b[3]);
          }
        }
      }
      __syncthreads();                             // sums and steps are there
      const float at[2] = {a_s[warp * 16 + g], a_s[warp * 16 + g + 8]};
#pragma unroll
      for (int n = 0; n < 8; ++n) {
        if ((n >> 1) <= warp) {
          const int s = n * 8 + 2 * tq;
          const float2 as = *reinterpret_cast<const float2*>(a_s + s), ds = *reinterpret_cast<const float2*>(d_s + s);
#pragma unroll
          for (int r = 0; r < 2; ++r) {
            const int t = warp * 16 + g + r * 8;
            float u0 = s <= t ? G[n][2 * r] * (exp2_fast(at[r] - as.x) * ds.x) : 0.f;
            float u1 = s + 1 <= t ? G[n][2 * r + 1] * (exp2_fast(at[r] - as.y) * ds.y) : 0.f;
            if (s == t) u0 += skip;
            if (s + 1 == t) u1 += skip;
            uint32_t hi, lo;
            split_pair(u0, u1, hi, lo);
            *reinterpret_cast<uint32_t*>(ah + t * kSmPA + s) = hi;
            *reinterpret_cast<uint32_t*>(ah + (kSmTokens + t) * kSmPA + s) = lo;
          }
        }
      }
      // the read-out of the state before these tokens
#pragma unroll
      for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) Y[n][i] = 0.f;
      if (owner) {
#pragma unroll
        for (int k = 0; k < KD; ++k) {
          uint32_t sh[4], sl[4];
          split_pair(S[2 * k][0], S[2 * k][1], sh[0], sl[0]);
          split_pair(S[2 * k][2], S[2 * k][3], sh[1], sl[1]);
          split_pair(S[2 * k + 1][0], S[2 * k + 1][1], sh[2], sl[2]);
          split_pair(S[2 * k + 1][2], S[2 * k + 1][3], sh[3], sl[3]);
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            uint32_t c[4];
            ldsm4(c_at + ((j * 16 + (lane & 7) + (mi >> 1) * 8) * PD + (mi & 1) * 8 + k * 16) * 2, c[0], c[1], c[2], c[3]);
#pragma unroll
            for (int nn = 0; nn < 2; ++nn) {
              mma16816(Y[2 * j + nn], sl[0], sl[1], sl[2], sl[3], c[2 * nn], c[2 * nn + 1]);
              mma16816(Y[2 * j + nn], sh[0], sh[1], sh[2], sh[3], c[2 * nn], c[2 * nn + 1]);
            }
          }
        }
      }
    }
    __syncthreads();                               // A (without outputs: sums and steps) is there
    if (owner) {
      if (OUT) {
#pragma unroll
        for (int n = 0; n < 8; ++n) {
          const float2 e = *reinterpret_cast<const float2*>(e_s + n * 8 + 2 * tq);
          Y[n][0] *= e.x;
          Y[n][1] *= e.y;
          Y[n][2] *= e.x;
          Y[n][3] *= e.y;
        }
      }
      const float keep = *keep_s;
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) S[n][i] *= keep;
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        uint32_t x[4];
        ldsm4_trans(x_at + ((k * 16 + (lane & 7) + (mi >> 1) * 8) * kSmPX + (mi & 1) * 8 + warp * 16) * 2, x[0], x[1], x[2], x[3]);
        if (OUT) {
#pragma unroll
          for (int j = k; j < 4; ++j) {
            uint32_t bh[4], bl[4];
            const uint32_t at = a_addr + ((j * 16 + (lane & 7) + (mi >> 1) * 8) * kSmPA + (mi & 1) * 8 + k * 16) * 2;
            ldsm4(at, bh[0], bh[1], bh[2], bh[3]);
            ldsm4(at + kLoA, bl[0], bl[1], bl[2], bl[3]);
#pragma unroll
            for (int nn = 0; nn < 2; ++nn) {
              mma16816(Y[2 * j + nn], x[0], x[1], x[2], x[3], bl[2 * nn], bl[2 * nn + 1]);
              mma16816(Y[2 * j + nn], x[0], x[1], x[2], x[3], bh[2 * nn], bh[2 * nn + 1]);
            }
          }
        }
        // S^T += (w x)^T B
        uint32_t xh[4], xl[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float2 w = *reinterpret_cast<const float2*>(w_s + k * 16 + (i >> 1) * 8 + 2 * tq);
          split_pair(__uint_as_float(x[i] << 16) * w.x, __uint_as_float(x[i] & 0xffff0000u) * w.y, xh[i], xl[i]);
        }
#pragma unroll
        for (int j = 0; j < KD; ++j) {
          uint32_t b[4];
          ldsm4_trans(b_at + ((k * 16 + (lane & 7) + (mi & 1) * 8) * PD + j * 16 + (mi >> 1) * 8) * 2, b[0], b[1], b[2], b[3]);
#pragma unroll
          for (int nn = 0; nn < 2; ++nn) {
            mma16816(S[2 * j + nn], xl[0], xl[1], xl[2], xl[3], b[2 * nn], b[2 * nn + 1]);
            mma16816(S[2 * j + nn], xh[0], xh[1], xh[2], xh[3], b[2 * nn], b[2 * nn + 1]);
          }
        }
      }
      if (OUT) {
        float* dst = p.out + (size_t)h * vdim + v0 + warp * 16 + g;
        const bool in0 = warp * 16 + g < cols, in1 = warp * 16 + g + 8 < cols;
#pragma unroll
        for (int n = 0; n < 8; ++n)
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            const int t = n * 8 + 2 * tq + i;
            if (t < nt) {
              if (in0) dst[(size_t)(tb + t) * p.ldo] = Y[n][i];
              if (in1) dst[(size_t)(tb + t) * p.ldo + 8] = Y[n][2 + i];
            }
          }
      }
    }
    if (STAGES == 2) {
      stage ^= 1;
    } else if (more) {
      __syncthreads();                             // this tile's operands are read
      request(tb + kSmTokens, 0);
    }
  }
  if (s_out != nullptr && owner) {
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int v = warp * 16 + g + (i >> 1) * 8, d = n * 8 + 2 * tq + (i & 1);
        if (v < cols && d < n_state) s_out[(size_t)d * vdim + v0 + v] = S[n][i];
      }
  }
  if (!OUT && blockIdx.x == 0 && warp == 0) {
    const float kept = exp2_fast(log_kept);
    float* dst = p.chunk_decay + ((size_t)blockIdx.z * p.heads + h) * n_state;
    for (int d = lane; d < n_state; d += 32) dst[d] = kept;
  }
}

}  // namespace leone

using namespace leone;

// 1 if the tensor-core form takes these sizes (rows of 16-byte loads).
extern "C" int leone_ssd_mma_supported(int n_state, int vdim) {
  return n_state > 0 && n_state <= 256 && n_state % 8 == 0 && vdim > 0 && vdim % 8 == 0;
}

// The arguments of leone_ssd with bfloat16 act and raw.  chunk: a multiple of 64 with scratch chunk_state fp32 [n_chunks,
// heads, n_state, vdim] and chunk_decay fp32 [n_chunks, heads, n_state], or 0.  lda and the offsets must be multiples of 8.
extern "C" int leone_ssd_mma(const void* act, int lda, int x_off, int b_off, int c_off, const void* raw, int ldr, int dt_off,
                             const float* a_log, const float* dt_bias, const float* d_skip, float* out, int ldo,
                             float* state, const int* q_start, const int* slot_ids, int n_seqs, int heads, int groups,
                             int n_state, int vdim, int n_slots, int chunk, int n_chunks, float* chunk_state,
                             float* chunk_decay, int* status, cudaStream_t stream) {
  if (n_seqs <= 0) return 0;
  if (!leone_ssd_mma_supported(n_state, vdim) || heads <= 0 || groups <= 0 || heads % groups != 0 || heads > 65535 ||
      n_seqs > 65535)
    return kRefusedSize;
  if (chunk < 0 || (chunk > 0 && (chunk % kSmTokens != 0 || n_chunks <= 0 || n_chunks > 65535 || chunk_state == nullptr ||
                                  chunk_decay == nullptr)))
    return kRefusedSize;
  if (lda % 8 || x_off % 8 || b_off % 8 || c_off % 8 || ((uintptr_t)act & 15) ||
      (((uintptr_t)state | (uintptr_t)chunk_state) & 15))
    return kRefusedAlignment;
  SsdParams p = {act, lda, x_off, b_off, c_off, raw, ldr, dt_off, a_log, dt_bias, d_skip, out, ldo, state, q_start, slot_ids,
                 n_seqs, heads, groups, n_state, vdim, n_slots, status, chunk, chunk_state, chunk_decay};
  const int slices = (vdim + kSmCols - 1) / kSmCols, grid_z = chunk > 0 ? n_chunks : n_seqs;
  int code = 0;
#define RUN(KD, OUT, ST)                                                                                             \
  do {                                                                                                               \
    constexpr size_t smem = SmLayout<KD, OUT, ST>::bytes;                                                            \
    static bool configured = false;                                                                                  \
    if (!configured && smem > 48 * 1024)                                                                             \
      cudaFuncSetAttribute(ssd_mma_kernel<KD, OUT, ST>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);     \
    configured = true;                                                                                               \
    code = launch_kernel(ssd_mma_kernel<KD, OUT, ST>, dim3(slices, heads, grid_z), dim3(kSmThreads), smem, stream, p); \
  } while (0)
  // (two stages of tiles and two blocks an SM; three blocks with one stage each measured 105 us where this takes 89)
#define RUN_D(OUT)                           \
  do {                                       \
    if (n_state <= 32) RUN(2, OUT, 2);       \
    else if (n_state <= 48) RUN(3, OUT, 2);  \
    else if (n_state <= 64) RUN(4, OUT, 2);  \
    else if (n_state <= 96) RUN(6, OUT, 2);  \
    else if (n_state <= 128) RUN(8, OUT, 2); \
    else RUN(16, OUT, 1);                    \
  } while (0)
  if (chunk > 0) {
    RUN_D(false);
    if (code != 0) return code;
    GlaParams pass = {};
    pass.state = state;
    pass.q_start = q_start;
    pass.slot_ids = slot_ids;
    pass.heads = heads;
    pass.dim = n_state;
    pass.vdim = vdim;
    pass.chunk = chunk;
    pass.n_seqs = n_seqs;
    pass.n_slots = n_slots;
    pass.chunk_state = chunk_state;
    pass.chunk_decay = chunk_decay;
    code = launch_gla_prefix(pass, stream);
    if (code != 0) return code;
  }
  RUN_D(true);
#undef RUN_D
#undef RUN
  return code;
}
