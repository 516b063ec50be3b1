// Gated linear attention (gated_linear_attention.cu) for prompt portions in bfloat16 runs: the recurrence 16
// tokens at a time on tensor cores (mma.sync m16n8k16), with fp32 operands as two bfloat16 terms each.
//
// With P_t the product of a channel's decays from the 16 tokens' start through token t, S the state before them:
//
//   o_t  = S^T (q_t P_t) + sum_{s <= t} A_ts v_s          A_ts = sum_d q_td k_sd P_td / P_sd
//   S'   = diag(P_15) S + sum_s (k_s P_15 / P_s) v_s^T
//
// A block owns (a slice of 128 value columns, head, a chunk of tokens or a whole sequence).  Warp w keeps rows
// 16 w .. 16 w + 15 of S^T (value columns) x all key channels as fp32 accumulator fragments, which are at the same time the A operand of
// the read-out.  Per 16 tokens: q, k, the decays and v arrive in shared memory (cp.async, the next 16 in
// flight); threads form q P, k / P, k P_15 / P (running products; the last from the end, so that it never
// exceeds k) and split everything into two bfloat16 terms (x = hi + lo, relative error 2^-17); a product of two
// such operands is hi hi + hi lo + lo hi.  A is summed over the channels by the warps (16 channels each) and
// masked.  k / P grows where decays are strong: if a channel's P_15 falls below 1e-12 (k / P would leave the
// range in which the products are exact to rounding), A of these 16 tokens is formed by plain fp32 sums with
// the decays multiplied up between s and t instead.
//
// Long portions run chunk-parallel as in the walk: contributions per chunk (the same kernel without
// outputs, from a zero state), the pass over the chunks, outputs per chunk.  The decays themselves are formed
// once, by a kernel before these, for all tokens and channels.
//
// Where one block holds all of a head's value columns (vdim <= 128) it also finishes the head: RMS norm over
// vdim, weight, times act(gate), stored as bfloat16.
#include "common.cuh"
#include "gla_parts.cuh"
#include "mma_tile.cuh"

namespace leone {

constexpr int kGmTokens = 16, kGmThreads = 256, kGmCols = 128;
constexpr int kGmOPitch = kGmCols + 4;            // floats per token row of the read-out
constexpr int kGmAPitch = kGmTokens + 8;          // bfloat16 per row of A

__device__ __forceinline__ float log2_fast(float x) {
  float y;
  asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rcp_fast(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// alpha[t, c] = sigmoid(z)^(1/tau) = 2^(-log2(1 + 2^(-z log2 e)) / tau) for 16 tokens a block.  The hardware's powers
// and logarithms of two are a few units in the last place of fp32 off; near alpha = 1 the logarithm's argument is
// 1 + small, whose rounding is 6e-8 absolute.
__global__ void __launch_bounds__(256)
gla_decay_kernel(const GlaParams p, float* __restrict__ alpha, int n_tokens) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ __align__(16) float u_s[];     // [rank][16]
  const int tb = blockIdx.y * kGmTokens, nt = min(kGmTokens, n_tokens - tb), hd = p.heads * p.dim;
  for (int i = threadIdx.x; i < kGmTokens * p.rank; i += blockDim.x) {
    const int tt = i / p.rank, r = i - tt * p.rank;
    u_s[r * kGmTokens + tt] = tt < nt ? p.proj[(size_t)(tb + tt) * p.ld + p.u_off + r] : 0.f;
  }
  __syncthreads();
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= hd) return;
  float z[kGmTokens];
  const float b = p.w2_bias[c];
#pragma unroll
  for (int j = 0; j < kGmTokens; ++j) z[j] = b;
#pragma unroll 8
  for (int r = 0; r < p.rank; ++r) {
    const float w = p.w2[(size_t)r * hd + c];
#pragma unroll
    for (int j = 0; j < kGmTokens; j += 4) {
      const float4 u = *reinterpret_cast<const float4*>(u_s + r * kGmTokens + j);
      z[j] = fmaf(w, u.x, z[j]);
      z[j + 1] = fmaf(w, u.y, z[j + 1]);
      z[j + 2] = fmaf(w, u.z, z[j + 2]);
      z[j + 3] = fmaf(w, u.w, z[j + 3]);
    }
  }
  float* dst = alpha + (size_t)tb * hd + c;
#pragma unroll
  for (int j = 0; j < kGmTokens; ++j) {
    const float y = -1.4426950408889634f * z[j];
    const float sp = y > 30.f ? y : log2_fast(1.f + exp2_fast(y));      // softplus(-z) in units of log 2
    if (j < nt) dst[(size_t)j * hd] = exp2_fast(-sp * p.inv_tau);
  }
}

template <int KD> struct GmLayout {
  static constexpr int DIMP = KD * 16;
  static constexpr int PD = DIMP + 8, PV = kGmCols + 8;                 // bfloat16 per row
  static constexpr int kStage = kGmTokens * (3 * DIMP + kGmCols);       // floats: q, k, alpha, v
  static constexpr int kOFloats = kGmTokens * kGmOPitch > KD * 256 ? kGmTokens * kGmOPitch : KD * 256;
  static constexpr size_t bytes = sizeof(float) * (2 * kStage + kOFloats + DIMP) +
                                  2 * (size_t)kGmTokens * (6 * PD + 2 * PV + 2 * kGmAPitch);
};

template <int KD, bool OUT>
__global__ void __launch_bounds__(kGmThreads, 2)
gla_mma_kernel(const GlaParams p, const float* __restrict__ alpha) {
  pdl_trigger();
  pdl_wait();
  using L = GmLayout<KD>;
  constexpr int DIMP = L::DIMP, PD = L::PD, PV = L::PV, NT = 2 * KD;
  extern __shared__ __align__(16) float smem[];
  float* part = smem + 2 * L::kStage;              // [KD][16][16] partial A, later [16][pitch] read-out
  float* ptot = part + L::kOFloats;                // [DIMP]
  __nv_bfloat16* qh = reinterpret_cast<__nv_bfloat16*>(ptot + DIMP);   // q P: hi, lo; k / P: hi, lo; k P_15 / P: hi, lo
  __nv_bfloat16* ih = qh + 2 * kGmTokens * PD;
  __nv_bfloat16* th = ih + 2 * kGmTokens * PD;
  __nv_bfloat16* vh = th + 2 * kGmTokens * PD;     // v: hi, lo
  __nv_bfloat16* ah = vh + 2 * kGmTokens * PV;     // A: hi, lo
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3, mi = lane >> 3;
  const int dim = p.dim, vdim = p.vdim, heads = p.heads, h = blockIdx.y, v0 = blockIdx.x * kGmCols;
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
  float* s_out = !OUT ? mine : (sp.last ? slot_state : nullptr);
  const int cols = min(kGmCols, vdim - v0);        // this block's value columns
  const bool owner = warp * 16 < cols;             // (warp-uniform) this warp holds rows of the state
  const int hd = heads * dim;

  auto request = [&](int tb, int stage) {
    const int nt = min(kGmTokens, sp.t1 - tb);
    float* dst = smem + stage * L::kStage;
    const uint32_t base = (uint32_t)__cvta_generic_to_shared(dst);
    constexpr int Q4 = DIMP / 4;
    for (int i = tid; i < kGmTokens * Q4; i += kGmThreads) {
      const int tt = i / Q4, d = (i - tt * Q4) * 4;
      const bool ok = tt < nt && d < dim;
      const float* row = p.proj + (size_t)(tb + (ok ? tt : 0)) * p.ld + (size_t)h * dim + (ok ? d : 0);
      const uint32_t at = base + (tt * DIMP + d) * 4;
      if (OUT) cp_async16_zfill(at, row + p.q_off, ok);
      cp_async16_zfill(at + kGmTokens * DIMP * 4, row + p.k_off, ok);
      cp_async16_zfill(at + 2 * kGmTokens * DIMP * 4, alpha + (size_t)(tb + (ok ? tt : 0)) * hd + (size_t)h * dim + (ok ? d : 0), ok);
    }
    for (int i = tid; i < kGmTokens * (kGmCols / 4); i += kGmThreads) {
      const int tt = i / (kGmCols / 4), c = (i - tt * (kGmCols / 4)) * 4;
      const bool ok = tt < nt && c < cols;
      cp_async16_zfill(base + (3 * kGmTokens * DIMP + tt * kGmCols + c) * 4,
                       p.proj + (size_t)(tb + (ok ? tt : 0)) * p.ld + p.v_off + (size_t)h * vdim + v0 + (ok ? c : 0), ok);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  request(sp.t0, 0);

  // S^T fragments: value row warp * 16 + g (+ 8), channels n * 8 + 2 tq (+ 1)
  float S[NT][4];
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int v = warp * 16 + g + (i >> 1) * 8, d = n * 8 + 2 * tq + (i & 1);
      S[n][i] = OUT && v < cols && d < dim ? mine[(size_t)d * vdim + v0 + v] : 0.f;
    }
  float decay0 = 1.f, decay1 = 1.f;                // !OUT: this thread's two channels' products over the chunk
  const uint32_t q_addr = (uint32_t)__cvta_generic_to_shared(qh), i_addr = (uint32_t)__cvta_generic_to_shared(ih);
  const uint32_t t_addr = (uint32_t)__cvta_generic_to_shared(th), v_addr = (uint32_t)__cvta_generic_to_shared(vh);
  const uint32_t a_addr = (uint32_t)__cvta_generic_to_shared(ah);
  constexpr uint32_t kLoD = kGmTokens * PD * 2, kLoV = kGmTokens * PV * 2, kLoA = kGmTokens * kGmAPitch * 2;

  int stage = 0;
  for (int tb = sp.t0; tb < sp.t1; tb += kGmTokens, stage ^= 1) {
    const int nt = min(kGmTokens, sp.t1 - tb);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                               // the 16 tokens are there; the last ones' operands are read
    if (tb + kGmTokens < sp.t1) request(tb + kGmTokens, stage ^ 1);
    const float* q_s = smem + stage * L::kStage;
    const float* k_s = q_s + kGmTokens * DIMP;
    const float* a_s = k_s + kGmTokens * DIMP;
    const float* v_s = a_s + kGmTokens * DIMP;
    // operands: two channels (or value columns) a thread, four jobs of 64 threads
    int weak = 0;
    {
      const int job = tid >> 6, c = (tid & 63) * 2;
      if (job == 3) {
#pragma unroll 2
        for (int tt = 0; tt < kGmTokens; ++tt) {
          const float2 x = *reinterpret_cast<const float2*>(v_s + tt * kGmCols + c);
          uint32_t hi, lo;
          split_pair(x.x, x.y, hi, lo);
          *reinterpret_cast<uint32_t*>(vh + tt * PV + c) = hi;
          *reinterpret_cast<uint32_t*>(vh + (kGmTokens + tt) * PV + c) = lo;
        }
      } else if (c < DIMP && (OUT || job == 2)) {
        const bool in0 = c < dim, in1 = c + 1 < dim;
        float p0 = 1.f, p1 = 1.f;
        if (job == 2) {                            // from the last token back
#pragma unroll 2
          for (int tt = kGmTokens - 1; tt >= 0; --tt) {
            const float2 k = *reinterpret_cast<const float2*>(k_s + tt * DIMP + c);
            uint32_t hi, lo;
            split_pair(k.x * p0, k.y * p1, hi, lo);
            *reinterpret_cast<uint32_t*>(th + tt * PD + c) = hi;
            *reinterpret_cast<uint32_t*>(th + (kGmTokens + tt) * PD + c) = lo;
            if (tt < nt) {
              const float2 a = *reinterpret_cast<const float2*>(a_s + tt * DIMP + c);
              if (in0) p0 *= a.x;
              if (in1) p1 *= a.y;
            }
          }
          ptot[c] = p0;
          ptot[c + 1] = p1;
          weak = fminf(p0, p1) < 1e-12f;
          decay0 *= p0;
          decay1 *= p1;
        } else {
          const float* src = job == 0 ? q_s : k_s;
          __nv_bfloat16* dst = job == 0 ? qh : ih;
#pragma unroll 2
          for (int tt = 0; tt < kGmTokens; ++tt) {
            if (tt < nt) {
              const float2 a = *reinterpret_cast<const float2*>(a_s + tt * DIMP + c);
              if (in0) p0 *= a.x;
              if (in1) p1 *= a.y;
            }
            const float2 x = *reinterpret_cast<const float2*>(src + tt * DIMP + c);
            const float f0 = job == 0 ? p0 * p.q_scale : rcp_fast(p0), f1 = job == 0 ? p1 * p.q_scale : rcp_fast(p1);
            uint32_t hi, lo;
            split_pair(x.x * f0, x.y * f1, hi, lo);
            *reinterpret_cast<uint32_t*>(dst + tt * PD + c) = hi;
            *reinterpret_cast<uint32_t*>(dst + (kGmTokens + tt) * PD + c) = lo;
          }
        }
      }
    }
    weak = __syncthreads_or(weak);
    float O[2][4];
    if (OUT) {
      // A over this warp's 16 channels
      if (warp < KD) {
        uint32_t xh[4], xl[4], yh[4], yl[4];
        const uint32_t arow = ((lane & 15) * PD + (lane >> 4) * 8 + warp * 16) * 2;
        const uint32_t brow = (((lane & 7) + (mi >> 1) * 8) * PD + (mi & 1) * 8 + warp * 16) * 2;
        ldsm4(q_addr + arow, xh[0], xh[1], xh[2], xh[3]);
        ldsm4(q_addr + kLoD + arow, xl[0], xl[1], xl[2], xl[3]);
        ldsm4(i_addr + brow, yh[0], yh[1], yh[2], yh[3]);
        ldsm4(i_addr + kLoD + brow, yl[0], yl[1], yl[2], yl[3]);
#pragma unroll
        for (int nn = 0; nn < 2; ++nn) {
          float acc[4] = {0.f, 0.f, 0.f, 0.f};
          mma16816(acc, xl[0], xl[1], xl[2], xl[3], yh[2 * nn], yh[2 * nn + 1]);
          mma16816(acc, xh[0], xh[1], xh[2], xh[3], yl[2 * nn], yl[2 * nn + 1]);
          mma16816(acc, xh[0], xh[1], xh[2], xh[3], yh[2 * nn], yh[2 * nn + 1]);
          float* dst = part + warp * 256 + g * 16 + nn * 8 + 2 * tq;
          *reinterpret_cast<float2*>(dst) = make_float2(acc[0], acc[1]);
          *reinterpret_cast<float2*>(dst + 8 * 16) = make_float2(acc[2], acc[3]);
        }
      }
      // the read-out of the state before these tokens
#pragma unroll
      for (int nn = 0; nn < 2; ++nn)
#pragma unroll
        for (int i = 0; i < 4; ++i) O[nn][i] = 0.f;
      if (owner) {
#pragma unroll
        for (int j = 0; j < KD; ++j) {
          uint32_t sh[4], sl[4], bh[4], bl[4];
          split_pair(S[2 * j][0], S[2 * j][1], sh[0], sl[0]);
          split_pair(S[2 * j][2], S[2 * j][3], sh[1], sl[1]);
          split_pair(S[2 * j + 1][0], S[2 * j + 1][1], sh[2], sl[2]);
          split_pair(S[2 * j + 1][2], S[2 * j + 1][3], sh[3], sl[3]);
          const uint32_t brow = (((lane & 7) + (mi >> 1) * 8) * PD + (mi & 1) * 8 + j * 16) * 2;
          ldsm4(q_addr + brow, bh[0], bh[1], bh[2], bh[3]);
          ldsm4(q_addr + kLoD + brow, bl[0], bl[1], bl[2], bl[3]);
#pragma unroll
          for (int nn = 0; nn < 2; ++nn) {
            mma16816(O[nn], sl[0], sl[1], sl[2], sl[3], bh[2 * nn], bh[2 * nn + 1]);
            mma16816(O[nn], sh[0], sh[1], sh[2], sh[3], bl[2 * nn], bl[2 * nn + 1]);
            mma16816(O[nn], sh[0], sh[1], sh[2], sh[3], bh[2 * nn], bh[2 * nn + 1]);
          }
        }
      }
      __syncthreads();
      {
        // one (token, earlier token) pair a thread
        const int t = tid >> 4, s = tid & 15;
        float a = 0.f;
        if (s <= t) {
          if (!weak) {
#pragma unroll
            for (int w = 0; w < KD; ++w) a += part[w * 256 + tid];
          } else if (t < nt) {
            for (int d = 0; d < dim; ++d) {
              float w = k_s[s * DIMP + d];
              for (int u = s + 1; u <= t; ++u) w *= a_s[u * DIMP + d];
              a = fmaf(q_s[t * DIMP + d] * p.q_scale, w, a);
            }
          }
        }
        const __nv_bfloat16 hi = __float2bfloat16_rn(a);
        ah[t * kGmAPitch + s] = hi;
        ah[(kGmTokens + t) * kGmAPitch + s] = __float2bfloat16_rn(a - __bfloat162float(hi));
      }
      __syncthreads();
    }
    float4 gate[2];
    if (owner) {
      uint32_t xh[4], xl[4];
      const uint32_t vrow = (((lane & 7) + (mi >> 1) * 8) * PV + (mi & 1) * 8 + warp * 16) * 2;
      ldsm4_trans(v_addr + vrow, xh[0], xh[1], xh[2], xh[3]);
      ldsm4_trans(v_addr + kLoV + vrow, xl[0], xl[1], xl[2], xl[3]);
      if (OUT) {
        uint32_t bh[4], bl[4];
        const uint32_t brow = (((lane & 7) + (mi >> 1) * 8) * kGmAPitch + (mi & 1) * 8) * 2;
        ldsm4(a_addr + brow, bh[0], bh[1], bh[2], bh[3]);
        ldsm4(a_addr + kLoA + brow, bl[0], bl[1], bl[2], bl[3]);
#pragma unroll
        for (int nn = 0; nn < 2; ++nn) {
          mma16816(O[nn], xl[0], xl[1], xl[2], xl[3], bh[2 * nn], bh[2 * nn + 1]);
          mma16816(O[nn], xh[0], xh[1], xh[2], xh[3], bl[2 * nn], bl[2 * nn + 1]);
          mma16816(O[nn], xh[0], xh[1], xh[2], xh[3], bh[2 * nn], bh[2 * nn + 1]);
#pragma unroll
          for (int i = 0; i < 4; ++i)
            part[(nn * 8 + 2 * tq + (i & 1)) * kGmOPitch + warp * 16 + g + (i >> 1) * 8] = O[nn][i];
        }
      }
      // S^T <- S^T diag(P_15) + V^T (k P_15 / P)
#pragma unroll
      for (int j = 0; j < KD; ++j) {
        uint32_t bh[4], bl[4];
        const uint32_t brow = (((lane & 7) + (mi & 1) * 8) * PD + j * 16 + (mi >> 1) * 8) * 2;
        ldsm4_trans(t_addr + brow, bh[0], bh[1], bh[2], bh[3]);
        ldsm4_trans(t_addr + kLoD + brow, bl[0], bl[1], bl[2], bl[3]);
#pragma unroll
        for (int nn = 0; nn < 2; ++nn) {
          float* c = S[2 * j + nn];
          const float2 f = *reinterpret_cast<const float2*>(ptot + (2 * j + nn) * 8 + 2 * tq);
          c[0] *= f.x;
          c[1] *= f.y;
          c[2] *= f.x;
          c[3] *= f.y;
          mma16816(c, xl[0], xl[1], xl[2], xl[3], bh[2 * nn], bh[2 * nn + 1]);
          mma16816(c, xh[0], xh[1], xh[2], xh[3], bl[2 * nn], bl[2 * nn + 1]);
          mma16816(c, xh[0], xh[1], xh[2], xh[3], bh[2 * nn], bh[2 * nn + 1]);
        }
      }
    }
    if (OUT) {
      // two tokens a warp, four value columns a lane
      const int c = lane * 4;
      if (p.gated != nullptr && c < cols) {
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int tt = warp + i * 8;
          if (tt < nt)
            gate[i] = *reinterpret_cast<const float4*>(p.proj + (size_t)(tb + tt) * p.ld + p.gate_off + (size_t)h * vdim + c);
        }
      }
      __syncthreads();
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int tt = warp + i * 8;
        if (tt >= nt) continue;                    // (warp-uniform)
        const size_t t = tb + tt;
        const bool in = c < cols;
        const float4 o = in ? *reinterpret_cast<const float4*>(part + tt * kGmOPitch + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        if (p.out != nullptr && in) *reinterpret_cast<float4*>(p.out + t * p.ldo + (size_t)h * vdim + v0 + c) = o;
        if (p.gated != nullptr) {
          const float ss = warp_sum(fmaf(o.x, o.x, fmaf(o.y, o.y, fmaf(o.z, o.z, o.w * o.w))));
          if (in) {
            const float r = 1.f / sqrtf(ss / (float)vdim + p.eps);
            const float4 w = *reinterpret_cast<const float4*>(p.norm_w + c);
            auto f = [&](float z) {
              const float sg = __fdividef(1.f, 1.f + __expf(-z));
              return p.gate_act == 1 ? z * sg : sg;
            };
            uint2 y;
            y.x = pack_bf16(o.x * r * w.x * f(gate[i].x), o.y * r * w.y * f(gate[i].y));
            y.y = pack_bf16(o.z * r * w.z * f(gate[i].z), o.w * r * w.w * f(gate[i].w));
            *reinterpret_cast<uint2*>(reinterpret_cast<__nv_bfloat16*>(p.gated) + t * p.ldg + (size_t)h * vdim + c) = y;
          }
        }
      }
    }
  }
  if (s_out != nullptr && owner) {
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int v = warp * 16 + g + (i >> 1) * 8, d = n * 8 + 2 * tq + (i & 1);
        if (v < cols && d < dim) s_out[(size_t)d * vdim + v0 + v] = S[n][i];
      }
  }
  if (!OUT && blockIdx.x == 0 && (tid >> 6) == 2) {
    const int c = (tid & 63) * 2;
    float* dst = p.chunk_decay + ((size_t)blockIdx.z * heads + h) * dim;
    if (c < dim) dst[c] = decay0;
    if (c + 1 < dim) dst[c + 1] = decay1;
  }
}

}  // namespace leone

using namespace leone;

// 1 if the tensor-core form takes these sizes (rows and columns that float4 loads fit).
extern "C" int leone_gla_mma_supported(int dim, int vdim) { return dim > 0 && dim <= 128 && dim % 4 == 0 && vdim > 0 && vdim % 4 == 0; }

// The arguments of leone_gla, bfloat16 results; alpha: fp32 scratch [n_tokens, heads * dim].  ld, the column
// offsets and ldo must be multiples of 4, ldg of 4.
extern "C" int leone_gla_mma(const float* proj, int ld, int q_off, int k_off, int v_off, int u_off, int gate_off,
                             const float* w2, const float* w2_bias, int rank, float inv_tau, float q_scale, float* out,
                             int ldo, void* gated, int ldg, const float* norm_w, int gate_act, float eps, float* state,
                             const int* q_start, const int* slot_ids, int n_tokens, int n_seqs, int heads, int dim,
                             int vdim, int n_slots, int chunk, int n_chunks, float* chunk_state, float* chunk_decay,
                             float* alpha, int* status, cudaStream_t stream) {
  if (n_seqs <= 0 || n_tokens <= 0) return 0;
  if (!leone_gla_mma_supported(dim, vdim) || heads <= 0 || heads > 65535 || n_seqs > 65535 || rank <= 0 || rank > 512 ||
      (n_tokens + kGmTokens - 1) / kGmTokens > 65535)
    return kRefusedSize;
  if (chunk < 0 || (chunk > 0 && (chunk % kGmTokens != 0 || n_chunks <= 0 || n_chunks > 65535 || chunk_state == nullptr ||
                                  chunk_decay == nullptr)))
    return kRefusedSize;
  if (ld % 4 || q_off % 4 || k_off % 4 || v_off % 4 || gate_off % 4 || ldo % 4 || ldg % 4 ||
      (((uintptr_t)proj | (uintptr_t)alpha | (uintptr_t)out | (uintptr_t)norm_w | (uintptr_t)state) & 15) ||
      ((uintptr_t)gated & 7))
    return kRefusedAlignment;
  const int slices = (vdim + kGmCols - 1) / kGmCols;
  if ((out == nullptr && gated == nullptr) || (gated != nullptr && (slices != 1 || norm_w == nullptr))) return kRefusedSize;
  GlaParams p = {proj, ld, q_off, k_off, v_off, u_off, w2, w2_bias, rank, inv_tau, q_scale, state, q_start, slot_ids,
                 heads, dim, vdim, chunk, n_seqs, n_slots, chunk_state, chunk_decay, out, ldo, gated, ldg, norm_w,
                 gate_off, gate_act, eps, status};
  const int hd = heads * dim;
  int code = launch_kernel(gla_decay_kernel, dim3((hd + 255) / 256, (n_tokens + kGmTokens - 1) / kGmTokens), dim3(256),
                           sizeof(float) * kGmTokens * rank, stream, p, alpha, n_tokens);
  if (code != 0) return code;
  const int grid_z = chunk > 0 ? n_chunks : n_seqs;
#define RUN(KD, OUT)                                                                                                 \
  do {                                                                                                               \
    constexpr size_t smem = GmLayout<KD>::bytes;                                                                     \
    static bool configured = false;                                                                                  \
    if (!configured) {                                                                                               \
      cudaFuncSetAttribute(gla_mma_kernel<KD, OUT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);         \
      configured = true;                                                                                             \
    }                                                                                                                \
    code = launch_kernel(gla_mma_kernel<KD, OUT>, dim3(slices, heads, grid_z), dim3(kGmThreads), smem, stream, p, alpha); \
  } while (0)
#define RUN_D(OUT)                  \
  do {                              \
    if (dim <= 32) RUN(2, OUT);     \
    else if (dim <= 48) RUN(3, OUT); \
    else if (dim <= 64) RUN(4, OUT); \
    else if (dim <= 96) RUN(6, OUT); \
    else RUN(8, OUT);               \
  } while (0)
  if (chunk > 0) {
    RUN_D(false);
    if (code != 0) return code;
    code = launch_gla_prefix(p, stream);
    if (code != 0) return code;
  }
  RUN_D(true);
#undef RUN_D
#undef RUN
  return code;
}
