// The gated delta rule (gated_delta.cu) for prompt portions in bfloat16 runs: 16 tokens at a time as matrix products on
// tensor cores (mma.sync m16n8k16), with fp32 operands as two bfloat16 terms each (hi + lo, relative error 2^-17).
//
// Let P_t be the product of a state row's decays from the 16 tokens' start through token t (the rows may decay alike or
// each at its own rate) and S the state before them.  Unrolling the recurrence over the 16 tokens gives
//
//   u_t = beta_t (v_t - S^T (k_t P_t) - sum_{s<t} M_ts u_s)      M_ts = sum_d k_td k_sd P_td / P_sd
//   o_t = S^T (q_t P_t) + sum_{s<=t} A_ts u_s                    A_ts = sum_d q_td k_sd P_td / P_sd
//   S'  = diag(P_15) S + sum_s (k_s P_15 / P_s) u_s^T
//
// so the corrections u solve a unit triangular system whose matrix does not depend on the state: U = T (V - (kP) S) with T =
// (I + diag(beta) M)^(-1) diag(beta).  Every ratio of P's is formed as a power of two of a difference of sums of logarithms,
// never positive, so nothing grows where decays are strong.
//
// delta_operands: a block per (16 tokens, head) makes unit vectors, decays, M, A and T and leaves k P, q P, k P_15 / P, T and A
// as pairs of bfloat16 terms in one image in the order of the next kernel's shared memory.
// delta_chain: a block per (16 or 32 value columns, head, sequence) walks the images.  Four warps to 16 value columns, a
// quarter of the state's rows each; S^T stays in fp32 accumulator fragments, which are at the same time the A
// operand of the read-outs; the four partial read-outs of a group meet in shared memory, after which every warp forms the
// corrections itself and moves its rows of the state.
#include "gla_parts.cuh"
#include "mma_tile.cuh"

namespace leone {

constexpr int kDmTokens = 16, kDmThreads = 256;
constexpr int kDmPT = kDmTokens + 8;              // bfloat16 per row of T and A

struct DeltaMmaParams {
  const float* act;                               // q, k (kv_heads x dim each) and v (heads x vdim) activations
  int lda, q_off, k_off, v_off;
  const void* raw;                                // one a (without zs) and one b per head
  int ldr, a_off, b_off;
  const float* zs;                                // decay logits per head and key channel, or null
  int ldz;
  const float* a_log;
  const float* dt_bias;                           // [heads], without zs
  float q_scale;
  float* out;
  int ldo;
  float* state;
  const int* q_start;
  const int* slot_ids;
  int heads, kv_heads, dim, vdim, n_seqs, n_slots, chunk;
  unsigned char* images;                          // [groups of 16 tokens, heads, image]
  int* status;
};

// KPW: 16-row steps of the state per warp (a quarter of them)
template <int KPW> struct DmImage {
  static constexpr int DIMP = 64 * KPW, PD = DIMP + 8;
  static constexpr int kTile = kDmTokens * PD * 2, kSmall = kDmTokens * kDmPT * 2;      // bytes
  // k P: hi, lo; q P: hi, lo; k P_15 / P: hi, lo; T: hi, lo; A: hi, lo; P_15 (fp32)
  static constexpr int kT = 6 * kTile, kA = kT + 2 * kSmall, kKeep = kA + 2 * kSmall;
  static constexpr int bytes = kKeep + DIMP * 4;
};

template <int KPW, bool CHANNEL, typename TR>
__global__ void __launch_bounds__(kDmThreads)
delta_operands_kernel(const DeltaMmaParams p) {
  pdl_trigger();
  pdl_wait();
  using I = DmImage<KPW>;
  constexpr int DIMP = I::DIMP, PD = I::PD, PF = DIMP + 4;
  extern __shared__ __align__(16) float smem[];
  float* q_s = smem;                              // [16][PF]
  float* k_s = q_s + kDmTokens * PF;
  float* a_s = k_s + kDmTokens * PF;              // logarithms (base 2) of the decays, then their sums from the start
  float* m_s = a_s + kDmTokens * PF;              // [16][17]: M
  float* am_s = m_s + kDmTokens * 17;             // [16][17]: A
  float* beta_s = am_s + kDmTokens * 17;          // [16]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int h = blockIdx.y, kvh = h / (p.heads / p.kv_heads), dim = p.dim;
  GlaSpan sp;
  if (!gla_span(p, blockIdx.x, sp)) return;
  const int tb = sp.t0, nt = sp.t1 - sp.t0;
  const TR* raw = reinterpret_cast<const TR*>(p.raw);
  const float rate2 = expf(p.a_log[h]) * 1.4426950408889634f;
  for (int i = tid; i < kDmTokens * DIMP; i += kDmThreads) {
    const int tt = i / DIMP, d = i - tt * DIMP;
    float q = 0.f, k = 0.f, l = 0.f;
    if (tt < nt && d < dim) {
      const float* row = p.act + (size_t)(tb + tt) * p.lda + (size_t)kvh * dim + d;
      q = row[p.q_off];
      k = row[p.k_off];
      float z;
      if (CHANNEL) z = p.zs[(size_t)(tb + tt) * p.ldz + (size_t)h * dim + d];
      else z = to_float<TR>(raw[(size_t)(tb + tt) * p.ldr + p.a_off + h]) + p.dt_bias[h];
      l = -rate2 * (z > 20.f ? z : log1pf(expf(z)));
    }
    q_s[tt * PF + d] = q;
    k_s[tt * PF + d] = k;
    a_s[tt * PF + d] = l;
  }
  if (tid < kDmTokens)
    beta_s[tid] = tid < nt ? 1.f / (1.f + expf(-to_float<TR>(raw[(size_t)(tb + tid) * p.ldr + p.b_off + h]))) : 0.f;
  __syncthreads();
  // unit vectors: two tokens a warp; sums of logarithms: a row of the state a thread
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int tt = warp * 2 + i;
    float sq = 0.f, sk = 0.f;
#pragma unroll
    for (int j = 0; j < DIMP / 32; ++j) {
      const float q = q_s[tt * PF + lane + 32 * j], k = k_s[tt * PF + lane + 32 * j];
      sq = fmaf(q, q, sq);
      sk = fmaf(k, k, sk);
    }
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    const float rq = p.q_scale / sqrtf(sq + 1e-6f), rk = 1.f / sqrtf(sk + 1e-6f);
#pragma unroll
    for (int j = 0; j < DIMP / 32; ++j) {
      q_s[tt * PF + lane + 32 * j] *= rq;
      k_s[tt * PF + lane + 32 * j] *= rk;
    }
  }
  if (tid < DIMP) {
    float run = 0.f;
#pragma unroll
    for (int tt = 0; tt < kDmTokens; ++tt) {
      run += a_s[tt * PF + tid];
      a_s[tt * PF + tid] = run;
    }
  }
  __syncthreads();
  unsigned char* image = p.images + ((size_t)blockIdx.x * p.heads + h) * I::bytes;
  for (int i = tid; i < kDmTokens * (DIMP / 2); i += kDmThreads) {
    const int tt = i / (DIMP / 2), d = (i - tt * (DIMP / 2)) * 2;
    const float2 q = *reinterpret_cast<const float2*>(q_s + tt * PF + d), k = *reinterpret_cast<const float2*>(k_s + tt * PF + d);
    const float2 a = *reinterpret_cast<const float2*>(a_s + tt * PF + d);
    const float2 e = *reinterpret_cast<const float2*>(a_s + (kDmTokens - 1) * PF + d);
    const float p0 = exp2_fast(a.x), p1 = exp2_fast(a.y);
    unsigned char* at = image + (tt * PD + d) * 2;
    uint32_t hi, lo;
    split_pair(k.x * p0, k.y * p1, hi, lo);
    *reinterpret_cast<uint32_t*>(at) = hi;
    *reinterpret_cast<uint32_t*>(at + I::kTile) = lo;
    split_pair(q.x * p0, q.y * p1, hi, lo);
    *reinterpret_cast<uint32_t*>(at + 2 * I::kTile) = hi;
    *reinterpret_cast<uint32_t*>(at + 3 * I::kTile) = lo;
    split_pair(k.x * exp2_fast(e.x - a.x), k.y * exp2_fast(e.y - a.y), hi, lo);
    *reinterpret_cast<uint32_t*>(at + 4 * I::kTile) = hi;
    *reinterpret_cast<uint32_t*>(at + 5 * I::kTile) = lo;
    if (tt == kDmTokens - 1) *reinterpret_cast<float2*>(image + I::kKeep + d * 4) = make_float2(p0, p1);
  }
  {
    // M and A: a half-warp per earlier token s (4 KPW channels a lane) against all tokens from it on
    const int s = warp * 2 + (lane >> 4), part = (lane & 15) * 4;
    float4 ks[KPW], as[KPW];
#pragma unroll
    for (int j = 0; j < KPW; ++j) {
      ks[j] = *reinterpret_cast<const float4*>(k_s + s * PF + part + 64 * j);
      as[j] = *reinterpret_cast<const float4*>(a_s + s * PF + part + 64 * j);
    }
    for (int t = warp * 2; t < kDmTokens; ++t) {
      float m = 0.f, am = 0.f;
#pragma unroll
      for (int j = 0; j < KPW; ++j) {
        const float4 kt = *reinterpret_cast<const float4*>(k_s + t * PF + part + 64 * j);
        const float4 qt = *reinterpret_cast<const float4*>(q_s + t * PF + part + 64 * j);
        const float4 at = *reinterpret_cast<const float4*>(a_s + t * PF + part + 64 * j);
        const float w0 = ks[j].x * exp2_fast(fminf(at.x - as[j].x, 0.f)), w1 = ks[j].y * exp2_fast(fminf(at.y - as[j].y, 0.f));
        const float w2 = ks[j].z * exp2_fast(fminf(at.z - as[j].z, 0.f)), w3 = ks[j].w * exp2_fast(fminf(at.w - as[j].w, 0.f));
        m = fmaf(kt.x, w0, fmaf(kt.y, w1, fmaf(kt.z, w2, fmaf(kt.w, w3, m))));
        am = fmaf(qt.x, w0, fmaf(qt.y, w1, fmaf(qt.z, w2, fmaf(qt.w, w3, am))));
      }
#pragma unroll
      for (int o = 8; o > 0; o >>= 1) {
        m += __shfl_xor_sync(0xffffffffu, m, o);
        am += __shfl_xor_sync(0xffffffffu, am, o);
      }
      if ((lane & 15) == 0) {
        m_s[t * 17 + s] = m;
        am_s[t * 17 + s] = am;
      }
    }
  }
  __syncthreads();
  if (tid < kDmTokens) {
    // column tid of T by forward substitution
    float x[kDmTokens];
    const float own = beta_s[tid];
#pragma unroll
    for (int t = 0; t < kDmTokens; ++t) {
      float sum = 0.f;
#pragma unroll
      for (int s = 0; s < t; ++s) sum = fmaf(m_s[t * 17 + s], x[s], sum);
      x[t] = t < tid ? 0.f : t == tid ? own : -beta_s[t] * sum;
    }
#pragma unroll
    for (int t = 0; t < kDmTokens; ++t) {
      const __nv_bfloat16 hi = __float2bfloat16_rn(x[t]);
      __nv_bfloat16* at = reinterpret_cast<__nv_bfloat16*>(image + I::kT) + t * kDmPT + tid;
      *at = hi;
      at[kDmTokens * kDmPT] = __float2bfloat16_rn(x[t] - __bfloat162float(hi));
    }
  } else if (warp == 1) {
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int t = i * 2 + (lane >> 4), s = lane & 15;
      const float x = s <= t ? am_s[t * 17 + s] : 0.f;
      const __nv_bfloat16 hi = __float2bfloat16_rn(x);
      __nv_bfloat16* at = reinterpret_cast<__nv_bfloat16*>(image + I::kA) + t * kDmPT + s;
      *at = hi;
      at[kDmTokens * kDmPT] = __float2bfloat16_rn(x - __bfloat162float(hi));
    }
  }
}

// VG: groups of 16 value columns a block
template <int KPW, int STAGES, int VG>
__global__ void __launch_bounds__(128 * VG)
delta_chain_kernel(const DeltaMmaParams p) {
  pdl_trigger();
  pdl_wait();
  using I = DmImage<KPW>;
  constexpr int PD = I::PD, NT = 2 * KPW;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  float4* red = reinterpret_cast<float4*>(smem_raw + STAGES * I::bytes);      // [VG column groups][4 quarters][4][32]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3, mi = lane >> 3;
  const int vg = warp >> 2, ks = warp & 3;        // this warp's group of value columns and quarter of the rows
  const int h = blockIdx.y, seq = blockIdx.z, vdim = p.vdim, dim = p.dim;
  const int t0 = p.q_start[seq], t1 = p.q_start[seq + 1];
  if (t0 >= t1) return;
  const int slot = p.slot_ids[seq];
  if (slot < 0 || slot >= p.n_slots) {
    if (tid == 0) set_status(p.status, kBadSequence, seq, slot);
    return;
  }
  int first = 0;
  for (int b = 0; b < seq; ++b) first += (p.q_start[b + 1] - p.q_start[b] + kDmTokens - 1) / kDmTokens;
  const int groups = (t1 - t0 + kDmTokens - 1) / kDmTokens;
  const uint32_t base = (uint32_t)__cvta_generic_to_shared(smem_raw);
  auto request = [&](int grp) {
    if (grp < groups) {
      const unsigned char* src = p.images + ((size_t)(first + grp) * p.heads + h) * I::bytes;
      const uint32_t dst = base + (grp % STAGES) * I::bytes;
      #pragma unroll
      for (int i = 0; i < I::bytes; i += 128 * VG * 16)
        if (i + tid * 16 < I::bytes) cp_async16_zfill(dst + i + tid * 16, src + i + tid * 16, true);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
#pragma unroll
  for (int i = 0; i < STAGES - 1; ++i) request(i);

  float* st = p.state + ((size_t)slot * p.heads + h) * (size_t)dim * vdim;
  const int va = blockIdx.x * (16 * VG) + vg * 16 + g, vb = va + 8;             // this thread's value columns
  float S[NT][4];
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int v = i < 2 ? va : vb, d = (ks * NT + n) * 8 + 2 * tq + (i & 1);
      S[n][i] = v < vdim && d < dim ? st[(size_t)d * vdim + v] : 0.f;
    }
  // the first quarter's warps bring the values into the sums: value (column, token) pairs as a fragment has them
  const float* v_src = p.act + p.v_off + (size_t)h * vdim;
  float V[2][4];
  auto values = [&](int grp) {
    if (ks != 0) return;
#pragma unroll
    for (int nn = 0; nn < 2; ++nn)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int t = t0 + grp * kDmTokens + nn * 8 + 2 * tq + (i & 1), v = i < 2 ? va : vb;
        V[nn][i] = t < t1 && v < vdim ? v_src[(size_t)t * p.lda + v] : 0.f;
      }
  };
#pragma unroll
  for (int i = 0; i < 8; ++i) V[i >> 2][i & 3] = 0.f;
  values(0);
  const uint32_t row_b = (lane & 7) + (mi >> 1) * 8, col_b = (mi & 1) * 8;    // rows are tokens read out, columns k
  for (int grp = 0; grp < groups; ++grp) {
    asm volatile("cp.async.wait_group %0;" ::"n"(STAGES - 2) : "memory");
    __syncthreads();                              // this image is there, the last one is read
    request(grp + STAGES - 1);
    const uint32_t im = base + (grp % STAGES) * I::bytes;
    float W[4][4];                                // S^T (k P) - v, S^T (q P): two tiles of eight tokens each
#pragma unroll
    for (int nn = 0; nn < 2; ++nn)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        W[nn][i] = -V[nn][i];
        W[2 + nn][i] = 0.f;
      }
    if (grp + 1 < groups) values(grp + 1);
#pragma unroll
    for (int kk = 0; kk < KPW; ++kk) {
      uint32_t sh[4], sl[4];
      split_pair(S[2 * kk][0], S[2 * kk][1], sh[0], sl[0]);
      split_pair(S[2 * kk][2], S[2 * kk][3], sh[1], sl[1]);
      split_pair(S[2 * kk + 1][0], S[2 * kk + 1][1], sh[2], sl[2]);
      split_pair(S[2 * kk + 1][2], S[2 * kk + 1][3], sh[3], sl[3]);
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        uint32_t bh[4], bl[4];
        const uint32_t at = im + 2 * x * I::kTile + (row_b * PD + col_b + (ks * KPW + kk) * 16) * 2;
        ldsm4(at, bh[0], bh[1], bh[2], bh[3]);
        ldsm4(at + I::kTile, bl[0], bl[1], bl[2], bl[3]);
#pragma unroll
        for (int nn = 0; nn < 2; ++nn) mma16816(W[2 * x + nn], sl[0], sl[1], sl[2], sl[3], bh[2 * nn], bh[2 * nn + 1]);
#pragma unroll
        for (int nn = 0; nn < 2; ++nn) mma16816(W[2 * x + nn], sh[0], sh[1], sh[2], sh[3], bl[2 * nn], bl[2 * nn + 1]);
#pragma unroll
        for (int nn = 0; nn < 2; ++nn) mma16816(W[2 * x + nn], sh[0], sh[1], sh[2], sh[3], bh[2 * nn], bh[2 * nn + 1]);
      }
    }
    float4* mine = red + (size_t)(vg * 4 + ks) * 4 * 32 + lane;
#pragma unroll
    for (int x = 0; x < 4; ++x) mine[x * 32] = make_float4(W[x][0], W[x][1], W[x][2], W[x][3]);
    asm volatile("bar.sync %0, 128;" ::"r"(1 + vg) : "memory");
    const float4* all = red + (size_t)vg * 16 * 32 + lane;
    auto total = [&](int x) {
      const float4 a = all[x * 32], b = all[(4 + x) * 32], c = all[(8 + x) * 32], d = all[(12 + x) * 32];
      return make_float4((a.x + b.x) + (c.x + d.x), (a.y + b.y) + (c.y + d.y), (a.z + b.z) + (c.z + d.z), (a.w + b.w) + (c.w + d.w));
    };
    // U^T = (V - W)^T T^T
    uint32_t xh[4], xl[4];
    {
      const float4 r0 = total(0), r1 = total(1);
      split_pair(-r0.x, -r0.y, xh[0], xl[0]);
      split_pair(-r0.z, -r0.w, xh[1], xl[1]);
      split_pair(-r1.x, -r1.y, xh[2], xl[2]);
      split_pair(-r1.z, -r1.w, xh[3], xl[3]);
    }
    float U[2][4];
    {
      uint32_t bh[4], bl[4];
      const uint32_t at = im + I::kT + (row_b * kDmPT + col_b) * 2;
      ldsm4(at, bh[0], bh[1], bh[2], bh[3]);
      ldsm4(at + I::kSmall, bl[0], bl[1], bl[2], bl[3]);
#pragma unroll
      for (int nn = 0; nn < 2; ++nn) {
#pragma unroll
        for (int i = 0; i < 4; ++i) U[nn][i] = 0.f;
        mma16816(U[nn], xl[0], xl[1], xl[2], xl[3], bh[2 * nn], bh[2 * nn + 1]);
        mma16816(U[nn], xh[0], xh[1], xh[2], xh[3], bl[2 * nn], bl[2 * nn + 1]);
        mma16816(U[nn], xh[0], xh[1], xh[2], xh[3], bh[2 * nn], bh[2 * nn + 1]);
      }
    }
    split_pair(U[0][0], U[0][1], xh[0], xl[0]);
    split_pair(U[0][2], U[0][3], xh[1], xl[1]);
    split_pair(U[1][0], U[1][1], xh[2], xl[2]);
    split_pair(U[1][2], U[1][3], xh[3], xl[3]);
    // S^T <- S^T diag(P_15) + U^T (k P_15 / P)
    const float* keep = reinterpret_cast<const float*>(smem_raw + (grp % STAGES) * I::bytes + I::kKeep) + ks * KPW * 16 + 2 * tq;
#pragma unroll
    for (int kk = 0; kk < KPW; ++kk) {
      uint32_t bh[4], bl[4];
      const uint32_t at = im + 4 * I::kTile + (((lane & 7) + (mi & 1) * 8) * PD + (ks * KPW + kk) * 16 + (mi >> 1) * 8) * 2;
      ldsm4_trans(at, bh[0], bh[1], bh[2], bh[3]);
      ldsm4_trans(at + I::kTile, bl[0], bl[1], bl[2], bl[3]);
#pragma unroll
      for (int nn = 0; nn < 2; ++nn) {
        float* c = S[2 * kk + nn];
        const float2 f = *reinterpret_cast<const float2*>(keep + kk * 16 + nn * 8);
        c[0] *= f.x;
        c[1] *= f.y;
        c[2] *= f.x;
        c[3] *= f.y;
        mma16816(c, xl[0], xl[1], xl[2], xl[3], bh[2 * nn], bh[2 * nn + 1]);
        mma16816(c, xh[0], xh[1], xh[2], xh[3], bl[2 * nn], bl[2 * nn + 1]);
        mma16816(c, xh[0], xh[1], xh[2], xh[3], bh[2 * nn], bh[2 * nn + 1]);
      }
    }
    if (ks >= 2) {                                // eight tokens' results each for two of the quarters' warps
      const int nn = ks - 2;
      const float4 w = total(2 + nn);
      float O[4] = {w.x, w.y, w.z, w.w};
      uint32_t bh[4], bl[4];
      const uint32_t at = im + I::kA + (row_b * kDmPT + col_b) * 2;
      ldsm4(at, bh[0], bh[1], bh[2], bh[3]);
      ldsm4(at + I::kSmall, bl[0], bl[1], bl[2], bl[3]);
      const uint32_t h0 = nn ? bh[2] : bh[0], h1 = nn ? bh[3] : bh[1], l0 = nn ? bl[2] : bl[0], l1 = nn ? bl[3] : bl[1];
      mma16816(O, xl[0], xl[1], xl[2], xl[3], h0, h1);
      mma16816(O, xh[0], xh[1], xh[2], xh[3], l0, l1);
      mma16816(O, xh[0], xh[1], xh[2], xh[3], h0, h1);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int t = t0 + grp * kDmTokens + nn * 8 + 2 * tq + (i & 1), v = i < 2 ? va : vb;
        if (t < t1 && v < vdim) p.out[(size_t)t * p.ldo + (size_t)h * vdim + v] = O[i];
      }
    }
  }
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int v = i < 2 ? va : vb, d = (ks * NT + n) * 8 + 2 * tq + (i & 1);
      if (v < vdim && d < dim) st[(size_t)d * vdim + v] = S[n][i];
    }
}

}  // namespace leone

using namespace leone;

// Bytes of scratch per (16 tokens of a sequence, head); 0: the tensor-core form does not take the size.
extern "C" int leone_gated_delta_mma_image(int dim) {
  return dim <= 0 || dim > 128 ? 0 : dim <= 64 ? DmImage<1>::bytes : DmImage<2>::bytes;
}

// The arguments of leone_gated_delta.  images: scratch of n_groups x heads images, n_groups = sum over sequences of
// ceil(tokens / 16), 16-byte aligned.
extern "C" int leone_gated_delta_mma(const float* act, int lda, int q_off, int k_off, int v_off, int raw_dtype, const void* raw,
                                     int ldr, int a_off, int b_off, const float* zs, int ldz, const float* a_log,
                                     const float* dt_bias, float q_scale, float* out, int ldo, float* state,
                                     const int* q_start, const int* slot_ids, int n_seqs, int heads, int kv_heads, int dim,
                                     int vdim, int n_slots, void* images, int n_groups, int* status, cudaStream_t stream) {
  if (n_seqs <= 0 || n_groups <= 0) return 0;
  if (heads <= 0 || kv_heads <= 0 || heads % kv_heads != 0 || leone_gated_delta_mma_image(dim) == 0 || vdim <= 0 || heads > 65535 ||
      n_seqs > 65535 || images == nullptr)
    return kRefusedSize;
  if (raw_dtype != 0 && raw_dtype != 1) return kRefusedDtype;
  if ((uintptr_t)images & 15) return kRefusedAlignment;
  DeltaMmaParams p = {act, lda, q_off, k_off, v_off, raw, ldr, a_off, b_off, zs, ldz, a_log, dt_bias, q_scale, out, ldo, state,
                      q_start, slot_ids, heads, kv_heads, dim, vdim, n_seqs, n_slots, kDmTokens, (unsigned char*)images, status};
  int code = 0;
#define OPERANDS(KPW, CH, TR)                                                                                              \
  code = launch_kernel(delta_operands_kernel<KPW, CH, TR>, dim3(n_groups, heads), dim3(kDmThreads),                       \
                       sizeof(float) * (size_t)kDmTokens * (3 * (DmImage<KPW>::DIMP + 4) + 2 * 17 + 1), stream, p)
#define RUN(KPW, ST, VG)                                                                                                     \
  do {                                                                                                                     \
    if (zs != nullptr && raw_dtype == 0) OPERANDS(KPW, true, float);                                                       \
    else if (zs != nullptr) OPERANDS(KPW, true, __nv_bfloat16);                                                            \
    else if (raw_dtype == 0) OPERANDS(KPW, false, float);                                                                  \
    else OPERANDS(KPW, false, __nv_bfloat16);                                                                              \
    if (code != 0) return code;                                                                                            \
    constexpr size_t smem = (size_t)ST * DmImage<KPW>::bytes + VG * 4 * 4 * 32 * sizeof(float4);                           \
    static bool configured = false;                                                                                        \
    if (!configured) {                                                                                                     \
      cudaFuncSetAttribute(delta_chain_kernel<KPW, ST, VG>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);       \
      configured = true;                                                                                                   \
    }                                                                                                                      \
    return launch_kernel(delta_chain_kernel<KPW, ST, VG>, dim3((vdim + 16 * VG - 1) / (16 * VG), heads, n_seqs),           \
                         dim3(128 * VG), smem, stream, p);                                                                 \
  } while (0)
  // a chain of groups is bound by its latency, so that few columns a block and many blocks are fastest while the SMs
  // last (16 heads of 128: 182 us against 229); beyond, two groups of columns share the images' copies (32 heads: 272
  // against 347)
  const long long narrow = (long long)((vdim + 15) / 16) * heads * n_seqs;
  if (narrow <= 148) {
    if (dim <= 64) RUN(1, 4, 1);
    RUN(2, 4, 1);
  }
  if (dim <= 64) RUN(1, 4, 2);
  RUN(2, 3, 2);
#undef RUN
#undef OPERANDS
}
