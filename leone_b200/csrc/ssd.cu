// The Mamba-2 recurrence (state-space duality: one decay per head and token) and the gated, grouped norm behind it.
//
//   per head, S: [n_state, vdim] fp32, per request, head h reading group h / (heads / groups) of B and C:
//     d_t = softplus(dt_t + dt_bias_h)                    a_t = exp(-exp(A_log_h) d_t)
//     S_t = a_t S_(t-1) + (d_t B_t) x_t^T                 y_t = S_t^T C_t + D_h x_t
//
// x, B and C arrive as activations (after their convolution and silu), dt as a raw projection.  Everything here is
// fp32.  The state is read from and written back to the request's state slot and the walk is token by token in the
// same order whatever the cut.  A step of one token per sequence (decode) has a form that asks for all of a head's state at
// once; prompt portions of bfloat16 runs have one of their own (ssd_mma.cu).
//
// A block owns (a slice of value columns, head, sequence).  A value column's rows are dealt to P lanes (row i belongs
// to lane part i % P), DPT rows each in registers; the sum over rows is P-lane shuffles.  Tokens are staged 16 at a time,
// in shared memory.
//
// (Dao and Gu, "Transformers are SSMs: Generalized Models and Efficient Algorithms Through Structured State Space
// Duality" describes this recurrence.)
//
// grouped_gate_norm: y * silu(z), RMS-normed in equal groups of columns, times a weight.
#include "ssd_parts.cuh"

namespace leone {

constexpr int kSsdTokens = 16;
constexpr int kSsdThreads = 128;

template <int P> __device__ __forceinline__ float lanes_sum(float v) {
#pragma unroll
  for (int o = P / 2; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

template <typename TA, typename TR, int DPT, int P>
__global__ void __launch_bounds__(kSsdThreads)
ssd_walk_kernel(const SsdParams p) {
  pdl_trigger();
  pdl_wait();
  constexpr int ROWS = DPT * P;                 // rows with padding
  constexpr int CW = 32 / P;                    // value columns per warp
  constexpr int COLS = CW * (kSsdThreads / 32);
  extern __shared__ __align__(16) float smem[];
  float* b_s = smem;                            // [tokens][ROWS]: B
  float* c_s = b_s + kSsdTokens * ROWS;         // [tokens][ROWS]: C
  float* x_s = c_s + kSsdTokens * ROWS;         // [tokens][COLS]
  float* d_s = x_s + kSsdTokens * COLS;         // [tokens] step, [tokens] decay
  const TA* act = reinterpret_cast<const TA*>(p.act);
  const TR* raw = reinterpret_cast<const TR*>(p.raw);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, part = lane % P;
  const int col_local = warp * CW + lane / P;
  const int h = blockIdx.y, s = blockIdx.z, v0 = blockIdx.x * COLS, col = v0 + col_local;
  const int n_state = p.n_state, vdim = p.vdim;
  const int t0 = p.q_start[s], t1 = p.q_start[s + 1];
  if (t0 >= t1) return;
  const int slot = p.slot_ids[s];
  if (slot < 0 || slot >= p.n_slots) {
    if (tid == 0) set_status(p.status, kBadSequence, s, slot);
    return;
  }
  const int grp = h / (p.heads / p.groups);
  float* st = p.state + ((size_t)slot * p.heads + h) * (size_t)n_state * vdim;
  float S[DPT];
#pragma unroll
  for (int r = 0; r < DPT; ++r) {
    const int i = part + P * r;
    S[r] = (i < n_state && col < vdim) ? st[(size_t)i * vdim + col] : 0.f;
  }
  const float rate = expf(p.a_log[h]), bias = p.dt_bias[h], skip = p.d_skip[h];
  for (int tb = t0; tb < t1; tb += kSsdTokens) {
    const int nt = min(kSsdTokens, t1 - tb);
    __syncthreads();
    for (int i = tid; i < nt * ROWS; i += kSsdThreads) {
      const int tt = i / ROWS, d = i - tt * ROWS;
      const TA* row = act + (size_t)(tb + tt) * p.lda + (size_t)grp * n_state + d;
      b_s[i] = d < n_state ? to_float<TA>(row[p.b_off]) : 0.f;
      c_s[i] = d < n_state ? to_float<TA>(row[p.c_off]) : 0.f;
    }
    for (int i = tid; i < nt * COLS; i += kSsdThreads) {
      const int tt = i / COLS, c = i - tt * COLS;
      x_s[i] = v0 + c < vdim ? to_float<TA>(act[(size_t)(tb + tt) * p.lda + p.x_off + (size_t)h * vdim + v0 + c]) : 0.f;
    }
    if (tid < nt) {
      const float d = ssd_step(to_float<TR>(raw[(size_t)(tb + tid) * p.ldr + p.dt_off + h]), bias);
      d_s[tid] = d;
      d_s[kSsdTokens + tid] = expf(-rate * d);
    }
    __syncthreads();
    for (int tt = 0; tt < nt; ++tt) {
      const float x = x_s[tt * COLS + col_local], dx = d_s[tt] * x, a = d_s[kSsdTokens + tt];
      const float* bb = b_s + tt * ROWS + part;
      const float* cc = c_s + tt * ROWS + part;
      float y4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int r = 0; r < DPT; ++r) {
        S[r] = fmaf(a, S[r], bb[P * r] * dx);
        y4[r & 3] = fmaf(S[r], cc[P * r], y4[r & 3]);
      }
      const float y = lanes_sum<P>((y4[0] + y4[1]) + (y4[2] + y4[3]));
      if (part == 0 && col < vdim) p.out[(size_t)(tb + tt) * p.ldo + (size_t)h * vdim + col] = fmaf(skip, x, y);
    }
  }
  if (col < vdim) {
#pragma unroll
    for (int r = 0; r < DPT; ++r) {
      const int i = part + P * r;
      if (i < n_state) st[(size_t)i * vdim + col] = S[r];
    }
  }
}

// One token a sequence (decode): a block per (head, sequence).  A thread owns four neighbouring value columns of the rows
// r, r + R, r + 2 R, ... and asks for up to eight of its rows of the state before it touches any; the row groups' partial
// read-outs are summed in shared memory, in order.  Rows of the state must start on 16-byte boundaries.
constexpr int kSsdStepThreads = 256, kSsdStepAhead = 8;

template <typename TA, typename TR>
__global__ void __launch_bounds__(kSsdStepThreads)
ssd_step_kernel(const SsdParams p) {
  pdl_trigger();
  pdl_wait();
  __shared__ __align__(16) float4 part_s[kSsdStepThreads];
  const int tid = threadIdx.x, h = blockIdx.x, s = blockIdx.y, n_state = p.n_state, vdim = p.vdim;
  const int quads = vdim >> 2, R = kSsdStepThreads / quads, r = tid / quads, c = (tid - r * quads) * 4;
  const int t = p.q_start[s];
  if (t >= p.q_start[s + 1]) return;
  const int slot = p.slot_ids[s];
  if (slot < 0 || slot >= p.n_slots) {
    if (tid == 0) set_status(p.status, kBadSequence, s, slot);
    return;
  }
  const TA* row = reinterpret_cast<const TA*>(p.act) + (size_t)t * p.lda;
  const TA* bc = row + (size_t)(h / (p.heads / p.groups)) * n_state;
  const float d = ssd_step(to_float<TR>(reinterpret_cast<const TR*>(p.raw)[(size_t)t * p.ldr + p.dt_off + h]), p.dt_bias[h]);
  const float a = expf(-expf(p.a_log[h]) * d);
  float x[4], y[4] = {0.f, 0.f, 0.f, 0.f};
  if (r < R) {
#pragma unroll
    for (int e = 0; e < 4; ++e) x[e] = to_float<TA>(row[p.x_off + (size_t)h * vdim + c + e]);
    float* st = p.state + ((size_t)slot * p.heads + h) * (size_t)n_state * vdim + c;
    for (int i0 = r; i0 < n_state; i0 += R * kSsdStepAhead) {
      float4 S[kSsdStepAhead];
      float b[kSsdStepAhead], q[kSsdStepAhead];
#pragma unroll
      for (int j = 0; j < kSsdStepAhead; ++j) {
        const int i = i0 + j * R;
        if (i < n_state) {
          S[j] = *reinterpret_cast<const float4*>(st + (size_t)i * vdim);
          b[j] = to_float<TA>(bc[p.b_off + i]) * d;
          q[j] = to_float<TA>(bc[p.c_off + i]);
        }
      }
#pragma unroll
      for (int j = 0; j < kSsdStepAhead; ++j) {
        const int i = i0 + j * R;
        if (i < n_state) {
          S[j].x = fmaf(a, S[j].x, b[j] * x[0]);
          S[j].y = fmaf(a, S[j].y, b[j] * x[1]);
          S[j].z = fmaf(a, S[j].z, b[j] * x[2]);
          S[j].w = fmaf(a, S[j].w, b[j] * x[3]);
          y[0] = fmaf(S[j].x, q[j], y[0]);
          y[1] = fmaf(S[j].y, q[j], y[1]);
          y[2] = fmaf(S[j].z, q[j], y[2]);
          y[3] = fmaf(S[j].w, q[j], y[3]);
          *reinterpret_cast<float4*>(st + (size_t)i * vdim) = S[j];
        }
      }
    }
    part_s[r * quads + (c >> 2)] = make_float4(y[0], y[1], y[2], y[3]);
  }
  __syncthreads();
  const float* part = reinterpret_cast<const float*>(part_s);
  for (int v = tid; v < vdim; v += kSsdStepThreads) {
    float sum = 0.f;
    for (int g = 0; g < R; ++g) sum += part[g * vdim + v];
    p.out[(size_t)t * p.ldo + (size_t)h * vdim + v] = fmaf(p.d_skip[h], to_float<TA>(row[p.x_off + (size_t)h * vdim + v]), sum);
  }
}

// One block per (token, group): out = (y * silu(z)) / rms over the group * w.
template <typename TZ, typename T>
__global__ void __launch_bounds__(256)
grouped_gate_norm_kernel(const float* __restrict__ y, int ldy, const TZ* __restrict__ z, int ldz, const float* __restrict__ w,
                         T* __restrict__ out, int ldo, int group, float eps) {
  pdl_trigger();
  pdl_wait();
  __shared__ float scratch[33];
  extern __shared__ float row_s[];              // [group]
  const size_t t = blockIdx.x;
  const int c0 = blockIdx.y * group;
  float ss = 0.f;
  for (int c = threadIdx.x; c < group; c += blockDim.x) {
    const float g = to_float<TZ>(z[t * ldz + c0 + c]);
    const float v = y[t * ldy + c0 + c] * (g / (1.f + expf(-g)));
    row_s[c] = v;
    ss = fmaf(v, v, ss);
  }
  ss = block_sum(ss, scratch);
  const float r = 1.f / sqrtf(ss / (float)group + eps);
  for (int c = threadIdx.x; c < group; c += blockDim.x) out[t * ldo + c0 + c] = from_float<T>(row_s[c] * r * w[c0 + c]);
}

// The same with four columns a thread, a row's group in registers (up to 4 x 4 columns a thread).
template <typename T> __device__ __forceinline__ float4 load4(const T* p);
template <> __device__ __forceinline__ float4 load4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <> __device__ __forceinline__ float4 load4<__nv_bfloat16>(const __nv_bfloat16* p) {
  const uint2 r = *reinterpret_cast<const uint2*>(p);
  return make_float4(__uint_as_float(r.x << 16), __uint_as_float(r.x & 0xffff0000u), __uint_as_float(r.y << 16),
                     __uint_as_float(r.y & 0xffff0000u));
}
template <typename T> __device__ __forceinline__ void store4(T* p, float4 v);
template <> __device__ __forceinline__ void store4<float>(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
template <> __device__ __forceinline__ void store4<__nv_bfloat16>(__nv_bfloat16* p, float4 v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  uint2 r;
  r.x = *reinterpret_cast<const uint32_t*>(&a);
  r.y = *reinterpret_cast<const uint32_t*>(&b);
  *reinterpret_cast<uint2*>(p) = r;
}

template <typename TZ, typename T, int R>
__global__ void __launch_bounds__(256)
grouped_gate_norm_vec_kernel(const float* __restrict__ y, int ldy, const TZ* __restrict__ z, int ldz,
                             const float* __restrict__ w, T* __restrict__ out, int ldo, int group, float eps) {
  pdl_trigger();
  pdl_wait();
  __shared__ float scratch[33];
  const size_t t = blockIdx.x;
  const int c0 = blockIdx.y * group;
  float4 v[R];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 4;
    v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < group) {
      v[i] = load4<float>(y + t * ldy + c0 + c);
      const float4 g = load4<TZ>(z + t * ldz + c0 + c);
      v[i].x *= g.x / (1.f + expf(-g.x));
      v[i].y *= g.y / (1.f + expf(-g.y));
      v[i].z *= g.z / (1.f + expf(-g.z));
      v[i].w *= g.w / (1.f + expf(-g.w));
    }
    ss = fmaf(v[i].x, v[i].x, fmaf(v[i].y, v[i].y, fmaf(v[i].z, v[i].z, fmaf(v[i].w, v[i].w, ss))));
  }
  ss = block_sum(ss, scratch);
  const float r = 1.f / sqrtf(ss / (float)group + eps);
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 4;
    if (c < group) {
      const float4 ww = load4<float>(w + c0 + c);
      store4<T>(out + t * ldo + c0 + c, make_float4(v[i].x * r * ww.x, v[i].y * r * ww.y, v[i].z * r * ww.z, v[i].w * r * ww.w));
    }
  }
}

}  // namespace leone

using namespace leone;

// act: `act_dtype` [n_tokens, lda] with x (heads x vdim), B and C (groups x n_state each) at their column offsets; raw:
// `raw_dtype` [n_tokens, ldr] with one dt per head at dt_off; out: fp32 [n_tokens, ldo], D x included.  one_token: every
// sequence of the step brings one token.
extern "C" int leone_ssd(int act_dtype, const void* act, int lda, int x_off, int b_off, int c_off, int raw_dtype,
                         const void* raw, int ldr, int dt_off, const float* a_log, const float* dt_bias,
                         const float* d_skip, float* out, int ldo, float* state, const int* q_start, const int* slot_ids,
                         int n_seqs, int heads, int groups, int n_state, int vdim, int n_slots, int one_token,
                         int* status, cudaStream_t stream) {
  if (n_seqs <= 0) return 0;
  if (heads <= 0 || groups <= 0 || heads % groups != 0 || n_state <= 0 || n_state > 512 || vdim <= 0 || heads > 65535 ||
      n_seqs > 65535)
    return kRefusedSize;
  if ((act_dtype | 1) != 1 || (raw_dtype | 1) != 1) return kRefusedDtype;
  SsdParams p = {act, lda, x_off, b_off, c_off, raw, ldr, dt_off, a_log, dt_bias, d_skip, out, ldo, state, q_start,
                 slot_ids, n_seqs, heads, groups, n_state, vdim, n_slots, status, 0, nullptr, nullptr};
  if (one_token && vdim % 4 == 0 && vdim <= 4 * kSsdStepThreads && ((uintptr_t)state & 15) == 0) {
#define STEP(TA, TR) return launch_kernel(ssd_step_kernel<TA, TR>, dim3(heads, n_seqs), dim3(kSsdStepThreads), 0, stream, p)
    if (act_dtype == 0 && raw_dtype == 0) STEP(float, float);
    if (act_dtype == 0) STEP(float, __nv_bfloat16);
    if (raw_dtype == 0) STEP(__nv_bfloat16, float);
    STEP(__nv_bfloat16, __nv_bfloat16);
#undef STEP
  }
#define SSD_AS(TA, TR, DPT, P)                                                                                        \
  {                                                                                                                   \
    constexpr int cols = (32 / P) * (kSsdThreads / 32);                                                               \
    const size_t smem = sizeof(float) * (size_t)kSsdTokens * (2 * DPT * P + cols + 2);                                \
    static bool configured = false;                                                                                   \
    if (!configured && smem > 48 * 1024) {                                                                            \
      cudaFuncSetAttribute(ssd_walk_kernel<TA, TR, DPT, P>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);  \
      configured = true;                                                                                              \
    }                                                                                                                 \
    return launch_kernel(ssd_walk_kernel<TA, TR, DPT, P>, dim3((vdim + cols - 1) / cols, heads, n_seqs),              \
                         dim3(kSsdThreads), smem, stream, p);                                                         \
  }
#define SSD(DPT, P)                                                          \
  {                                                                          \
    if (act_dtype == 0 && raw_dtype == 0) SSD_AS(float, float, DPT, P)       \
    if (act_dtype == 0) SSD_AS(float, __nv_bfloat16, DPT, P)                 \
    if (raw_dtype == 0) SSD_AS(__nv_bfloat16, float, DPT, P)                 \
    SSD_AS(__nv_bfloat16, __nv_bfloat16, DPT, P)                             \
  }
  if (n_state <= 16) SSD(4, 4)
  if (n_state <= 32) SSD(8, 4)
  if (n_state <= 64) SSD(16, 4)
  if (n_state <= 128) SSD(16, 8)
  if (n_state <= 256) SSD(16, 16)
  SSD(16, 32)
#undef SSD
#undef SSD_AS
}

// y: fp32 [n_tokens, ldy]; z: `z_dtype` [n_tokens, ldz]; w: fp32 [groups * group]; out: `dtype` [n_tokens, ldo].
extern "C" int leone_grouped_gate_norm(int dtype, const float* y, int ldy, int z_dtype, const void* z, int ldz,
                                       const float* w, void* out, int ldo, int n_tokens, int groups, int group, float eps,
                                       cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  if (groups <= 0 || groups > 65535 || group <= 0 || group > 40000) return kRefusedSize;
  if ((dtype | 1) != 1 || (z_dtype | 1) != 1) return kRefusedDtype;
  const bool vec = group % 4 == 0 && group <= 4096 && ldy % 4 == 0 && ldz % 4 == 0 && ldo % 4 == 0 &&
                   (((uintptr_t)y | (uintptr_t)w) & 15) == 0 && ((uintptr_t)z & 15) == 0 && ((uintptr_t)out & 15) == 0;
  if (vec) {
    int threads = (group / 4 + 31) / 32 * 32;
    if (threads > 256) threads = 256;
    const int rows = (group / 4 + threads - 1) / threads;
#define GV(TZ, T, R)                                                                                                 \
  return launch_kernel(grouped_gate_norm_vec_kernel<TZ, T, R>, dim3(n_tokens, groups), dim3(threads), 0, stream, y,  \
                       ldy, (const TZ*)z, ldz, w, (T*)out, ldo, group, eps)
#define GVR(TZ, T)                \
  {                               \
    if (rows == 1) GV(TZ, T, 1);  \
    if (rows == 2) GV(TZ, T, 2);  \
    GV(TZ, T, 4);                 \
  }
    if (z_dtype == 0 && dtype == 0) GVR(float, float)
    if (z_dtype == 0) GVR(float, __nv_bfloat16)
    if (dtype == 0) GVR(__nv_bfloat16, float)
    GVR(__nv_bfloat16, __nv_bfloat16)
#undef GVR
#undef GV
  }
  const size_t smem = sizeof(float) * (size_t)group;
#define GN(TZ, T)                                                                                                        \
  {                                                                                                                      \
    if (smem > 40 * 1024)                                                                                                \
      cudaFuncSetAttribute(grouped_gate_norm_kernel<TZ, T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);     \
    return launch_kernel(grouped_gate_norm_kernel<TZ, T>, dim3(n_tokens, groups), dim3(256), smem, stream, y, ldy,       \
                         (const TZ*)z, ldz, w, (T*)out, ldo, group, eps);                                                \
  }
  if (z_dtype == 0 && dtype == 0) GN(float, float)
  if (z_dtype == 0) GN(float, __nv_bfloat16)
  if (dtype == 0) GN(__nv_bfloat16, float)
  GN(__nv_bfloat16, __nv_bfloat16)
#undef GN
}
