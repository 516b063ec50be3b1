// Small kernels shared by several parts: two RMS norms of the same rows in one pass, the squared
// ReLU, a product batched over heads, the norm of a sublayer's output added to the residual stream,
// elementwise gates.
#include "common.cuh"
#include "mma_tile.cuh"

namespace leone {

// out_a = x * r * w_a, out_b = x * r * w_b with r = 1/sqrt(mean(x^2) + eps): both norms of a layer
// whose branches read the same residual rows share the row's sum of squares.
template <typename T, typename TW>
__global__ void __launch_bounds__(256)
rms_norm_pair_kernel(const float* __restrict__ x, const TW* __restrict__ w_a, const TW* __restrict__ w_b,
                     T* __restrict__ out_a, T* __restrict__ out_b, int width, float eps) {
  pdl_trigger();      // the next kernel may be scheduled; it waits for this one before it touches data
  pdl_wait();
  __shared__ float scratch[33];
  const size_t base = (size_t)blockIdx.x * width;
  float ss = 0.f;
  for (int c = threadIdx.x; c < width; c += blockDim.x) ss = fmaf(x[base + c], x[base + c], ss);
  ss = block_sum(ss, scratch);
  const float r = 1.f / sqrtf(ss / (float)width + eps);
  for (int c = threadIdx.x; c < width; c += blockDim.x) {
    const float v = x[base + c] * r;
    out_a[base + c] = from_float<T>(v * to_float<TW>(w_a[c]));
    out_b[base + c] = from_float<T>(v * to_float<TW>(w_b[c]));
  }
}

template <typename T>
__global__ void relu_squared_kernel(T* __restrict__ x, long long n) {
  pdl_trigger();      // the next kernel may be scheduled; it waits for this one before it touches data
  pdl_wait();
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
    const float v = fmaxf(to_float<T>(x[i]), 0.f);
    x[i] = from_float<T>(v * v);
  }
}

// C_b[M, N] = A_b[M, K] W_b[N, K]^T for b < batch, fp32 accumulation with k ascending; the three
// operands of batch b start b * (their batch stride) elements after those of batch 0.
constexpr int BM = 64, BN = 64, BK = 16;

template <typename T>
__global__ void __launch_bounds__(256)
gemm_batched_kernel(const T* __restrict__ A, const T* __restrict__ W, T* __restrict__ C, int M, int N, int K,
                    int lda, int ldw, int ldc, long long a_bs, long long w_bs, long long c_bs) {
  pdl_trigger();      // the next kernel may be scheduled; it waits for this one before it touches data
  pdl_wait();
  __shared__ float As[BK][BM + 4];
  __shared__ float Ws[BK][BN + 4];
  A += (size_t)blockIdx.z * a_bs;
  W += (size_t)blockIdx.z * w_bs;
  C += (size_t)blockIdx.z * c_bs;
  const int tid = threadIdx.x;
  const int m0 = blockIdx.y * BM, n0 = blockIdx.x * BN;
  const int ty = tid >> 4, tx = tid & 15;
  const int lr = tid >> 2, lk = (tid & 3) * 4;
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  const T* a_row = A + (size_t)(m0 + lr) * lda;
  const T* w_row = W + (size_t)(n0 + lr) * ldw;
  const bool a_ok = m0 + lr < M, w_ok = n0 + lr < N;
  for (int k0 = 0; k0 < K; k0 += BK) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int k = k0 + lk + i;
      As[lk + i][lr] = (a_ok && k < K) ? to_float<T>(a_row[k]) : 0.f;
      Ws[lk + i][lr] = (w_ok && k < K) ? to_float<T>(w_row[k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < BK; ++k) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) a[i] = As[k][ty * 4 + i];
#pragma unroll
      for (int j = 0; j < 4; ++j) b[j] = Ws[k][tx * 4 + j];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= M) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n < N) C[(size_t)m * ldc + n] = from_float<T>(acc[i][j]);
    }
  }
}

// The same product on tensor cores (bfloat16): a block owns 64 rows x 64 columns of one batch.
__global__ void __launch_bounds__(128)
gemm_batched_mma_kernel(const __nv_bfloat16* __restrict__ A, const __nv_bfloat16* __restrict__ W,
                        __nv_bfloat16* __restrict__ C, int M, int N, int K, int lda, int ldw, int ldc, long long a_bs,
                        long long w_bs, long long c_bs) {
  pdl_trigger();      // the next kernel may be scheduled; it waits for this one before it touches data
  pdl_wait();
  extern __shared__ __align__(16) unsigned char smem_m[];
  __shared__ int a_index[TM];
  A += (size_t)blockIdx.z * a_bs;
  W += (size_t)blockIdx.z * w_bs;
  C += (size_t)blockIdx.z * c_bs;
  const int m0 = blockIdx.y * TM, n0 = blockIdx.x * TN;
  for (int r = threadIdx.x; r < TM; r += 128) a_index[r] = m0 + r < M ? m0 + r : -1;
  __syncthreads();
  float acc[1][2][4][4];
#pragma unroll
  for (int mt = 0; mt < 2; ++mt)
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[0][mt][n][i] = 0.f;
  grouped_mainloop<1>(smem_m, A, a_index, lda, W + (size_t)n0 * ldw, nullptr, min(TN, N - n0), K, acc, ldw);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, tq = lane & 3;
  const int wm = warp >> 1, wn = warp & 1;
#pragma unroll
  for (int mt = 0; mt < 2; ++mt)
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int m = m0 + wm * 32 + mt * 16 + g + 8 * i;
      if (m >= M) continue;
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        const int col = n0 + wn * 32 + n * 8 + 2 * tq;
        if (col >= N) continue;
        *reinterpret_cast<__nv_bfloat162*>(C + (size_t)m * ldc + col) =
            __floats2bfloat162_rn(acc[0][mt][n][2 * i], acc[0][mt][n][2 * i + 1]);
      }
    }
}


// dst[t, :] (+)= coef * (a[t, :] / rms(a[t, :]) * w_a  [+ b[t, :] / rms(b[t, :]) * w_b]), every norm over its own
// row with eps inside the root.  The norm of a sublayer's *output*, added to the residual stream (or
// written, if not `accumulate`); with two sources, the normed outputs of two branches side by side.
// `rounded`: also the new dst row in the run dtype, for the next reader of the stream.  `w_then`: the
// combination is itself RMS-normed with that weight before it is added (a norm on the sum of normed branches).
template <typename TW, typename TR>
__global__ void __launch_bounds__(256)
rms_norm_add_kernel(float* __restrict__ dst, const float* __restrict__ a, const TW* __restrict__ w_a,
                    const float* __restrict__ b, const TW* __restrict__ w_b, int width, float coef, float eps,
                    int accumulate, TR* __restrict__ rounded, const TW* __restrict__ w_then) {
  pdl_trigger();
  pdl_wait();
  __shared__ float scratch[33];
  extern __shared__ float row_s[];      // [width], only with w_then
  const size_t base = (size_t)blockIdx.x * width;
  float sa = 0.f, sb = 0.f;
  for (int c = threadIdx.x; c < width; c += blockDim.x) {
    sa = fmaf(a[base + c], a[base + c], sa);
    if (b != nullptr) sb = fmaf(b[base + c], b[base + c], sb);
  }
  sa = block_sum(sa, scratch);
  const float ra = 1.f / sqrtf(sa / (float)width + eps);
  float rb = 0.f;
  if (b != nullptr) {
    sb = block_sum(sb, scratch);
    rb = 1.f / sqrtf(sb / (float)width + eps);
  }
  float rt = 1.f;
  if (w_then != nullptr) {
    // the combined row is itself normed (with w_then) before it is added: a second pass over the row in shared memory
    float st = 0.f;
    for (int c = threadIdx.x; c < width; c += blockDim.x) {
      float v = a[base + c] * ra * to_float<TW>(w_a[c]);
      if (b != nullptr) v += b[base + c] * rb * to_float<TW>(w_b[c]);
      v *= coef;
      row_s[c] = v;
      st = fmaf(v, v, st);
    }
    st = block_sum(st, scratch);
    rt = 1.f / sqrtf(st / (float)width + eps);
  }
  for (int c = threadIdx.x; c < width; c += blockDim.x) {
    float v;
    if (w_then != nullptr) {
      v = row_s[c] * rt * to_float<TW>(w_then[c]);
    } else {
      v = a[base + c] * ra * to_float<TW>(w_a[c]);
      if (b != nullptr) v += b[base + c] * rb * to_float<TW>(w_b[c]);
      v *= coef;
    }
    if (accumulate) v += dst[base + c];
    dst[base + c] = v;
    if (rounded != nullptr) rounded[base + c] = from_float<TR>(v);
  }
}

// The same for rows that vector accesses fit, with a row in registers (four columns a thread at a time), and one thing
// more: `next_out` = the new dst row RMS-normed with `next_w` (fp32), for the sublayer that reads the stream next, so that a
// norm on a sublayer's output and the norm before the sublayer after it are one pass over the row.
template <typename T> __device__ __forceinline__ float4 row_load4(const T* p);
template <> __device__ __forceinline__ float4 row_load4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <> __device__ __forceinline__ float4 row_load4<__nv_bfloat16>(const __nv_bfloat16* p) {
  const uint2 r = *reinterpret_cast<const uint2*>(p);
  return make_float4(__uint_as_float(r.x << 16), __uint_as_float(r.x & 0xffff0000u), __uint_as_float(r.y << 16),
                     __uint_as_float(r.y & 0xffff0000u));
}
template <typename T> __device__ __forceinline__ void row_store4(T* p, float4 v);
template <> __device__ __forceinline__ void row_store4<float>(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
template <> __device__ __forceinline__ void row_store4<__nv_bfloat16>(__nv_bfloat16* p, float4 v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  uint2 r;
  r.x = *reinterpret_cast<const uint32_t*>(&a);
  r.y = *reinterpret_cast<const uint32_t*>(&b);
  *reinterpret_cast<uint2*>(p) = r;
}
__device__ __forceinline__ float sq4(float4 v, float s) { return fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, s)))); }

template <typename TW, typename TR, int R>
__global__ void __launch_bounds__(256)
rms_norm_add_vec_kernel(float* __restrict__ dst, const float* __restrict__ a, const TW* __restrict__ w_a,
                        const float* __restrict__ b, const TW* __restrict__ w_b, int width, float coef, float eps,
                        int accumulate, TR* __restrict__ rounded, const TW* __restrict__ w_then,
                        const float* __restrict__ next_w, float next_eps, TR* __restrict__ next_out) {
  pdl_trigger();
  pdl_wait();
  __shared__ float scratch[33];
  const size_t base = (size_t)blockIdx.x * width;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 va[R], vb[R], vd[R];
  // short rows: the weights are asked for with the row, so that no load stands between two sums
  constexpr bool kAhead = R <= 2;
  float4 wa_r[kAhead ? R : 1], wn_r[kAhead ? R : 1];
  float sa = 0.f, sb = 0.f;
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 4;
    const bool in = c < width;
    if (kAhead) {
      wa_r[i] = in ? row_load4<TW>(w_a + c) : zero;
      wn_r[i] = in && next_out != nullptr ? row_load4<float>(next_w + c) : zero;
    }
    va[i] = in ? row_load4<float>(a + base + c) : zero;
    vb[i] = in && b != nullptr ? row_load4<float>(b + base + c) : zero;
    vd[i] = in && accumulate ? row_load4<float>(dst + base + c) : zero;
    sa = sq4(va[i], sa);
    sb = sq4(vb[i], sb);
  }
  sa = block_sum(sa, scratch);
  const float ra = coef / sqrtf(sa / (float)width + eps);
  float rb = 0.f;
  if (b != nullptr) {
    sb = block_sum(sb, scratch);
    rb = coef / sqrtf(sb / (float)width + eps);
  }
  float st = 0.f;
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 4;
    if (c < width) {
      const float4 wa = kAhead ? wa_r[kAhead ? i : 0] : row_load4<TW>(w_a + c);
      float4 v = make_float4(va[i].x * ra * wa.x, va[i].y * ra * wa.y, va[i].z * ra * wa.z, va[i].w * ra * wa.w);
      if (b != nullptr) {
        const float4 wb = row_load4<TW>(w_b + c);
        v.x = fmaf(vb[i].x * rb, wb.x, v.x);
        v.y = fmaf(vb[i].y * rb, wb.y, v.y);
        v.z = fmaf(vb[i].z * rb, wb.z, v.z);
        v.w = fmaf(vb[i].w * rb, wb.w, v.w);
      }
      va[i] = v;
      st = sq4(v, st);
    }
  }
  float rt = 1.f;
  if (w_then != nullptr) {
    st = block_sum(st, scratch);
    rt = 1.f / sqrtf(st / (float)width + eps);
  }
  float sn = 0.f;
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 4;
    if (c < width) {
      float4 v = va[i];
      if (w_then != nullptr) {
        const float4 wt = row_load4<TW>(w_then + c);
        v = make_float4(v.x * rt * wt.x, v.y * rt * wt.y, v.z * rt * wt.z, v.w * rt * wt.w);
      }
      v = make_float4(v.x + vd[i].x, v.y + vd[i].y, v.z + vd[i].z, v.w + vd[i].w);
      row_store4<float>(dst + base + c, v);
      if (rounded != nullptr) row_store4<TR>(rounded + base + c, v);
      va[i] = v;
      sn = sq4(v, sn);
    }
  }
  if (next_out != nullptr) {
    sn = block_sum(sn, scratch);
    const float rn = 1.f / sqrtf(sn / (float)width + next_eps);
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const int c = (threadIdx.x + i * blockDim.x) * 4;
      if (c < width) {
        const float4 wn = kAhead ? wn_r[kAhead ? i : 0] : row_load4<float>(next_w + c);
        row_store4<TR>(next_out + base + c, make_float4(va[i].x * rn * wn.x, va[i].y * rn * wn.y, va[i].z * rn * wn.z, va[i].w * rn * wn.w));
      }
    }
  }
}

// a[t, c] *= act(gate[t, c]): act 0 sigmoid, 1 silu.
template <typename T>
__global__ void __launch_bounds__(256)
gate_rows_kernel(T* __restrict__ a, int lda, const T* __restrict__ gate, int ldg, int n_rows, int cols, int act) {
  pdl_trigger();
  pdl_wait();
  const long long total = (long long)n_rows * cols;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long t = i / cols;
    const int c = (int)(i - t * cols);
    const float z = to_float<T>(gate[t * ldg + c]);
    const float sg = 1.f / (1.f + expf(-z));
    a[t * lda + c] = from_float<T>(to_float<T>(a[t * lda + c]) * (act == 1 ? z * sg : sg));
  }
}

// The same with eight bfloat16 columns a thread (rows, columns and bases that 16-byte accesses fit).
__global__ void __launch_bounds__(256)
gate_rows_vec_kernel(__nv_bfloat16* __restrict__ a, int lda, const __nv_bfloat16* __restrict__ gate, int ldg, int n_rows,
                     int cols8, int act) {
  pdl_trigger();
  pdl_wait();
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= cols8) return;
  for (int t = blockIdx.y; t < n_rows; t += gridDim.y) {
    uint4* at = reinterpret_cast<uint4*>(a + (size_t)t * lda) + c;
    const uint4 zr = *(reinterpret_cast<const uint4*>(gate + (size_t)t * ldg) + c);
    uint4 ar = *at;
    const __nv_bfloat162* z2 = reinterpret_cast<const __nv_bfloat162*>(&zr);
    __nv_bfloat162* a2 = reinterpret_cast<__nv_bfloat162*>(&ar);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 z = __bfloat1622float2(z2[i]), x = __bfloat1622float2(a2[i]);
      const float s0 = 1.f / (1.f + expf(-z.x)), s1 = 1.f / (1.f + expf(-z.y));
      a2[i] = __floats2bfloat162_rn(x.x * (act == 1 ? z.x * s0 : s0), x.y * (act == 1 ? z.y * s1 : s1));
    }
    *at = ar;
  }
}

// out[t, c] = gelu_tanh(z[t, c]) * rows[t, off + c]: a projection's fp32 result gates a slice of a
// per-token row.  gelu_tanh(z) = z/2 (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3))).
template <typename T>
__global__ void __launch_bounds__(256)
gelu_gate_kernel(const float* __restrict__ z, int ldz, const float* __restrict__ rows, int ldr, int off,
                 T* __restrict__ out, int ldo, int n_rows, int cols) {
  pdl_trigger();
  pdl_wait();
  const long long total = (long long)n_rows * cols;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long t = i / cols;
    const int c = (int)(i - t * cols);
    const float v = z[t * ldz + c];
    const float g = 0.5f * v * (1.f + tanhf(0.7978845608028654f * (v + 0.044715f * v * v * v)));
    out[t * ldo + c] = from_float<T>(g * rows[t * ldr + off + c]);
  }
}

}  // namespace leone

using namespace leone;

extern "C" void leone_mixers_set_pdl(int enabled) { pdl_flag() = enabled ? 1 : 0; }

extern "C" int leone_rms_norm_pair(const float* x, const void* w_a, const void* w_b, int w_dtype, void* out_a,
                                   void* out_b, int out_dtype, int n, int width, float eps, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (width <= 0) return kRefusedSize;
#define NP(T, TW)                                                                                            \
  launch_kernel(rms_norm_pair_kernel<T, TW>, dim3(n), dim3(256), 0, stream, x, (const TW*)w_a, (const TW*)w_b, (T*)out_a, (T*)out_b, \
                                                     width, eps)
  if (out_dtype == 0 && w_dtype == 0) NP(float, float);
  else if (out_dtype == 1 && w_dtype == 0) NP(__nv_bfloat16, float);
  else if (out_dtype == 1 && w_dtype == 1) NP(__nv_bfloat16, __nv_bfloat16);
  else if (out_dtype == 0 && w_dtype == 1) NP(float, __nv_bfloat16);
  else return kRefusedDtype;
#undef NP
  return launch_result();
}

extern "C" int leone_relu_squared(int dtype, void* x, long long n, cudaStream_t stream) {
  if (n <= 0) return 0;
  const long long want = (n + 255) / 256;
  const unsigned blocks = (unsigned)(want < 148 * 16 ? want : 148 * 16);
  if (dtype == 0) launch_kernel(relu_squared_kernel<float>, dim3(blocks), dim3(256), 0, stream, (float*)x, n);
  else if (dtype == 1) launch_kernel(relu_squared_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, stream, (__nv_bfloat16*)x, n);
  else return kRefusedDtype;
  return launch_result();
}

extern "C" int leone_gemm_batched(int dtype, const void* a, const void* w, void* c, int m, int n, int k, int lda,
                                  int ldw, int ldc, long long a_bs, long long w_bs, long long c_bs, int batch,
                                  cudaStream_t stream) {
  if (m <= 0 || n <= 0 || batch <= 0) return 0;
  if (k <= 0 || lda < k || ldw < k || ldc < n || batch > 65535) return kRefusedSize;
  const dim3 grid((n + BN - 1) / BN, (m + BM - 1) / BM, batch);
  if (grid.y > 65535) return kRefusedSize;
  // bfloat16 with 16-byte aligned rows: tensor cores
  if (dtype == 1 && k % 8 == 0 && n % 2 == 0 && lda % 8 == 0 && ldw % 8 == 0 && ldc % 2 == 0 && a_bs % 8 == 0 &&
      w_bs % 8 == 0 && c_bs % 2 == 0 && ((uintptr_t)a % 16) == 0 && ((uintptr_t)w % 16) == 0 && ((uintptr_t)c % 4) == 0) {
    const dim3 tgrid((n + TN - 1) / TN, (m + TM - 1) / TM, batch);
    if (tgrid.y > 65535) return kRefusedSize;
    const size_t smem = (size_t)TSTAGES * (TM + TN) * TPITCH;
    static bool configured = false;
    if (!configured) {
      cudaFuncSetAttribute(gemm_batched_mma_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      configured = true;
    }
    launch_kernel(gemm_batched_mma_kernel, tgrid, dim3(128), smem, stream, (const __nv_bfloat16*)a, (const __nv_bfloat16*)w,
                                                          (__nv_bfloat16*)c, m, n, k, lda, ldw, ldc, a_bs, w_bs, c_bs);
    return launch_result();
  }
  if (dtype == 0)
    launch_kernel(gemm_batched_kernel<float>, grid, dim3(256), 0, stream, (const float*)a, (const float*)w, (float*)c, m, n, k, lda,
                                                         ldw, ldc, a_bs, w_bs, c_bs);
  else if (dtype == 1)
    launch_kernel(gemm_batched_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, (const __nv_bfloat16*)a, (const __nv_bfloat16*)w,
                                                                 (__nv_bfloat16*)c, m, n, k, lda, ldw, ldc, a_bs,
                                                                 w_bs, c_bs);
  else
    return kRefusedDtype;
  return launch_result();
}

// dst: fp32 [n, width]; a, b: fp32 [n, width] (b and w_b may be null); w in `w_dtype`; rounded: [n, width] in
// `rounded_dtype`, or null; w_then: [width] in `w_dtype`, or null (width at most 12,000 with it).
extern "C" int leone_rms_norm_add(float* dst, const float* a, const void* w_a, const float* b, const void* w_b,
                                  int w_dtype, int n, int width, float coef, float eps, int accumulate, void* rounded,
                                  int rounded_dtype, const void* w_then, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (width <= 0 || (b != nullptr) != (w_b != nullptr) || (w_then != nullptr && width > 12000)) return kRefusedSize;
  const size_t smem = w_then != nullptr ? sizeof(float) * (size_t)width : 0;
#define NA(TW, TR)                                                                                                    \
  return launch_kernel(rms_norm_add_kernel<TW, TR>, dim3(n), dim3(256), smem, stream, dst, a, (const TW*)w_a, b,      \
                       (const TW*)w_b, width, coef, eps, accumulate, (TR*)rounded, (const TW*)w_then)
  if (w_dtype == 0 && rounded_dtype == 0) NA(float, float);
  if (w_dtype == 0 && rounded_dtype == 1) NA(float, __nv_bfloat16);
  if (w_dtype == 1 && rounded_dtype == 0) NA(__nv_bfloat16, float);
  if (w_dtype == 1 && rounded_dtype == 1) NA(__nv_bfloat16, __nv_bfloat16);
#undef NA
  return kRefusedDtype;
}

// The same and, with next_out (in `rounded_dtype`, as `rounded` is) and next_w (fp32), the new dst rows RMS-normed for
// their next reader; width a multiple of 4 up to 8,192, all rows 16-byte aligned.
extern "C" int leone_rms_norm_add_next(float* dst, const float* a, const void* w_a, const float* b, const void* w_b,
                                       int w_dtype, int n, int width, float coef, float eps, int accumulate, void* rounded,
                                       int rounded_dtype, const void* w_then, const float* next_w, float next_eps,
                                       void* next_out, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (width <= 0 || width % 4 != 0 || width > 8192 || (b != nullptr) != (w_b != nullptr) || (next_out != nullptr) != (next_w != nullptr))
    return kRefusedSize;
  if (((uintptr_t)dst | (uintptr_t)a | (uintptr_t)b | (uintptr_t)w_a | (uintptr_t)w_b | (uintptr_t)rounded |
       (uintptr_t)w_then | (uintptr_t)next_w | (uintptr_t)next_out) & 15)
    return kRefusedAlignment;
  const int quads = width / 4;
  const int threads = quads >= 256 ? 256 : (quads + 31) / 32 * 32, rows = (quads + threads - 1) / threads;
#define NV(TW, TR, R)                                                                                                  \
  return launch_kernel(rms_norm_add_vec_kernel<TW, TR, R>, dim3(n), dim3(threads), 0, stream, dst, a, (const TW*)w_a, b, \
                       (const TW*)w_b, width, coef, eps, accumulate, (TR*)rounded, (const TW*)w_then, next_w, next_eps,  \
                       (TR*)next_out)
#define NVR(TW, TR)                 \
  {                                 \
    if (rows == 1) NV(TW, TR, 1);   \
    if (rows == 2) NV(TW, TR, 2);   \
    if (rows <= 4) NV(TW, TR, 4);   \
    NV(TW, TR, 8);                  \
  }
  if (w_dtype == 0 && rounded_dtype == 0) NVR(float, float)
  if (w_dtype == 0 && rounded_dtype == 1) NVR(float, __nv_bfloat16)
  if (w_dtype == 1 && rounded_dtype == 0) NVR(__nv_bfloat16, float)
  if (w_dtype == 1 && rounded_dtype == 1) NVR(__nv_bfloat16, __nv_bfloat16)
#undef NVR
#undef NV
  return kRefusedDtype;
}

extern "C" int leone_gate_rows(int dtype, void* a, int lda, const void* gate, int ldg, int n_rows, int cols, int act,
                               cudaStream_t stream) {
  if (n_rows <= 0 || cols <= 0) return 0;
  const long long want = ((long long)n_rows * cols + 255) / 256;
  const unsigned blocks = (unsigned)(want < 148 * 16 ? want : 148 * 16);
  if (dtype == 1 && cols % 8 == 0 && lda % 8 == 0 && ldg % 8 == 0 && (((uintptr_t)a | (uintptr_t)gate) & 15) == 0) {
    const int c8 = cols / 8, threads = c8 >= 256 ? 256 : (c8 + 31) / 32 * 32;
    return launch_kernel(gate_rows_vec_kernel, dim3((c8 + threads - 1) / threads, n_rows < 65535 ? n_rows : 65535), dim3(threads),
                         0, stream, (__nv_bfloat16*)a, lda, (const __nv_bfloat16*)gate, ldg, n_rows, c8, act);
  }
  if (dtype == 0)
    return launch_kernel(gate_rows_kernel<float>, dim3(blocks), dim3(256), 0, stream, (float*)a, lda, (const float*)gate,
                         ldg, n_rows, cols, act);
  if (dtype == 1)
    return launch_kernel(gate_rows_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, stream, (__nv_bfloat16*)a, lda,
                         (const __nv_bfloat16*)gate, ldg, n_rows, cols, act);
  return kRefusedDtype;
}

extern "C" int leone_gelu_gate(int dtype, const float* z, int ldz, const float* rows, int ldr, int off, void* out, int ldo,
                               int n_rows, int cols, cudaStream_t stream) {
  if (n_rows <= 0 || cols <= 0) return 0;
  const long long want = ((long long)n_rows * cols + 255) / 256;
  const unsigned blocks = (unsigned)(want < 148 * 16 ? want : 148 * 16);
  if (dtype == 0)
    return launch_kernel(gelu_gate_kernel<float>, dim3(blocks), dim3(256), 0, stream, z, ldz, rows, ldr, off, (float*)out,
                         ldo, n_rows, cols);
  if (dtype == 1)
    return launch_kernel(gelu_gate_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, stream, z, ldz, rows, ldr, off,
                         (__nv_bfloat16*)out, ldo, n_rows, cols);
  return kRefusedDtype;
}

extern "C" int leone_zero(void* p, long long bytes, cudaStream_t stream) {
  if (bytes <= 0) return 0;
  return (int)cudaMemsetAsync(p, 0, (size_t)bytes, stream);
}
