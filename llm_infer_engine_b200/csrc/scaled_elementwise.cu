// Row kernels of blocks that scale a branch's output on its way into the residual stream, and of a feed-forward whose
// activation is a sum of normalised powers:
//
//   scaled_add_rmsnorm   h += s (.) (c1 d1 + c2 d2) + b;  y = h / sqrt(mean(h^2) + eps) * w
//                        s a vector over the width (a learned scale per channel, or none), c1 and c2 constants, d1 and
//                        d2 branch outputs (the second optional: two mixers side by side), b a vector over the width (a
//                        branch's output bias, or none); either half may be left out: no w and y = only the add, no d1
//                        = only the norm, y without w = a copy of the new stream in y's type
//   sandwich_add_norm    b = c1 e1 + c2 e2, e = d or N(d) w_d;  h += N(b) w_out;  y = N(h) w      (N = division by the
//                        root mean square): a branch with a norm behind it closes and the next one, with a norm in front
//                        of it, opens, in one pass over the rows; each of the norms may be left out but the one behind
//   poly_norm            y = a N(z) + b N(z^2) + c N(z^3) + e, N(t) = t / sqrt(mean(t^2) + eps) over the row, powers
//                        element by element; a, b, c, e learned numbers in device memory
//
// The stream h and all arithmetic are float32 in both precisions; d1, d2, z and y have the activation type or float32.
// A block per row; the row is staged in shared memory between the sum of squares and the store.
#include "common.cuh"

namespace llmie {

__device__ __forceinline__ float load_any(const void* p, int dtype, size_t i) {
  return dtype == LLMIE_F32 ? reinterpret_cast<const float*>(p)[i] : to_f32(reinterpret_cast<const __nv_bfloat16*>(p)[i]);
}

__device__ __forceinline__ float4 load4_any(const void* p, int dtype, size_t i) {
  if (dtype == LLMIE_F32) return *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(p) + i);
  const uint2 raw = *reinterpret_cast<const uint2*>(reinterpret_cast<const __nv_bfloat16*>(p) + i);
  const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  return make_float4(lo.x, lo.y, hi.x, hi.y);
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  uint2 raw;
  raw.x = *reinterpret_cast<const uint32_t*>(&lo);
  raw.y = *reinterpret_cast<const uint32_t*>(&hi);
  *reinterpret_cast<uint2*>(p) = raw;
}

// The same kernel four channels a thread (d a multiple of 4, every row 16-byte aligned): the element's arithmetic is
// the scalar kernel's, only who sums which squares differs.
template <typename TY>
__global__ void scaled_add_rmsnorm4_kernel(float* __restrict__ h, const void* __restrict__ d1, int d1_dtype, float c1,
                                           const void* __restrict__ d2, int d2_dtype, float c2,
                                           const float* __restrict__ s, const float* __restrict__ bias,
                                           const float* __restrict__ w, float eps, TY* __restrict__ y, int y_ld,
                                           const int* __restrict__ rows, int d) {
  extern __shared__ float row_smem[];
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const size_t r_out = blockIdx.x;
  const size_t src = (rows ? (size_t)rows[r_out] : r_out) * d;
  float ss = 0.f;
  for (int c = threadIdx.x * 4; c < d; c += blockDim.x * 4) {
    float4 x = *reinterpret_cast<const float4*>(h + src + c);
    if (d1) {
      const float4 a = load4_any(d1, d1_dtype, src + c);
      float4 b = make_float4(c1 * a.x, c1 * a.y, c1 * a.z, c1 * a.w);
      if (d2) {
        const float4 e = load4_any(d2, d2_dtype, src + c);
        b = make_float4(fmaf(c2, e.x, b.x), fmaf(c2, e.y, b.y), fmaf(c2, e.z, b.z), fmaf(c2, e.w, b.w));
      }
      if (s) {
        const float4 sv = *reinterpret_cast<const float4*>(s + c);
        x = make_float4(fmaf(sv.x, b.x, x.x), fmaf(sv.y, b.y, x.y), fmaf(sv.z, b.z, x.z), fmaf(sv.w, b.w, x.w));
      } else {
        x = make_float4(x.x + b.x, x.y + b.y, x.z + b.z, x.w + b.w);
      }
      if (bias) {
        const float4 bv = *reinterpret_cast<const float4*>(bias + c);
        x = make_float4(x.x + bv.x, x.y + bv.y, x.z + bv.z, x.w + bv.w);
      }
      if (!rows) *reinterpret_cast<float4*>(h + src + c) = x;
    }
    if (y && !w) {
      store4(y + r_out * y_ld + c, x);
      continue;
    }
    *reinterpret_cast<float4*>(row_smem + c) = x;
    ss = fmaf(x.x, x.x, ss);
    ss = fmaf(x.y, x.y, ss);
    ss = fmaf(x.z, x.z, ss);
    ss = fmaf(x.w, x.w, ss);
  }
  if (!y || !w) return;
  ss = block_sum(ss, red);
  const float rstd = 1.f / sqrtf(ss / (float)d + eps);
  for (int c = threadIdx.x * 4; c < d; c += blockDim.x * 4) {
    const float4 x = *reinterpret_cast<const float4*>(row_smem + c);
    const float4 wv = *reinterpret_cast<const float4*>(w + c);
    store4(y + r_out * y_ld + c, make_float4(x.x * rstd * wv.x, x.y * rstd * wv.y, x.z * rstd * wv.z, x.w * rstd * wv.w));
  }
}

template <typename TY>
__global__ void scaled_add_rmsnorm_kernel(float* __restrict__ h, const void* __restrict__ d1, int d1_dtype, float c1,
                                          const void* __restrict__ d2, int d2_dtype, float c2,
                                          const float* __restrict__ s, const float* __restrict__ bias,
                                          const float* __restrict__ w, float eps, TY* __restrict__ y, int y_ld,
                                          const int* __restrict__ rows, int d) {
  extern __shared__ float row_smem[];
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const size_t r_out = blockIdx.x;
  const size_t src = (rows ? (size_t)rows[r_out] : r_out) * d;
  float ss = 0.f;
  for (int c = threadIdx.x; c < d; c += blockDim.x) {
    float x = h[src + c];
    if (d1) {
      float b = c1 * load_any(d1, d1_dtype, src + c);
      if (d2) b = fmaf(c2, load_any(d2, d2_dtype, src + c), b);
      x = s ? fmaf(s[c], b, x) : x + b;
      if (bias) x += bias[c];
      if (!rows) h[src + c] = x;
    }
    if (y && !w) {
      y[r_out * y_ld + c] = from_f32<TY>(x);
      continue;
    }
    row_smem[c] = x;
    ss = fmaf(x, x, ss);
  }
  if (!y || !w) return;
  ss = block_sum(ss, red);
  const float rstd = 1.f / sqrtf(ss / (float)d + eps);
  for (int c = threadIdx.x; c < d; c += blockDim.x) y[r_out * y_ld + c] = from_f32<TY>(row_smem[c] * rstd * w[c]);
}

// A branch that has a norm behind it closes and the next branch's norm opens it (see the list at the top). A thread owns
// NR runs of four channels and keeps them in registers from the branch outputs to the last store; weights are asked for
// before the wait on the kernel that makes the branch outputs. d a multiple of 4 with d / 4 <= NR * blockDim.x.
template <typename TY, int NR>
__global__ void sandwich_add_norm4_kernel(float* __restrict__ h, const void* __restrict__ d1, int d1_dtype, float c1,
                                          const float* __restrict__ w1, const void* __restrict__ d2, int d2_dtype,
                                          float c2, const float* __restrict__ w2, float eps_in,
                                          const float* __restrict__ w_out, float eps_out, const float* __restrict__ w,
                                          float eps, TY* __restrict__ y, int y_ld, const int* __restrict__ rows, int d) {
  __shared__ float red[32];
  pdl_launch_dependents();
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 wo[NR], wn[NR];
#pragma unroll
  for (int r = 0; r < NR; ++r) {
    const int c = (threadIdx.x + r * blockDim.x) * 4;
    wo[r] = c < d ? *reinterpret_cast<const float4*>(w_out + c) : zero;
    wn[r] = y && w && c < d ? *reinterpret_cast<const float4*>(w + c) : zero;
  }
  pdl_wait();
  const size_t r_out = blockIdx.x;
  const size_t src = (rows ? (size_t)rows[r_out] : r_out) * d;
  float4 b[NR], e[NR], x[NR];
#pragma unroll
  for (int r = 0; r < NR; ++r) {
    const int c = (threadIdx.x + r * blockDim.x) * 4;
    const bool ok = c < d;
    b[r] = ok ? load4_any(d1, d1_dtype, src + c) : zero;
    e[r] = ok && d2 ? load4_any(d2, d2_dtype, src + c) : zero;
    x[r] = ok ? *reinterpret_cast<const float4*>(h + src + c) : zero;
  }
  float k1 = c1, k2 = c2;
  auto squares = [](const float4& v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; };
  if (w1) {
    float ss = 0.f;
#pragma unroll
    for (int r = 0; r < NR; ++r) ss += squares(b[r]);
    k1 = c1 / sqrtf(block_sum(ss, red) / (float)d + eps_in);
  }
  if (w2 && d2) {
    float ss = 0.f;
#pragma unroll
    for (int r = 0; r < NR; ++r) ss += squares(e[r]);
    k2 = c2 / sqrtf(block_sum(ss, red) / (float)d + eps_in);
  }
  float ss = 0.f;
#pragma unroll
  for (int r = 0; r < NR; ++r) {
    const int c = (threadIdx.x + r * blockDim.x) * 4;
    float4 u = make_float4(k1 * b[r].x, k1 * b[r].y, k1 * b[r].z, k1 * b[r].w);
    if (w1 && c < d) {
      const float4 v = *reinterpret_cast<const float4*>(w1 + c);
      u = make_float4(u.x * v.x, u.y * v.y, u.z * v.z, u.w * v.w);
    }
    if (d2) {
      float4 t = make_float4(k2 * e[r].x, k2 * e[r].y, k2 * e[r].z, k2 * e[r].w);
      if (w2 && c < d) {
        const float4 v = *reinterpret_cast<const float4*>(w2 + c);
        t = make_float4(t.x * v.x, t.y * v.y, t.z * v.z, t.w * v.w);
      }
      u = make_float4(u.x + t.x, u.y + t.y, u.z + t.z, u.w + t.w);
    }
    b[r] = u;
    ss += squares(u);
  }
  const float rb = 1.f / sqrtf(block_sum(ss, red) / (float)d + eps_out);
  ss = 0.f;
#pragma unroll
  for (int r = 0; r < NR; ++r) {
    const int c = (threadIdx.x + r * blockDim.x) * 4;
    x[r] = make_float4(fmaf(b[r].x * rb, wo[r].x, x[r].x), fmaf(b[r].y * rb, wo[r].y, x[r].y),
                       fmaf(b[r].z * rb, wo[r].z, x[r].z), fmaf(b[r].w * rb, wo[r].w, x[r].w));
    if (c < d) {
      if (!rows) *reinterpret_cast<float4*>(h + src + c) = x[r];
      if (y && !w) store4(y + r_out * y_ld + c, x[r]);
    }
    ss += squares(x[r]);
  }
  if (!y || !w) return;
  const float rn = 1.f / sqrtf(block_sum(ss, red) / (float)d + eps);
#pragma unroll
  for (int r = 0; r < NR; ++r) {
    const int c = (threadIdx.x + r * blockDim.x) * 4;
    if (c < d)
      store4(y + r_out * y_ld + c, make_float4(x[r].x * rn * wn[r].x, x[r].y * rn * wn[r].y, x[r].z * rn * wn[r].z,
                                               x[r].w * rn * wn[r].w));
  }
}

// The same for every width that fits shared memory, element by element.
template <typename TY>
__global__ void sandwich_add_norm_kernel(float* __restrict__ h, const void* __restrict__ d1, int d1_dtype, float c1,
                                         const float* __restrict__ w1, const void* __restrict__ d2, int d2_dtype,
                                         float c2, const float* __restrict__ w2, float eps_in,
                                         const float* __restrict__ w_out, float eps_out, const float* __restrict__ w,
                                         float eps, TY* __restrict__ y, int y_ld, const int* __restrict__ rows, int d) {
  extern __shared__ float row_smem[];
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const size_t r_out = blockIdx.x;
  const size_t src = (rows ? (size_t)rows[r_out] : r_out) * d;
  float k1 = c1, k2 = c2;
  if (w1) {
    float ss = 0.f;
    for (int c = threadIdx.x; c < d; c += blockDim.x) { const float v = load_any(d1, d1_dtype, src + c); ss = fmaf(v, v, ss); }
    k1 = c1 / sqrtf(block_sum(ss, red) / (float)d + eps_in);
  }
  if (w2 && d2) {
    float ss = 0.f;
    for (int c = threadIdx.x; c < d; c += blockDim.x) { const float v = load_any(d2, d2_dtype, src + c); ss = fmaf(v, v, ss); }
    k2 = c2 / sqrtf(block_sum(ss, red) / (float)d + eps_in);
  }
  float ss = 0.f;
  for (int c = threadIdx.x; c < d; c += blockDim.x) {
    float b = k1 * load_any(d1, d1_dtype, src + c);
    if (w1) b *= w1[c];
    if (d2) {
      float t = k2 * load_any(d2, d2_dtype, src + c);
      if (w2) t *= w2[c];
      b += t;
    }
    row_smem[c] = b;
    ss = fmaf(b, b, ss);
  }
  const float rb = 1.f / sqrtf(block_sum(ss, red) / (float)d + eps_out);
  ss = 0.f;
  for (int c = threadIdx.x; c < d; c += blockDim.x) {
    const float x = fmaf(row_smem[c] * rb, w_out[c], h[src + c]);
    if (!rows) h[src + c] = x;
    if (y && !w) y[r_out * y_ld + c] = from_f32<TY>(x);
    row_smem[c] = x;
    ss = fmaf(x, x, ss);
  }
  if (!y || !w) return;
  const float rn = 1.f / sqrtf(block_sum(ss, red) / (float)d + eps);
  for (int c = threadIdx.x; c < d; c += blockDim.x) y[r_out * y_ld + c] = from_f32<TY>(row_smem[c] * rn * w[c]);
}

template <typename T>
__global__ void poly_norm_kernel(const T* __restrict__ z, const float* __restrict__ coef, float eps, T* __restrict__ y,
                                 int n) {
  extern __shared__ float row_smem[];
  __shared__ float red[32];
  pdl_launch_dependents();
  const float a = coef[0], b = coef[1], c3 = coef[2], e = coef[3];      // weights: no kernel writes them
  pdl_wait();
  const size_t base = (size_t)blockIdx.x * n;
  float s2 = 0.f, s4 = 0.f, s6 = 0.f;
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    const float x = to_f32(z[base + i]);
    const float x2 = x * x, x3 = x2 * x;
    row_smem[i] = x;
    s2 += x2;
    s4 = fmaf(x2, x2, s4);
    s6 = fmaf(x3, x3, s6);
  }
  s2 = block_sum(s2, red);
  s4 = block_sum(s4, red);
  s6 = block_sum(s6, red);
  const float r1 = a / sqrtf(s2 / (float)n + eps), r2 = b / sqrtf(s4 / (float)n + eps),
              r3 = c3 / sqrtf(s6 / (float)n + eps);
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    const float x = row_smem[i];
    const float x2 = x * x;
    y[base + i] = from_f32<T>(fmaf(r1, x, fmaf(r2, x2, fmaf(r3, x2 * x, e))));
  }
}

// Eight values a thread (n a multiple of 8, rows 16-byte aligned); the element's arithmetic is the scalar kernel's.
template <typename T>
__global__ void poly_norm8_kernel(const T* __restrict__ z, const float* __restrict__ coef, float eps, T* __restrict__ y,
                                  int n) {
  extern __shared__ float row_smem[];
  __shared__ float red[32];
  pdl_launch_dependents();
  const float a = coef[0], b = coef[1], c3 = coef[2], e = coef[3];
  pdl_wait();
  const size_t base = (size_t)blockIdx.x * n;
  float s2 = 0.f, s4 = 0.f, s6 = 0.f;
  for (int i = threadIdx.x * 8; i < n; i += blockDim.x * 8) {
    float x[8];
    load8(z + base + i, x);
    store8(row_smem + i, x);
#pragma unroll
    for (int k = 0; k < 8; ++k) {
      const float x2 = x[k] * x[k], x3 = x2 * x[k];
      s2 += x2;
      s4 = fmaf(x2, x2, s4);
      s6 = fmaf(x3, x3, s6);
    }
  }
  s2 = block_sum(s2, red);
  s4 = block_sum(s4, red);
  s6 = block_sum(s6, red);
  const float r1 = a / sqrtf(s2 / (float)n + eps), r2 = b / sqrtf(s4 / (float)n + eps),
              r3 = c3 / sqrtf(s6 / (float)n + eps);
  for (int i = threadIdx.x * 8; i < n; i += blockDim.x * 8) {
    float xs[8], v[8];
    load8(row_smem + i, xs);
#pragma unroll
    for (int k = 0; k < 8; ++k) {
      const float x = xs[k];
      const float x2 = x * x;
      v[k] = fmaf(r1, x, fmaf(r2, x2, fmaf(r3, x2 * x, e)));
    }
    store8(y + base + i, v);
  }
}

static inline int row_block(int d) {
  int t = ((d / 4 + 31) / 32) * 32;
  return t < 64 ? 64 : (t > 512 ? 512 : t);
}

}  // namespace llmie

using namespace llmie;

// h float32 [T, d]; d1, d2 (d2 only with d1) [T, d] of their own dtypes, or null; s, bias float32 [d] or null (bias only
// with d1); y rows of d elements of y_dtype, y_ld apart, or null (the add alone); w float32 [d] or null (with y: the new
// stream itself is stored); rows int32 [n_out] or null (then n_out == T and h is updated in place). A row must fit shared
// memory (d <= 12,288).
extern "C" int llmie_scaled_add_rmsnorm(float* h, const void* d1, int d1_dtype, float c1, const void* d2, int d2_dtype,
                                        float c2, const float* s, const float* bias, const float* w, float eps, void* y,
                                        int y_ld, int y_dtype, const int* rows, int n_out, int d, cudaStream_t stream) {
  if (n_out < 0 || d <= 0 || !h || (d2 && !d1) || (bias && !d1) || (w && !y) || (!y && (rows || !d1)) || (y && y_ld < d))
    return LLMIE_ERR_BAD_ARG;
  if ((y && y_dtype != LLMIE_F32 && y_dtype != LLMIE_BF16) || (d1 && d1_dtype != LLMIE_F32 && d1_dtype != LLMIE_BF16) ||
      (d2 && d2_dtype != LLMIE_F32 && d2_dtype != LLMIE_BF16))
    return LLMIE_ERR_DTYPE;
  if ((size_t)d * sizeof(float) > 48 * 1024) return LLMIE_ERR_UNSUPPORTED_SIZE;
  if (n_out == 0) return LLMIE_OK;
  const dim3 grid(n_out), block(row_block(d));
  const size_t smem = (size_t)d * sizeof(float);
  const bool by4 = d % 4 == 0 && aligned16(h) && (!s || aligned16(s)) && (!w || aligned16(w)) && (!bias || aligned16(bias)) &&
                   (!d1 || aligned16(d1)) && (!d2 || aligned16(d2)) && (!y || (aligned16(y) && y_ld % 4 == 0));
  if (by4) {
    if (y && y_dtype == LLMIE_BF16)
      launch_k(scaled_add_rmsnorm4_kernel<__nv_bfloat16>, grid, block, smem, stream, h, d1, d1_dtype, c1, d2, d2_dtype,
               c2, s, bias, w, eps, (__nv_bfloat16*)y, y_ld, rows, d);
    else
      launch_k(scaled_add_rmsnorm4_kernel<float>, grid, block, smem, stream, h, d1, d1_dtype, c1, d2, d2_dtype, c2, s,
               bias, w, eps, (float*)y, y_ld, rows, d);
    LLMIE_LAUNCH_CHECK();
    return LLMIE_OK;
  }
  if (y && y_dtype == LLMIE_BF16)
    launch_k(scaled_add_rmsnorm_kernel<__nv_bfloat16>, grid, block, smem, stream, h, d1, d1_dtype, c1, d2, d2_dtype, c2, s,
             bias, w, eps, (__nv_bfloat16*)y, y_ld, rows, d);
  else
    launch_k(scaled_add_rmsnorm_kernel<float>, grid, block, smem, stream, h, d1, d1_dtype, c1, d2, d2_dtype, c2, s, bias, w,
             eps, (float*)y, y_ld, rows, d);
  LLMIE_LAUNCH_CHECK();
  return LLMIE_OK;
}

// z, y [T, n] of `dtype`; coef float32 [4] = (a, b, c, e) on the device. n <= 51,200 (a row in shared memory).
extern "C" int llmie_poly_norm(const void* z, const float* coef, float eps, void* y, int n_tokens, int n, int dtype,
                               cudaStream_t stream) {
  if (n_tokens < 0 || n <= 0 || !coef) return LLMIE_ERR_BAD_ARG;
  if ((size_t)n * sizeof(float) > 200 * 1024) return LLMIE_ERR_UNSUPPORTED_SIZE;
  if (n_tokens == 0) return LLMIE_OK;
  const dim3 grid(n_tokens), block(row_block(n));
  const size_t smem = (size_t)n * sizeof(float);
  if (smem > 48 * 1024) {
    cudaFuncSetAttribute(poly_norm_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    cudaFuncSetAttribute(poly_norm_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  }
  if (n % 8 == 0 && aligned16(z) && aligned16(y)) {
    const dim3 block8(row_block(n / 2));
    if (smem > 48 * 1024) {
      cudaFuncSetAttribute(poly_norm8_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      cudaFuncSetAttribute(poly_norm8_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    }
    if (dtype == LLMIE_F32)
      launch_k(poly_norm8_kernel<float>, grid, block8, smem, stream, (const float*)z, coef, eps, (float*)y, n);
    else if (dtype == LLMIE_BF16)
      launch_k(poly_norm8_kernel<__nv_bfloat16>, grid, block8, smem, stream, (const __nv_bfloat16*)z, coef, eps,
               (__nv_bfloat16*)y, n);
    else
      return LLMIE_ERR_DTYPE;
    LLMIE_LAUNCH_CHECK();
    return LLMIE_OK;
  }
  if (dtype == LLMIE_F32)
    launch_k(poly_norm_kernel<float>, grid, block, smem, stream, (const float*)z, coef, eps, (float*)y, n);
  else if (dtype == LLMIE_BF16)
    launch_k(poly_norm_kernel<__nv_bfloat16>, grid, block, smem, stream, (const __nv_bfloat16*)z, coef, eps,
             (__nv_bfloat16*)y, n);
  else
    return LLMIE_ERR_DTYPE;
  LLMIE_LAUNCH_CHECK();
  return LLMIE_OK;
}

// h, rows, y, w, eps as in llmie_scaled_add_rmsnorm; d1 and d2 (or null) [T, d] of their own dtypes; w1, w2 float32 [d] or
// null (null: that output enters as it is); w_out float32 [d].
extern "C" int llmie_sandwich_add_norm(float* h, const void* d1, int d1_dtype, float c1, const float* w1, const void* d2,
                                       int d2_dtype, float c2, const float* w2, float eps_in, const float* w_out,
                                       float eps_out, const float* w, float eps, void* y, int y_ld, int y_dtype,
                                       const int* rows, int n_out, int d, cudaStream_t stream) {
  if (n_out < 0 || d <= 0 || !h || !d1 || !w_out || (w && !y) || (y && y_ld < d)) return LLMIE_ERR_BAD_ARG;
  if (d > 12288) return LLMIE_ERR_UNSUPPORTED_SIZE;
  if ((y_dtype != LLMIE_F32 && y_dtype != LLMIE_BF16) || (d1_dtype != LLMIE_F32 && d1_dtype != LLMIE_BF16) ||
      (d2 && d2_dtype != LLMIE_F32 && d2_dtype != LLMIE_BF16))
    return LLMIE_ERR_DTYPE;
  if (n_out == 0) return LLMIE_OK;
  bool by4 = d % 4 == 0 && y_ld % 4 == 0;
  for (const void* p : {(const void*)h, d1, d2, (const void*)w1, (const void*)w2, (const void*)w_out, (const void*)w,
                        (const void*)y})
    by4 = by4 && aligned16(p);
  const size_t smem = by4 ? 0 : (size_t)d * sizeof(float);
#define LLMIE_SANDWICH(K, TY, THREADS)                                                                                   \
  launch_k(K, dim3(n_out), dim3(THREADS), smem, stream, h, d1, d1_dtype, c1, w1, d2, d2_dtype, c2, w2, eps_in, w_out,    \
           eps_out, w, eps, (TY*)y, y_ld, rows, d)
#define LLMIE_SANDWICH_TY(TY)                                                                                            \
  do {                                                                                                                   \
    const int runs = by4 ? d / 4 : 0;                                                                                    \
    if (!by4) LLMIE_SANDWICH(sandwich_add_norm_kernel<TY>, TY, row_block(d));                                            \
    else if (runs <= 512) LLMIE_SANDWICH((sandwich_add_norm4_kernel<TY, 1>), TY, (runs + 31) / 32 * 32);                 \
    else if (runs <= 1024) LLMIE_SANDWICH((sandwich_add_norm4_kernel<TY, 2>), TY, ((runs + 1) / 2 + 31) / 32 * 32);      \
    else LLMIE_SANDWICH((sandwich_add_norm4_kernel<TY, 6>), TY, ((runs + 5) / 6 + 31) / 32 * 32);                        \
  } while (0)
  if (y_dtype == LLMIE_F32) LLMIE_SANDWICH_TY(float);
  else LLMIE_SANDWICH_TY(__nv_bfloat16);
#undef LLMIE_SANDWICH_TY
#undef LLMIE_SANDWICH
  LLMIE_LAUNCH_CHECK();
  return LLMIE_OK;
}
