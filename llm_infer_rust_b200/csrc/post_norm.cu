// A residual stream that is kept in float whatever the engine's dtype, for layers whose norms sit on the sublayers'
// OUTPUTS:  x <- x + N(y),  N(y) = (y + bias) / sqrt(mean((y + bias)^2) + eps) * w, or with CENTER (a layer norm without
// bias) the same of y + bias less its mean over the row: the sum of squares is taken of the deviations, in a pass of its
// own.
//
//   norm_add      the update above for every token; x (float) is changed in place, and if `cast_out` is given it also
//                 receives x rounded once to the engine's dtype (what the next sublayer's first product reads), so the
//                 stream is never read again just to be rounded.  y: float or the engine's dtype; bias: float, per
//                 column, or none (an output projection's bias, added here in float instead of in a kernel of its own).
//   norm_add_pair the same update with the mean of two normed branches in place of y: y = (R(a; wa) + R(b; wb)) / 2, R the
//                 RMS norm of a branch with its own weights (a layer of two mixers side by side)
//   residual_sum  the other arrangement, whose norm sits on a sublayer's INPUT and is handed the sum of the layer before:
//                 x <- x + m (y + bias + f), y the mixer's output (or the mean of two normed branches, as above) and f the
//                 feed-forward's, both of the same input; then out = R(x) w or, without a weight, x itself, rounded once
//                 (rows of `out` may lie further apart than they are wide).
//   norm_rows     out[r] = N(x[rows[r]]) without the add (the model's last norm, at the rows whose logits are wanted).
//
// One block a token; a row's sum of squares is added in an order fixed by the thread layout, so a token's result does
// not depend on what else is in the step.
#include "common.cuh"

constexpr int PN_THREADS = 256, PN_MAX_THREADS = 1024;

template <typename T> __device__ __forceinline__ void store4(T* p, float a, float b, float c, float d);
template <> __device__ __forceinline__ void store4<float>(float* p, float a, float b, float c, float d) {
  *reinterpret_cast<float4*>(p) = make_float4(a, b, c, d);
}
template <> __device__ __forceinline__ void store4<__nv_bfloat16>(__nv_bfloat16* p, float a, float b, float c, float d) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
  uint2 v;
  v.x = *reinterpret_cast<const uint32_t*>(&lo);
  v.y = *reinterpret_cast<const uint32_t*>(&hi);
  *reinterpret_cast<uint2*>(p) = v;
}

// Up to PN_MAX_THREADS threads a block (the launcher gives a step of few tokens more threads each); a width that is a
// multiple of four is taken four columns at a time.
// The factor 1 / sqrt(mean(v^2) + eps) of a row of `width` floats in shared memory whose sum and sum of squares the
// block's threads hold in parts; CENTER: the row's mean is taken off the row first (every thread changes the elements
// that it wrote itself, VEC neighbouring ones at a time).
template <bool CENTER, int VEC>
__device__ __forceinline__ float row_factor(float* row, float sum, float ss, float eps, int width, float* scratch) {
  if constexpr (CENTER) {
    const float mean = block_sum(sum, scratch) / static_cast<float>(width);
    ss = 0.0f;
    for (int c = VEC * threadIdx.x; c < width; c += VEC * blockDim.x)
#pragma unroll
      for (int i = 0; i < VEC; ++i) {
        const float v = row[c + i] - mean;
        row[c + i] = v;
        ss = fmaf(v, v, ss);
      }
  }
  ss = block_sum(ss, scratch);
  return 1.0f / sqrtf(ss / static_cast<float>(width) + eps);
}

template <typename TY, typename TO, bool CENTER>
__global__ void __launch_bounds__(PN_MAX_THREADS)
norm_add_kernel(float* __restrict__ x, const TY* __restrict__ y, const float* __restrict__ bias,
                const float* __restrict__ w, float eps, TO* __restrict__ cast_out, int width) {
  pdl_launch_dependents();                          // the kernel after this one may be scheduled; it waits before it reads
  pdl_wait();                                        // what this kernel reads belongs to the kernels before it
  __shared__ float scratch[33];
  extern __shared__ float row[];                     // width floats: y + bias
  const size_t t = blockIdx.x;
  const TY* src = y + t * width;
  float* xr = x + t * width;
  float ss = 0.0f, sum = 0.0f;
  if (width % 4 == 0) {
#pragma unroll 2
    for (int c = 4 * threadIdx.x; c < width; c += 4 * blockDim.x) {
      float v[4];
      load_floats<TY, 4>(src + c, v);
      if (bias != nullptr) {
        const float4 b = *reinterpret_cast<const float4*>(bias + c);
        v[0] += b.x; v[1] += b.y; v[2] += b.z; v[3] += b.w;
      }
      *reinterpret_cast<float4*>(row + c) = make_float4(v[0], v[1], v[2], v[3]);
      if constexpr (CENTER) sum += (v[0] + v[1]) + (v[2] + v[3]);
      else { ss = fmaf(v[0], v[0], ss); ss = fmaf(v[1], v[1], ss); ss = fmaf(v[2], v[2], ss); ss = fmaf(v[3], v[3], ss); }
    }
    const float r = row_factor<CENTER, 4>(row, sum, ss, eps, width, scratch);
#pragma unroll 2
    for (int c = 4 * threadIdx.x; c < width; c += 4 * blockDim.x) {
      const float4 a = *reinterpret_cast<const float4*>(xr + c);
      const float4 g = *reinterpret_cast<const float4*>(w + c);
      const float4 v = *reinterpret_cast<const float4*>(row + c);
      const float s0 = a.x + v.x * r * g.x, s1 = a.y + v.y * r * g.y, s2 = a.z + v.z * r * g.z, s3 = a.w + v.w * r * g.w;
      *reinterpret_cast<float4*>(xr + c) = make_float4(s0, s1, s2, s3);
      if (cast_out != nullptr) store4<TO>(cast_out + t * width + c, s0, s1, s2, s3);
    }
    return;
  }
  for (int c = threadIdx.x; c < width; c += blockDim.x) {
    float v = to_f32<TY>(src[c]);
    if (bias != nullptr) v += bias[c];
    row[c] = v;
    if constexpr (CENTER) sum += v;
    else ss = fmaf(v, v, ss);
  }
  const float r = row_factor<CENTER, 1>(row, sum, ss, eps, width, scratch);
  for (int c = threadIdx.x; c < width; c += blockDim.x) {
    const float s = xr[c] + row[c] * r * w[c];
    xr[c] = s;
    if (cast_out != nullptr) cast_out[t * width + c] = from_f32<TO>(s);
  }
}

// The sums of both branches' squares meet first; then the row of their mean is made in shared memory and goes on as in
// norm_add.  Shared memory: width floats (the branches are read twice; a row is a few KB).
template <typename TY, typename TO, bool CENTER>
__global__ void __launch_bounds__(PN_MAX_THREADS)
norm_add_pair_kernel(float* __restrict__ x, const TY* __restrict__ a, const TY* __restrict__ b, const float* __restrict__ wa,
                     const float* __restrict__ wb, const float* __restrict__ w, float eps, TO* __restrict__ cast_out, int width) {
  pdl_launch_dependents();                          // the kernel after this one may be scheduled; it waits before it reads
  pdl_wait();                                        // what this kernel reads belongs to the kernels before it
  __shared__ float scratch[33];
  extern __shared__ float row[];
  const size_t t = blockIdx.x;
  const TY* ar = a + t * width;
  const TY* br = b + t * width;
  float* xr = x + t * width;
  float sa = 0.0f, sb = 0.0f, ss = 0.0f, sum = 0.0f;
  if (width % 4 == 0) {
    for (int c = 4 * threadIdx.x; c < width; c += 4 * blockDim.x) {
      float u[4], v[4];
      load_floats<TY, 4>(ar + c, u);
      load_floats<TY, 4>(br + c, v);
#pragma unroll
      for (int i = 0; i < 4; ++i) { sa = fmaf(u[i], u[i], sa); sb = fmaf(v[i], v[i], sb); }
    }
    const float fa = 0.5f / sqrtf(block_sum(sa, scratch) / static_cast<float>(width) + eps);
    const float fb = 0.5f / sqrtf(block_sum(sb, scratch) / static_cast<float>(width) + eps);
    for (int c = 4 * threadIdx.x; c < width; c += 4 * blockDim.x) {
      float u[4], v[4];
      load_floats<TY, 4>(ar + c, u);
      load_floats<TY, 4>(br + c, v);
      const float4 ga = *reinterpret_cast<const float4*>(wa + c), gb = *reinterpret_cast<const float4*>(wb + c);
      const float y[4] = {u[0] * fa * ga.x + v[0] * fb * gb.x, u[1] * fa * ga.y + v[1] * fb * gb.y,
                          u[2] * fa * ga.z + v[2] * fb * gb.z, u[3] * fa * ga.w + v[3] * fb * gb.w};
      *reinterpret_cast<float4*>(row + c) = make_float4(y[0], y[1], y[2], y[3]);
#pragma unroll
      for (int i = 0; i < 4; ++i) { sum += y[i]; ss = fmaf(y[i], y[i], ss); }
    }
    const float r = row_factor<CENTER, 4>(row, sum, ss, eps, width, scratch);
    for (int c = 4 * threadIdx.x; c < width; c += 4 * blockDim.x) {
      const float4 o = *reinterpret_cast<const float4*>(xr + c);
      const float4 g = *reinterpret_cast<const float4*>(w + c);
      const float4 v = *reinterpret_cast<const float4*>(row + c);
      const float s0 = o.x + v.x * r * g.x, s1 = o.y + v.y * r * g.y, s2 = o.z + v.z * r * g.z, s3 = o.w + v.w * r * g.w;
      *reinterpret_cast<float4*>(xr + c) = make_float4(s0, s1, s2, s3);
      if (cast_out != nullptr) store4<TO>(cast_out + t * width + c, s0, s1, s2, s3);
    }
    return;
  }
  for (int c = threadIdx.x; c < width; c += blockDim.x) {
    const float u = to_f32<TY>(ar[c]), v = to_f32<TY>(br[c]);
    sa = fmaf(u, u, sa);
    sb = fmaf(v, v, sb);
  }
  const float fa = 0.5f / sqrtf(block_sum(sa, scratch) / static_cast<float>(width) + eps);
  const float fb = 0.5f / sqrtf(block_sum(sb, scratch) / static_cast<float>(width) + eps);
  for (int c = threadIdx.x; c < width; c += blockDim.x) {
    const float y = to_f32<TY>(ar[c]) * fa * wa[c] + to_f32<TY>(br[c]) * fb * wb[c];
    row[c] = y;
    sum += y;
    ss = fmaf(y, y, ss);
  }
  const float r = row_factor<CENTER, 1>(row, sum, ss, eps, width, scratch);
  for (int c = threadIdx.x; c < width; c += blockDim.x) {
    const float s = xr[c] + row[c] * r * w[c];
    xr[c] = s;
    if (cast_out != nullptr) cast_out[t * width + c] = from_f32<TO>(s);
  }
}

// Shared memory: width floats.  rows (null: every token): out[r] is made of token rows[r].
template <typename TY>
struct ResidualTerms {
  const TY* y;               // the mixer's output, or null
  const TY* b;               // the second branch: y and b are then normed with wa and wb and their mean taken
  const TY* f;               // the feed-forward's output, or null
  const float* bias;         // per column, on y (without a second branch), or null
  const float* wa;
  const float* wb;
};

template <typename TY, typename TO, int VEC>
__global__ void __launch_bounds__(PN_MAX_THREADS)
residual_sum_kernel(float* __restrict__ x, ResidualTerms<TY> in, float mult, const float* __restrict__ w, float eps,
                    const int* __restrict__ rows, TO* __restrict__ out, size_t out_stride, int store, int width) {
  pdl_launch_dependents();                          // the kernel after this one may be scheduled; it waits before it reads
  pdl_wait();                                        // what this kernel reads belongs to the kernels before it
  __shared__ float scratch[33];
  extern __shared__ float row[];                     // x after the sum
  const size_t t = rows != nullptr ? static_cast<size_t>(rows[blockIdx.x]) : blockIdx.x;
  float* xr = x + t * width;
  auto load = [](const TY* p, float (&v)[VEC]) {
    if constexpr (VEC == 4) load_floats<TY, 4>(p, v);
    else v[0] = to_f32<TY>(*p);
  };
  auto load_f = [](const float* p, float (&v)[VEC]) {
    if constexpr (VEC == 4) load_floats<float, 4>(p, v);
    else v[0] = *p;
  };
  float fa = 0.0f, fb = 0.0f;
  if (in.b != nullptr) {
    float sa = 0.0f, sb = 0.0f;
    for (int c = VEC * threadIdx.x; c < width; c += VEC * blockDim.x) {
      float u[VEC], v[VEC];
      load(in.y + t * width + c, u);
      load(in.b + t * width + c, v);
#pragma unroll
      for (int i = 0; i < VEC; ++i) { sa = fmaf(u[i], u[i], sa); sb = fmaf(v[i], v[i], sb); }
    }
    fa = 0.5f / sqrtf(block_sum(sa, scratch) / static_cast<float>(width) + eps);
    fb = 0.5f / sqrtf(block_sum(sb, scratch) / static_cast<float>(width) + eps);
  }
  float ss = 0.0f;
#pragma unroll 2
  for (int c = VEC * threadIdx.x; c < width; c += VEC * blockDim.x) {
    float s[VEC] = {}, v[VEC], g[VEC];
    if (in.y != nullptr) {
      load(in.y + t * width + c, s);
      if (in.b != nullptr) {
        float h[VEC];
        load(in.b + t * width + c, v);
        load_f(in.wa + c, g);
        load_f(in.wb + c, h);
#pragma unroll
        for (int i = 0; i < VEC; ++i) s[i] = s[i] * fa * g[i] + v[i] * fb * h[i];
      } else if (in.bias != nullptr) {
        load_f(in.bias + c, g);
#pragma unroll
        for (int i = 0; i < VEC; ++i) s[i] += g[i];
      }
    }
    if (in.f != nullptr) {
      load(in.f + t * width + c, v);
#pragma unroll
      for (int i = 0; i < VEC; ++i) s[i] += v[i];
    }
    load_f(xr + c, v);
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      v[i] = fmaf(mult, s[i], v[i]);
      ss = fmaf(v[i], v[i], ss);
    }
    if constexpr (VEC == 4) {
      const float4 sum = make_float4(v[0], v[1], v[2], v[3]);
      *reinterpret_cast<float4*>(row + c) = sum;
      if (store) *reinterpret_cast<float4*>(xr + c) = sum;
    } else {
      row[c] = v[0];
      if (store) xr[c] = v[0];
    }
  }
  if (out == nullptr) return;
  float r = 1.0f;
  if (w != nullptr) r = 1.0f / sqrtf(block_sum(ss, scratch) / static_cast<float>(width) + eps);
  for (int c = VEC * threadIdx.x; c < width; c += VEC * blockDim.x) {     // (a thread reads what it wrote itself)
    float v[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = w != nullptr ? row[c + i] * r * w[c + i] : row[c + i];
    TO* dst = out + blockIdx.x * out_stride + c;
    if constexpr (VEC == 4) store4<TO>(dst, v[0], v[1], v[2], v[3]);
    else *dst = from_f32<TO>(v[0]);
  }
}

template <typename TO, bool CENTER>
__global__ void __launch_bounds__(PN_THREADS)
norm_rows_kernel(TO* __restrict__ out, const float* __restrict__ x, const int* __restrict__ rows,
                 const float* __restrict__ w, float eps, int width) {
  pdl_launch_dependents();                          // the kernel after this one may be scheduled; it waits before it reads
  pdl_wait();                                        // what this kernel reads belongs to the kernels before it
  __shared__ float scratch[33];
  const size_t r_out = blockIdx.x;
  const size_t t = rows != nullptr ? static_cast<size_t>(rows[r_out]) : r_out;
  const float* src = x + t * width;
  float ss = 0.0f, mean = 0.0f;
  if constexpr (CENTER) {
    float sum = 0.0f;
    for (int c = threadIdx.x; c < width; c += blockDim.x) sum += src[c];
    mean = block_sum(sum, scratch) / static_cast<float>(width);
  }
  for (int c = threadIdx.x; c < width; c += blockDim.x) {
    const float v = src[c] - mean;
    ss = fmaf(v, v, ss);
  }
  ss = block_sum(ss, scratch);
  const float r = 1.0f / sqrtf(ss / static_cast<float>(width) + eps);
  for (int c = threadIdx.x; c < width; c += blockDim.x) out[r_out * width + c] = from_f32<TO>((src[c] - mean) * r * w[c]);
}

// y_dtype: dtype of y (and of b); out_dtype: dtype of cast_out (ignored when cast_out is null); center: the norm takes the
// row's mean off first.  b (null: none): y and b are two branches with their own weights wa and wb (see norm_add_pair).
static int run_norm_add(float* x, const void* y, const void* b, int y_dtype, const float* bias, const float* wa,
                        const float* wb, const float* w, float eps, int center, void* cast_out, int out_dtype, int tokens,
                        int width, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (width <= 0 || width * sizeof(float) > 200 * 1024) return B200_BAD_SIZE;
  const size_t smem = static_cast<size_t>(width) * sizeof(float);
  // a step of few tokens: as many threads a block as the row has groups of four columns, up to PN_MAX_THREADS
  const int threads = tokens <= 64 ? min(PN_MAX_THREADS, max(PN_THREADS, (width / 4 + 31) / 32 * 32)) : PN_THREADS;
#define B200_NORM_ADD_C(TY, TO, C)                                                                             \
  do {                                                                                                         \
    if (smem > 48 * 1024) {                                                                                    \
      cudaError_t e = b != nullptr                                                                             \
          ? cudaFuncSetAttribute(norm_add_pair_kernel<TY, TO, C>, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                                 static_cast<int>(smem))                                                       \
          : cudaFuncSetAttribute(norm_add_kernel<TY, TO, C>, cudaFuncAttributeMaxDynamicSharedMemorySize,      \
                                 static_cast<int>(smem));                                                      \
      if (e != cudaSuccess) return static_cast<int>(e);                                                        \
    }                                                                                                          \
    if (b != nullptr)                                                                                          \
      return b200_launch(norm_add_pair_kernel<TY, TO, C>, dim3(tokens), dim3(threads), smem, stream, 0, x,     \
                         static_cast<const TY*>(y), static_cast<const TY*>(b), wa, wb, w, eps,                 \
                         static_cast<TO*>(cast_out), width);                                                   \
    return b200_launch(norm_add_kernel<TY, TO, C>, dim3(tokens), dim3(threads), smem, stream, 0, x,            \
                       static_cast<const TY*>(y), bias, w, eps, static_cast<TO*>(cast_out), width);            \
  } while (0)
#define B200_NORM_ADD(TY, TO)              \
  do {                                     \
    if (center) B200_NORM_ADD_C(TY, TO, true); \
    B200_NORM_ADD_C(TY, TO, false);        \
  } while (0)
  const bool to_bf16 = cast_out != nullptr && out_dtype == B200_BF16;
  if (cast_out != nullptr && out_dtype != B200_BF16 && out_dtype != B200_F32) return B200_BAD_DTYPE;
  if (y_dtype == B200_F32) {
    if (to_bf16) B200_NORM_ADD(float, __nv_bfloat16);
    B200_NORM_ADD(float, float);
  } else if (y_dtype == B200_BF16) {
    if (to_bf16) B200_NORM_ADD(__nv_bfloat16, __nv_bfloat16);
    B200_NORM_ADD(__nv_bfloat16, float);
  }
#undef B200_NORM_ADD
#undef B200_NORM_ADD_C
  return B200_BAD_DTYPE;
}

B200_EXPORT int b200_norm_add(float* x, const void* y, int y_dtype, const float* bias, const float* w, float eps, int center,
                              void* cast_out, int out_dtype, int tokens, int width, cudaStream_t stream) {
  return run_norm_add(x, y, nullptr, y_dtype, bias, nullptr, nullptr, w, eps, center, cast_out, out_dtype, tokens, width, stream);
}

B200_EXPORT int b200_norm_add_pair(float* x, const void* a, const void* b, int y_dtype, const float* wa, const float* wb,
                                   const float* w, float eps, int center, void* cast_out, int out_dtype, int tokens, int width,
                                   cudaStream_t stream) {
  if (a == nullptr || b == nullptr) return B200_BAD_SIZE;
  return run_norm_add(x, a, b, y_dtype, nullptr, wa, wb, w, eps, center, cast_out, out_dtype, tokens, width, stream);
}

// x [.., width] float.  y, b, f: dtype y_dtype, any of them null (b only with y, wa and wb); w null: no norm.  n: rows of
// out (and of `rows`); store 0: x stays as it is.
B200_EXPORT int b200_residual_sum(float* x, const void* y, const void* b, const void* f, int y_dtype, const float* bias,
                                  const float* wa, const float* wb, float mult, const float* w, float eps, const int* rows,
                                  void* out, int out_dtype, int out_stride, int store, int n, int width,
                                  cudaStream_t stream) {
  if (n <= 0) return 0;
  if (width <= 0 || width * sizeof(float) > 200 * 1024 || (b != nullptr && (y == nullptr || wa == nullptr || wb == nullptr)))
    return B200_BAD_SIZE;
  if (out != nullptr && out_stride < width) return B200_BAD_SIZE;
  const size_t smem = static_cast<size_t>(width) * sizeof(float);
  const int threads = n <= 64 ? min(PN_MAX_THREADS, max(PN_THREADS, (width / 4 + 31) / 32 * 32)) : PN_THREADS;
  const bool vec = width % 4 == 0 && out_stride % 4 == 0 && reinterpret_cast<uintptr_t>(out) % 16 == 0;
#define B200_RESIDUAL(TY, TO, V)                                                                                     \
  do {                                                                                                               \
    const ResidualTerms<TY> in = {static_cast<const TY*>(y), static_cast<const TY*>(b), static_cast<const TY*>(f),   \
                                  bias, wa, wb};                                                                     \
    if (smem > 48 * 1024) {                                                                                          \
      cudaError_t e = cudaFuncSetAttribute(residual_sum_kernel<TY, TO, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                                           static_cast<int>(smem));                                                  \
      if (e != cudaSuccess) return static_cast<int>(e);                                                              \
    }                                                                                                                \
    return b200_launch(residual_sum_kernel<TY, TO, V>, dim3(n), dim3(threads), smem, stream, 0, x, in, mult, w, eps,  \
                       rows, static_cast<TO*>(out), static_cast<size_t>(out_stride), store, width);                  \
  } while (0)
#define B200_RESIDUAL_V(TY, TO)        \
  do {                                 \
    if (vec) B200_RESIDUAL(TY, TO, 4); \
    B200_RESIDUAL(TY, TO, 1);          \
  } while (0)
  if (y_dtype == B200_F32 && out_dtype == B200_F32) B200_RESIDUAL_V(float, float);
  if (y_dtype == B200_F32 && out_dtype == B200_BF16) B200_RESIDUAL_V(float, __nv_bfloat16);
  if (y_dtype == B200_BF16 && out_dtype == B200_F32) B200_RESIDUAL_V(__nv_bfloat16, float);
  if (y_dtype == B200_BF16 && out_dtype == B200_BF16) B200_RESIDUAL_V(__nv_bfloat16, __nv_bfloat16);
#undef B200_RESIDUAL_V
#undef B200_RESIDUAL
  return B200_BAD_DTYPE;
}

B200_EXPORT int b200_norm_rows(void* out, int out_dtype, const float* x, const int* rows, const float* w, float eps, int center,
                               int n, int width, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (width <= 0) return B200_BAD_SIZE;
#define B200_NORM_ROWS(TO)                                                                                                  \
  return b200_launch(center ? norm_rows_kernel<TO, true> : norm_rows_kernel<TO, false>, dim3(n), dim3(PN_THREADS), 0, stream, \
                     0, static_cast<TO*>(out), x, rows, w, eps, width)
  if (out_dtype == B200_F32) B200_NORM_ROWS(float);
  if (out_dtype == B200_BF16) B200_NORM_ROWS(__nv_bfloat16);
#undef B200_NORM_ROWS
  return B200_BAD_DTYPE;
}
