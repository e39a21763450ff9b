// A real-gated linear recurrent unit, channel by channel, with the state of every request in float32:
//
//   r = sigmoid(R_b u_b + r_bias),  i = sigmoid(I_b u_b + i_bias)      u in `blocks` equal parts u_b, R_b and I_b square
//   log a = -8 r softplus(lam),     S <- a S + sqrt(1 - a^2) i u,      out = S * gelu_tanh(y + y_bias)
//
// u [tokens, width] comes out of a short convolution, y is a column range of a packed projection.  sqrt(1 - a^2) is taken
// as sqrt(-expm1(2 log a)), which keeps its digits where a is close to one.
//
//   lru_few      a step of few rows of one token each: the block products, the recurrence and the gate in one kernel
//   lru_rows     rows of one token each, the block products `pre` given
//   lru_scan     rows of any length, `pre` given, in windows of 32 tokens: (1) a and the added term of every token, left in
//                place of their pre-activations, and every window's own contribution, (2) the windows of a row folded in
//                order, (3) the recurrence of every window from the state it starts with.  Inside a window the recurrence
//                runs token by token.
// pre [blocks, tokens, 2 * size] float: R_b u_b, then I_b u_b.  state [slots + 1, width]; a row whose prefix_len is 0
// starts from zeros; slot 0 takes padding rows.
#include "common.cuh"

constexpr int LRU_WINDOW = 32;

struct LruParams {
  int width, size;             // size: channels of a block
  const float *r_bias, *i_bias, *lam, *y_bias;
  int y_stride;                // columns of a row that y lies in
};

__device__ __forceinline__ float softplus_of(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float gelu_tanh_of(float z) {
  return 0.5f * z * (1.0f + tanhf(0.79788456080286535588f * (z + 0.044715f * z * z * z)));
}

// a and the term that is added to a S
__device__ __forceinline__ void lru_terms(float r_pre, float i_pre, float u, float rate /* 8 softplus(lam) */, float& a, float& add) {
  const float r = 1.0f / (1.0f + expf(-r_pre)), i = 1.0f / (1.0f + expf(-i_pre));
  const float log_a = -rate * r;
  a = expf(log_a);
  add = sqrtf(-expm1f(2.0f * log_a)) * (i * u);
}

// grid (ceil(width / 8)), 8 warps: a warp takes one channel, streams that channel's row of R and of I once for up to
// LRU_FEW rows at a time, then lane m runs row m's recurrence.
constexpr int LRU_FEW = 8;
template <typename T>
__global__ void __launch_bounds__(256)
lru_few_kernel(const T* __restrict__ u, const T* __restrict__ y, const T* __restrict__ gates /* [blocks, 2 size, size] */,
               LruParams p, float* __restrict__ state, const int* __restrict__ prefix_len, const int* __restrict__ state_slots,
               T* __restrict__ out, int rows) {
  pdl_launch_dependents();                          // the kernel after this one may be scheduled; it waits before it reads
  pdl_wait();                                        // what this kernel reads belongs to the kernels before it
  const int lane = threadIdx.x & 31;
  const int c = blockIdx.x * 8 + (threadIdx.x >> 5);
  if (c >= p.width) return;
  const int b = c / p.size, j = c - b * p.size;
  const T* wr = gates + (static_cast<size_t>(b) * 2 * p.size + j) * p.size;
  const T* wi = wr + static_cast<size_t>(p.size) * p.size;
  const float rate = 8.0f * softplus_of(p.lam[c]);
  const bool wide = p.size % 8 == 0 && p.width % 8 == 0;
  for (int m0 = 0; m0 < rows; m0 += LRU_FEW) {
    const int nr = min(LRU_FEW, rows - m0);
    float ar[LRU_FEW], ai[LRU_FEW];
#pragma unroll
    for (int m = 0; m < LRU_FEW; ++m) ar[m] = ai[m] = 0.0f;
    const T* ub = u + static_cast<size_t>(m0) * p.width + b * p.size;
    if (wide) {
      for (int k = lane * 8; k < p.size; k += 256) {
        float g[8], h[8];
        load_floats<T, 8>(wr + k, g);
        load_floats<T, 8>(wi + k, h);
#pragma unroll
        for (int m = 0; m < LRU_FEW; ++m) {          // a row beyond the last reads the last one; its sums are dropped
          float v[8];
          load_floats<T, 8>(ub + static_cast<size_t>(min(m, nr - 1)) * p.width + k, v);
#pragma unroll
          for (int e = 0; e < 8; ++e) {
            ar[m] = fmaf(g[e], v[e], ar[m]);
            ai[m] = fmaf(h[e], v[e], ai[m]);
          }
        }
      }
    } else {
      for (int k = lane; k < p.size; k += 32) {
        const float g = to_f32<T>(wr[k]), h = to_f32<T>(wi[k]);
#pragma unroll
        for (int m = 0; m < LRU_FEW; ++m) {
          const float v = to_f32<T>(ub[static_cast<size_t>(min(m, nr - 1)) * p.width + k]);
          ar[m] = fmaf(g, v, ar[m]);
          ai[m] = fmaf(h, v, ai[m]);
        }
      }
    }
    float mine_r = 0.0f, mine_i = 0.0f;
#pragma unroll
    for (int m = 0; m < LRU_FEW; ++m) {
      const float s = warp_sum(ar[m]), q = warp_sum(ai[m]);
      if (lane == m) { mine_r = s; mine_i = q; }
    }
    if (lane < nr) {
      const int m = m0 + lane;
      float a, add;
      lru_terms(mine_r + p.r_bias[c], mine_i + p.i_bias[c], to_f32<T>(u[static_cast<size_t>(m) * p.width + c]), rate, a, add);
      float* st = state + static_cast<size_t>(state_slots[m]) * p.width + c;
      const float S = prefix_len[m] > 0 ? fmaf(a, *st, add) : add;
      *st = S;
      out[static_cast<size_t>(m) * p.width + c] =
          from_f32<T>(S * gelu_tanh_of(to_f32<T>(y[static_cast<size_t>(m) * p.y_stride + c]) + p.y_bias[c]));
    }
  }
}

// One element's pre-activations (biases included).
__device__ __forceinline__ void pre_of(const float* __restrict__ pre, const LruParams& p, int tokens, int t, int c, float& r, float& i) {
  const int b = c / p.size, j = c - b * p.size;
  const float* at = pre + (static_cast<size_t>(b) * tokens + t) * 2 * p.size + j;
  r = at[0] + p.r_bias[c];
  i = at[p.size] + p.i_bias[c];
}

// grid (rows, channel tiles of 256): row m is token m
template <typename T>
__global__ void __launch_bounds__(256)
lru_rows_kernel(const T* __restrict__ u, const T* __restrict__ y, const float* __restrict__ pre, LruParams p,
                float* __restrict__ state, const int* __restrict__ prefix_len, const int* __restrict__ state_slots,
                T* __restrict__ out, int rows) {
  pdl_launch_dependents();                          // the kernel after this one may be scheduled; it waits before it reads
  pdl_wait();                                        // what this kernel reads belongs to the kernels before it
  const int m = blockIdx.x, c = blockIdx.y * 256 + threadIdx.x;
  if (c >= p.width) return;
  float r, i, a, add;
  pre_of(pre, p, rows, m, c, r, i);
  lru_terms(r, i, to_f32<T>(u[static_cast<size_t>(m) * p.width + c]), 8.0f * softplus_of(p.lam[c]), a, add);
  float* st = state + static_cast<size_t>(state_slots[m]) * p.width + c;
  const float S = prefix_len[m] > 0 ? fmaf(a, *st, add) : add;
  *st = S;
  out[static_cast<size_t>(m) * p.width + c] =
      from_f32<T>(S * gelu_tanh_of(to_f32<T>(y[static_cast<size_t>(m) * p.y_stride + c]) + p.y_bias[c]));
}

// (1) grid (windows, channel tiles of 128).  Besides every token's terms, the segment of the window's LAST row: the product
// of its a and the state it leaves when it starts from zero.  (Rows that end inside the window leave nothing to a later
// one.)  Four tokens' loads are in flight at a time.
template <typename T>
__global__ void __launch_bounds__(128)
lru_window_kernel(const T* __restrict__ u, float* __restrict__ pre, LruParams p, const int* __restrict__ row_of_token,
                  const int* __restrict__ cu_q, float* __restrict__ win_a, float* __restrict__ win_s, int tokens) {
  const int w = blockIdx.x, c = blockIdx.y * 128 + threadIdx.x;
  if (c >= p.width) return;
  const int t0 = w * LRU_WINDOW, end = min(t0 + LRU_WINDOW, tokens);
  const int begin = cu_q[row_of_token[end - 1]];
  const float rate = 8.0f * softplus_of(p.lam[c]), rb = p.r_bias[c], ib = p.i_bias[c];
  const int b = c / p.size, j = c - b * p.size;
  float* at = pre + static_cast<size_t>(b) * tokens * 2 * p.size + j;
  float A = 1.0f, S = 0.0f;
  for (int t = t0; t < end; t += 4) {
    float r[4], i[4], x[4];
#pragma unroll
    for (int m = 0; m < 4; ++m) {
      const int s = min(t + m, end - 1);
      r[m] = at[static_cast<size_t>(s) * 2 * p.size];
      i[m] = at[static_cast<size_t>(s) * 2 * p.size + p.size];
      x[m] = to_f32<T>(u[static_cast<size_t>(s) * p.width + c]);
    }
#pragma unroll
    for (int m = 0; m < 4; ++m) {
      if (t + m >= end) break;
      float a, add;
      lru_terms(r[m] + rb, i[m] + ib, x[m], rate, a, add);
      at[static_cast<size_t>(t + m) * 2 * p.size] = a;
      at[static_cast<size_t>(t + m) * 2 * p.size + p.size] = add;
      if (t + m >= begin) {
        A *= a;
        S = fmaf(a, S, add);
      }
    }
  }
  win_a[static_cast<size_t>(w) * p.width + c] = A;
  win_s[static_cast<size_t>(w) * p.width + c] = S;
}

// (2) grid (rows, channel tiles of 128): start[r] = the state the row begins with (its slot is written in (3), by another
// block), carry[w] = the state with which the row enters window w, for the windows it does not begin in.
__global__ void __launch_bounds__(128)
lru_fold_kernel(LruParams p, const float* __restrict__ state, const int* __restrict__ cu_q, const int* __restrict__ prefix_len,
                const int* __restrict__ state_slots, const float* __restrict__ win_a, const float* __restrict__ win_s,
                float* __restrict__ carry, float* __restrict__ start) {
  const int r = blockIdx.x, c = blockIdx.y * 128 + threadIdx.x;
  if (c >= p.width) return;
  const int first = cu_q[r], last = cu_q[r + 1] - 1;
  float S = prefix_len[r] > 0 ? state[static_cast<size_t>(state_slots[r]) * p.width + c] : 0.0f;
  start[static_cast<size_t>(r) * p.width + c] = S;
  if (last < first) return;
  const int w0 = first / LRU_WINDOW, w1 = last / LRU_WINDOW;
#pragma unroll 4
  for (int w = w0; w < w1; ++w) {
    const size_t at = static_cast<size_t>(w) * p.width + c;
    S = fmaf(win_a[at], S, win_s[at]);
    carry[at + p.width] = S;
  }
}

// (3) grid (windows, channel tiles of 128)
template <typename T>
__global__ void __launch_bounds__(128)
lru_output_kernel(const T* __restrict__ y, const float* __restrict__ terms, LruParams p, const int* __restrict__ row_of_token,
                  const int* __restrict__ cu_q, const int* __restrict__ state_slots, const float* __restrict__ carry,
                  const float* __restrict__ start, float* __restrict__ state, T* __restrict__ out, int tokens) {
  const int w = blockIdx.x, c = blockIdx.y * 128 + threadIdx.x;
  if (c >= p.width) return;
  const float yb = p.y_bias[c];
  const int b = c / p.size, j = c - b * p.size;
  const float* at = terms + static_cast<size_t>(b) * tokens * 2 * p.size + j;
  const int end = min((w + 1) * LRU_WINDOW, tokens);
  int t = w * LRU_WINDOW;
  while (t < end) {
    const int r = row_of_token[t];
    const int row_end = cu_q[r + 1], stop = min(row_end, end);
    float S = t == cu_q[r] ? start[static_cast<size_t>(r) * p.width + c] : carry[static_cast<size_t>(w) * p.width + c];
#pragma unroll 4
    for (; t < stop; ++t) {
      S = fmaf(at[static_cast<size_t>(t) * 2 * p.size], S, at[static_cast<size_t>(t) * 2 * p.size + p.size]);
      out[static_cast<size_t>(t) * p.width + c] =
          from_f32<T>(S * gelu_tanh_of(to_f32<T>(y[static_cast<size_t>(t) * p.y_stride + c]) + yb));
    }
    if (stop == row_end) state[static_cast<size_t>(state_slots[r]) * p.width + c] = S;
  }
}

// ------------------------------------------------------------------ C interface
static LruParams lru_params(int width, int blocks, const float* r_bias, const float* i_bias, const float* lam,
                            const float* y_bias, int y_stride) {
  LruParams p = {};
  p.width = width;
  p.size = blocks > 0 ? width / blocks : 0;
  p.r_bias = r_bias; p.i_bias = i_bias; p.lam = lam; p.y_bias = y_bias;
  p.y_stride = y_stride;
  return p;
}

// y points at its first column; rows of y are y_stride elements apart.  gates [blocks, 2 size, size] in u's dtype, rows of
// one token each (row m = token m).
B200_EXPORT int b200_lru_few(const void* u, const void* y, int dtype, int y_stride, const void* gates, const float* r_bias,
                             const float* i_bias, const float* lam, const float* y_bias, int width, int blocks, float* state,
                             const int* prefix_len, const int* state_slots, void* out, int rows, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (width <= 0 || blocks <= 0 || width % blocks) return B200_BAD_SIZE;
  const LruParams p = lru_params(width, blocks, r_bias, i_bias, lam, y_bias, y_stride);
  const dim3 grid((width + 7) / 8);
#define B200_LRU_FEW(T)                                                                                                     \
  return b200_launch(lru_few_kernel<T>, grid, dim3(256), 0, stream, 0, static_cast<const T*>(u), static_cast<const T*>(y), \
                     static_cast<const T*>(gates), p, state, prefix_len, state_slots, static_cast<T*>(out), rows)
  if (dtype == B200_F32) B200_LRU_FEW(float);
  if (dtype == B200_BF16) B200_LRU_FEW(__nv_bfloat16);
#undef B200_LRU_FEW
  return B200_BAD_DTYPE;
}

B200_EXPORT int b200_lru_rows(const void* u, const void* y, int dtype, int y_stride, const float* pre, const float* r_bias,
                              const float* i_bias, const float* lam, const float* y_bias, int width, int blocks, float* state,
                              const int* prefix_len, const int* state_slots, void* out, int rows, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (width <= 0 || blocks <= 0 || width % blocks || (width + 255) / 256 > 65535) return B200_BAD_SIZE;
  const LruParams p = lru_params(width, blocks, r_bias, i_bias, lam, y_bias, y_stride);
  const dim3 grid(rows, (width + 255) / 256);
#define B200_LRU_ROWS(T)                                                                                                     \
  return b200_launch(lru_rows_kernel<T>, grid, dim3(256), 0, stream, 0, static_cast<const T*>(u), static_cast<const T*>(y), pre, \
                     p, state, prefix_len, state_slots, static_cast<T*>(out), rows)
  if (dtype == B200_F32) B200_LRU_ROWS(float);
  if (dtype == B200_BF16) B200_LRU_ROWS(__nv_bfloat16);
#undef B200_LRU_ROWS
  return B200_BAD_DTYPE;
}

// `pre` is overwritten.  Scratch: win_a, win_s, carry [ceil(tokens / 32), width] floats each, start [num_rows, width] floats.
B200_EXPORT int b200_lru_window() { return LRU_WINDOW; }

B200_EXPORT int b200_lru_scan(const void* u, const void* y, int dtype, int y_stride, float* pre, const float* r_bias,
                              const float* i_bias, const float* lam, const float* y_bias, int width, int blocks, float* state,
                              const int* row_of_token, const int* cu_q, const int* prefix_len, const int* state_slots,
                              float* win_a, float* win_s, float* carry, float* start, void* out, int tokens, int num_rows,
                              cudaStream_t stream) {
  if (tokens <= 0 || num_rows <= 0) return 0;
  if (width <= 0 || blocks <= 0 || width % blocks || (width + 127) / 128 > 65535) return B200_BAD_SIZE;
  const LruParams p = lru_params(width, blocks, r_bias, i_bias, lam, y_bias, y_stride);
  const int windows = (tokens + LRU_WINDOW - 1) / LRU_WINDOW;
  const dim3 wgrid(windows, (width + 127) / 128), rgrid(num_rows, (width + 127) / 128);
#define B200_LRU_SCAN(T)                                                                                                  \
  do {                                                                                                                    \
    lru_window_kernel<T><<<wgrid, 128, 0, stream>>>(static_cast<const T*>(u), pre, p, row_of_token, cu_q, win_a, win_s, tokens); \
    lru_fold_kernel<<<rgrid, 128, 0, stream>>>(p, state, cu_q, prefix_len, state_slots, win_a, win_s, carry, start);      \
    lru_output_kernel<T><<<wgrid, 128, 0, stream>>>(static_cast<const T*>(y), pre, p, row_of_token, cu_q, state_slots,     \
                                                    carry, start, state, static_cast<T*>(out), tokens);                   \
    return b200_check_launch();                                                                                           \
  } while (0)
  if (dtype == B200_F32) B200_LRU_SCAN(float);
  if (dtype == B200_BF16) B200_LRU_SCAN(__nv_bfloat16);
#undef B200_LRU_SCAN
  return B200_BAD_DTYPE;
}
