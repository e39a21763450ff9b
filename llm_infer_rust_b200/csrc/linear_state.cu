// Linear attention whose state decays per key channel, with or without the delta rule, the state of every request in
// float32.  Per head, with S [d, dv] and the decay g [d] of a token acting on the rows of S:
//
//   plain   S <- diag(g) S + k v^T                                                             o = S^T q
//   delta   S <- diag(g) S;   u = beta (v - S^T k);   S <- S + k u^T                           o = S^T q
//
// What enters it comes out of a packed projection row x (q heads, k heads, v heads, then whatever else):
//   q, k, v   optionally through a short causal convolution over time (its last inputs are per-request state) and an
//             activation; q and k optionally made unit vectors (x / sqrt(sum x^2 + eps)); q times q_scale
//   g         from z [heads * d] (float) and a bias:   LOGISTIC  sigmoid(z + bias)^(1 / tau)
//                                                     SOFTPLUS  exp(-exp(a_log_h) softplus(z + bias))
//   beta      sigmoid of one column a head of x
// heads may be a multiple of the q/k heads: head h uses q and k of head h / (heads / kv_heads).
//
//   state_prepare   the four inputs of every token in float (qf, kf [tokens, kv_heads * d], vf [tokens, heads * dv],
//                   gf [tokens, heads * d], beta [tokens, heads])
//   state_scan      the recurrence, token by token in the sequence's order whatever the step's cut: a position's
//                   result has the same bits however the prompt was cut and whatever else is in the step
//   state_decode    a step whose rows bring one token each: inputs, recurrence, per-head norm and output gate in one
//                   kernel, a block a (row, head)
//
// state [slots + 1, heads, d, dv]; a row whose prefix_len is 0 starts from zeros; slot 0 takes padding rows.
#include "token_conv.cuh"

enum : int { DECAY_LOGISTIC = 0, DECAY_SOFTPLUS = 1 };

struct LinearStateShape {
  int heads, kv_heads, d, dv;
  int beta_column;             // column of x, or -1: no delta rule
  int silu;                    // 1: silu after the convolution (on q, k and v)
  float unit_eps;              // > 0: q and k become unit vectors
  float q_scale;
  int decay_kind;
  float inv_tau;               // LOGISTIC
  const float* decay_bias;     // [heads * d] or null
  const float* a_log;          // [heads], SOFTPLUS
};

__device__ __forceinline__ float silu_of(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float sigmoid_of(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_of(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }

// The decay of one key channel from its pre-activation (bias included) and exp(a_log) of its head.
__device__ __forceinline__ float decay_of(float z, const LinearStateShape& s, float rate) {
  return s.decay_kind == DECAY_LOGISTIC ? expf(-softplus_of(-z) * s.inv_tau) : expf(-rate * softplus_of(z));
}

// ------------------------------------------------------------------ inputs of the recurrence, every token
// grid (tokens, units / 4): a warp takes one unit: a q head, a k head, a v head or a head's decays (and beta).
constexpr int LS_PREP_WARPS = 4;

template <typename T>
__global__ void __launch_bounds__(LS_PREP_WARPS * 32)
state_prepare_kernel(TapsInput<T> in, LinearStateShape s, const float* __restrict__ z, float* __restrict__ qf,
                     float* __restrict__ kf, float* __restrict__ vf, float* __restrict__ gf, float* __restrict__ beta) {
  const int t = blockIdx.x;
  const int lane = threadIdx.x & 31;
  int unit = blockIdx.y * LS_PREP_WARPS + (threadIdx.x >> 5);
  const T* xr = in.x + static_cast<size_t>(t) * in.in_stride;
  if (unit >= 2 * s.kv_heads + 2 * s.heads) return;
  if (unit >= 2 * s.kv_heads + s.heads) {                            // a head's decays
    const int h = unit - 2 * s.kv_heads - s.heads;
    const float rate = s.decay_kind == DECAY_SOFTPLUS ? expf(s.a_log[h]) : 0.0f;
    const size_t base = static_cast<size_t>(t) * s.heads * s.d + static_cast<size_t>(h) * s.d;
    for (int e = lane; e < s.d; e += 32) {
      const float b = s.decay_bias != nullptr ? s.decay_bias[h * s.d + e] : 0.0f;
      gf[base + e] = decay_of(z[base + e] + b, s, rate);
    }
    if (s.beta_column >= 0 && lane == 0)
      beta[static_cast<size_t>(t) * s.heads + h] = sigmoid_of(to_f32<T>(xr[s.beta_column + h]));
    return;
  }
  TapsRow row = {};
  const bool conv = in.w != nullptr;
  if (conv) row = taps_row(in, t);
  auto value = [&](int c) {
    float y = conv ? taps_value(in, row, t, c, false) : to_f32<T>(xr[c]);
    if (s.silu) y = silu_of(y);
    return y;
  };
  if (unit >= 2 * s.kv_heads) {                                      // a v head
    const int h = unit - 2 * s.kv_heads;
    const int c0 = 2 * s.kv_heads * s.d + h * s.dv;
    float* dst = vf + static_cast<size_t>(t) * s.heads * s.dv + static_cast<size_t>(h) * s.dv;
    for (int e = lane; e < s.dv; e += 32) dst[e] = value(c0 + e);
    return;
  }
  const bool is_k = unit >= s.kv_heads;
  const int h = is_k ? unit - s.kv_heads : unit;
  const int c0 = (is_k ? s.kv_heads * s.d : 0) + h * s.d;
  float* dst = (is_k ? kf : qf) + static_cast<size_t>(t) * s.kv_heads * s.d + static_cast<size_t>(h) * s.d;
  float f = is_k ? 1.0f : s.q_scale;
  if (s.unit_eps > 0.0f) {
    constexpr int KEEP = 16;                                         // d <= 512
    float kept[KEEP], ss = 0.0f;
#pragma unroll
    for (int n = 0; n < KEEP; ++n) {
      const int e = lane + 32 * n;
      if (32 * n >= s.d) break;
      kept[n] = e < s.d ? value(c0 + e) : 0.0f;
      ss = fmaf(kept[n], kept[n], ss);
    }
    ss = warp_sum(ss);
    f *= 1.0f / sqrtf(ss + s.unit_eps);
#pragma unroll
    for (int n = 0; n < KEEP; ++n) {
      const int e = lane + 32 * n;
      if (32 * n >= s.d) break;
      if (e < s.d) dst[e] = kept[n] * f;
    }
    return;
  }
  for (int e = lane; e < s.d; e += 32) dst[e] = value(c0 + e) * f;
}

// ------------------------------------------------------------------ the recurrence, token by token
// grid (rows, heads, column tiles of 32).  A block owns 32 columns of one head's state; a column belongs to eight
// neighbouring lanes, lane l of them holding the rows 32 n + 4 l .. + 3 in registers (DI = 4 ceil(d / 32) of them).
// A column's products with k and q are sums over its eight lanes (three shuffles), so a token needs no barrier: the
// block meets only when the next eight tokens have been fetched into shared memory (copies in flight beside the
// recurrence, two buffers).
constexpr int LS_TOKENS = 8;
constexpr int LS_COLS = 32;
constexpr int LS_LANES = 8;

template <int DI, bool DELTA>
__global__ void __launch_bounds__(256)
state_scan_kernel(const float* __restrict__ qf, const float* __restrict__ kf, const float* __restrict__ vf,
                  const float* __restrict__ gf, const float* __restrict__ beta, float* __restrict__ o,
                  float* __restrict__ state, const int* __restrict__ cu_q, const int* __restrict__ prefix_len,
                  const int* __restrict__ state_slots, int heads, int kv_heads, int d, int dv) {
  constexpr int DP = DI * LS_LANES;                                  // d, rounded up to a multiple of 32
  constexpr int TOK = 3 * DP + LS_COLS + 4;                          // q, k, g, v, beta of one token
  extern __shared__ __align__(16) float smem[];                      // [2][LS_TOKENS][TOK]
  const int r = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * LS_COLS;
  const int hk = h / (heads / kv_heads);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int l = lane & (LS_LANES - 1);
  const int cj = warp * 4 + (lane >> 3);                             // column inside the tile
  const int col = col0 + cj;
  const bool col_ok = col < dv;
  const int first = cu_q[r], n = cu_q[r + 1] - first;
  float* st = state + (static_cast<size_t>(state_slots[r]) * heads + h) * d * dv;
  const bool has_past = prefix_len[r] > 0;

  float S[DI];
#pragma unroll
  for (int i = 0; i < DI; ++i) {
    const int e = (i >> 2) * 32 + l * 4 + (i & 3);
    S[i] = (has_past && col_ok && e < d) ? st[static_cast<size_t>(e) * dv + col] : 0.0f;
  }
  // columns of q, k and g beyond d stay zero in both buffers, and so do columns of v beyond dv
  for (int i = threadIdx.x; i < 2 * LS_TOKENS * TOK; i += blockDim.x) smem[i] = 0.0f;
  __syncthreads();
  const bool wide = d % 4 == 0 && dv % 4 == 0;                       // rows of whole 16-byte pieces
  auto fetch = [&](int base, int buf) {
    float* dst = smem + buf * LS_TOKENS * TOK;
    const int nt = min(LS_TOKENS, n - base);
    if (wide) {
      const int dq = d >> 2, vq = min(LS_COLS, dv - col0) >> 2;
      const int per = 3 * dq + vq;
      for (int idx = threadIdx.x; idx < nt * per; idx += blockDim.x) {
        const int tb = idx / per, p = idx - tb * per;
        const size_t t = first + base + tb;
        const float* src;
        float* to = dst + tb * TOK;
        if (p < dq) { src = qf + (t * kv_heads + hk) * d + 4 * p; to += 4 * p; }
        else if (p < 2 * dq) { src = kf + (t * kv_heads + hk) * d + 4 * (p - dq); to += DP + 4 * (p - dq); }
        else if (p < 3 * dq) { src = gf + (t * heads + h) * d + 4 * (p - 2 * dq); to += 2 * DP + 4 * (p - 2 * dq); }
        else { src = vf + (t * heads + h) * dv + col0 + 4 * (p - 3 * dq); to += 3 * DP + 4 * (p - 3 * dq); }
        cp_async16(to, src, true);
      }
    } else {
      const int vq = min(LS_COLS, dv - col0), per = 3 * d + vq;
      for (int idx = threadIdx.x; idx < nt * per; idx += blockDim.x) {
        const int tb = idx / per, p = idx - tb * per;
        const size_t t = first + base + tb;
        float* to = dst + tb * TOK;
        if (p < d) to[p] = qf[(t * kv_heads + hk) * d + p];
        else if (p < 2 * d) to[DP + p - d] = kf[(t * kv_heads + hk) * d + p - d];
        else if (p < 3 * d) to[2 * DP + p - 2 * d] = gf[(t * heads + h) * d + p - 2 * d];
        else to[3 * DP + p - 3 * d] = vf[(t * heads + h) * dv + col0 + p - 3 * d];
      }
    }
    if (DELTA && threadIdx.x < nt)
      dst[threadIdx.x * TOK + 3 * DP + LS_COLS] = beta[static_cast<size_t>(first + base + threadIdx.x) * heads + h];
    cp_async_commit();
  };
  auto over_lanes = [](float v) {
    v += __shfl_xor_sync(0xffffffffu, v, 1);
    v += __shfl_xor_sync(0xffffffffu, v, 2);
    v += __shfl_xor_sync(0xffffffffu, v, 4);
    return v;
  };
  if (n > 0) fetch(0, 0);
  for (int base = 0, buf = 0; base < n; base += LS_TOKENS, buf ^= 1) {
    if (base + LS_TOKENS < n) {
      fetch(base + LS_TOKENS, buf ^ 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const int nt = min(LS_TOKENS, n - base);
    const float* cur = smem + buf * LS_TOKENS * TOK;
    for (int tb = 0; tb < nt; ++tb) {
      const float* tk = cur + tb * TOK;
      const float4* q4 = reinterpret_cast<const float4*>(tk) + l;
      const float4* k4 = reinterpret_cast<const float4*>(tk + DP) + l;
      const float4* g4 = reinterpret_cast<const float4*>(tk + 2 * DP) + l;
      const float v = tk[3 * DP + cj];
      float acc[4] = {0.0f, 0.0f, 0.0f, 0.0f};
      if constexpr (DELTA) {
        float kk[DI];
        float dot[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
        for (int i = 0; i < DI / 4; ++i) {
          const float4 g = g4[8 * i], k = k4[8 * i];
          kk[4 * i] = k.x; kk[4 * i + 1] = k.y; kk[4 * i + 2] = k.z; kk[4 * i + 3] = k.w;
          S[4 * i] *= g.x; S[4 * i + 1] *= g.y; S[4 * i + 2] *= g.z; S[4 * i + 3] *= g.w;
          dot[0] = fmaf(S[4 * i], k.x, dot[0]); dot[1] = fmaf(S[4 * i + 1], k.y, dot[1]);
          dot[2] = fmaf(S[4 * i + 2], k.z, dot[2]); dot[3] = fmaf(S[4 * i + 3], k.w, dot[3]);
        }
        const float past = over_lanes((dot[0] + dot[1]) + (dot[2] + dot[3]));
        const float u = tk[3 * DP + LS_COLS] * (v - past);
#pragma unroll
        for (int i = 0; i < DI / 4; ++i) {
          const float4 q = q4[8 * i];
          S[4 * i] = fmaf(kk[4 * i], u, S[4 * i]); S[4 * i + 1] = fmaf(kk[4 * i + 1], u, S[4 * i + 1]);
          S[4 * i + 2] = fmaf(kk[4 * i + 2], u, S[4 * i + 2]); S[4 * i + 3] = fmaf(kk[4 * i + 3], u, S[4 * i + 3]);
          acc[0] = fmaf(S[4 * i], q.x, acc[0]); acc[1] = fmaf(S[4 * i + 1], q.y, acc[1]);
          acc[2] = fmaf(S[4 * i + 2], q.z, acc[2]); acc[3] = fmaf(S[4 * i + 3], q.w, acc[3]);
        }
      } else {
#pragma unroll
        for (int i = 0; i < DI / 4; ++i) {
          const float4 g = g4[8 * i], k = k4[8 * i], q = q4[8 * i];
          S[4 * i] = fmaf(g.x, S[4 * i], k.x * v); S[4 * i + 1] = fmaf(g.y, S[4 * i + 1], k.y * v);
          S[4 * i + 2] = fmaf(g.z, S[4 * i + 2], k.z * v); S[4 * i + 3] = fmaf(g.w, S[4 * i + 3], k.w * v);
          acc[0] = fmaf(S[4 * i], q.x, acc[0]); acc[1] = fmaf(S[4 * i + 1], q.y, acc[1]);
          acc[2] = fmaf(S[4 * i + 2], q.z, acc[2]); acc[3] = fmaf(S[4 * i + 3], q.w, acc[3]);
        }
      }
      const float out = over_lanes((acc[0] + acc[1]) + (acc[2] + acc[3]));
      if (l == 0 && col_ok) o[(static_cast<size_t>(first + base + tb) * heads + h) * dv + col] = out;
    }
    __syncthreads();                                                 // the buffer may be filled again
  }
  if (col_ok) {
#pragma unroll
    for (int i = 0; i < DI; ++i) {
      const int e = (i >> 2) * 32 + l * 4 + (i & 3);
      if (e < d) st[static_cast<size_t>(e) * dv + col] = S[i];
    }
  }
}

template <int DI>
static int launch_state_scan(const float* qf, const float* kf, const float* vf, const float* gf, const float* beta, float* o,
                             float* state, const int* cu_q, const int* prefix_len, const int* state_slots, int num_rows,
                             int heads, int kv_heads, int d, int dv, cudaStream_t stream) {
  const size_t smem = 2 * LS_TOKENS * (3 * DI * LS_LANES + LS_COLS + 4) * sizeof(float);
  const dim3 grid(num_rows, heads, (dv + LS_COLS - 1) / LS_COLS);
  auto kernel = beta != nullptr ? state_scan_kernel<DI, true> : state_scan_kernel<DI, false>;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return static_cast<int>(e);
  }
  kernel<<<grid, 256, smem, stream>>>(qf, kf, vf, gf, beta, o, state, cu_q, prefix_len, state_slots, heads, kv_heads, d, dv);
  return b200_check_launch();
}

// ------------------------------------------------------------------ a step whose rows bring one token each
// grid (rows, heads).  Thread (rg, cg): four neighbouring columns 4 cg .. of the state on the rows rg, rg + RG, ...
// The state is the kernel's traffic (d * dv floats in and out); everything else about the token (convolution,
// activation, unit vectors, the two low-rank products behind decay and gate, norm, gate) is computed in between.
//   decay pre-activation   z_e = a2[h d + e] . x[a_column ..] (rank a_rank), float sums over the rounded row
//   gate                   kind 0: sigmoid(g2[h dv + e] . x[g_column ..]) (rank g_rank);  kind 1: silu(x[g_column + h dv + e])
//   out[t][h dv + e] = o / sqrt(mean(o^2) + eps) * norm_w[e] * gate,   rounded once
struct StateDecodeParams {
  const void *a2, *g2;
  int a_column, a_rank, g_column, g_rank, gate_kind;
  const float* norm_w;
  float eps;
  int own_conv;                // every channel has one reader (as many q/k heads as heads): it brings the row's convolution
                               // state up to date itself
};

template <typename T>
__device__ __forceinline__ float low_rank_dot(const T* __restrict__ w, const float* __restrict__ v, int rank) {
  float s = 0.0f;
  if (rank % 8 == 0) {
    for (int k = 0; k < rank; k += 8) {
      float a[8];
      load_floats<T, 8>(w + k, a);
#pragma unroll
      for (int j = 0; j < 8; ++j) s = fmaf(a[j], v[k + j], s);
    }
  } else {
    for (int k = 0; k < rank; ++k) s = fmaf(to_f32<T>(w[k]), v[k], s);
  }
  return s;
}

template <typename T, int MAXR, bool DELTA, int THREADS>
__global__ void __launch_bounds__(THREADS, THREADS == 256 ? 2 : 1)
state_decode_kernel(TapsInput<T> in, LinearStateShape s, StateDecodeParams p, T* __restrict__ out, float* __restrict__ state) {
  pdl_launch_dependents();                          // the kernel after this one may be scheduled; it waits before it reads
  extern __shared__ __align__(16) float smem[];
  __shared__ float scratch[33];
  const int t = blockIdx.x, h = blockIdx.y;         // a row has one token: row number = token number
  const int d = s.d, dv = s.dv;
  const int hk = h / (s.heads / s.kv_heads);
  float* q = smem;                                  // [d]
  float* k = q + d;                                 // [d]
  float* g = k + d;                                 // [d]
  float* v = g + d;                                 // [dv]
  float* gate = v + dv;                             // [dv]
  float* low = gate + dv;                           // [a_rank + g_rank]
  const int CG = dv >> 2, RG = THREADS / CG;
  float* part = low + ((p.a_rank + p.g_rank + 3) & ~3);   // [RG][dv] (16-byte aligned: d and dv are multiples of 4)
  const int rg = threadIdx.x / CG, cg = threadIdx.x - rg * CG;
  pdl_wait();                                        // what this kernel reads belongs to the kernels before it
  const T* xr = in.x + static_cast<size_t>(t) * in.in_stride;
  const bool has_past = in.prefix_len[t] > 0;
  float* st = state + (static_cast<size_t>(in.state_slots[t]) * s.heads + h) * d * dv;
  // the state, on its way while the token's inputs are computed
  float4 S[MAXR];
#pragma unroll
  for (int i = 0; i < MAXR; ++i) {
    const int e = rg + i * RG;
    S[i] = (has_past && rg < RG && e < d) ? *reinterpret_cast<const float4*>(st + static_cast<size_t>(e) * dv + 4 * cg)
                                          : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  }
  for (int i = threadIdx.x; i < p.a_rank + (p.gate_kind == 0 ? p.g_rank : 0); i += blockDim.x)
    low[i] = to_f32<T>(xr[i < p.a_rank ? p.a_column + i : p.g_column + i - p.a_rank]);
  TapsRow row = {};
  const bool conv = in.w != nullptr;
  if (conv) row = taps_row(in, t);
  auto value = [&](int c) {
    float y = conv ? taps_value(in, row, t, c, false) : to_f32<T>(xr[c]);
    if (p.own_conv && in.taps > 1) {                 // this thread is the channel's only reader and has read it
      float* past = in.state + static_cast<size_t>(in.state_slots[t]) * (in.taps - 1) * in.channels + c;
      for (int j = 0; j + 2 < in.taps; ++j) past[static_cast<size_t>(j) * in.channels] = has_past ? past[static_cast<size_t>(j + 1) * in.channels] : 0.0f;
      past[static_cast<size_t>(in.taps - 2) * in.channels] = to_f32<T>(xr[c]);
    }
    if (s.silu) y = silu_of(y);
    return y;
  };
  float qq = 0.0f, kk = 0.0f;
  for (int i = threadIdx.x; i < 2 * d + dv; i += blockDim.x) {
    if (i < d) {
      const float y = value(hk * d + i);
      q[i] = y;
      qq = fmaf(y, y, qq);
    } else if (i < 2 * d) {
      const float y = value((s.kv_heads + hk) * d + i - d);
      k[i - d] = y;
      kk = fmaf(y, y, kk);
    } else {
      v[i - 2 * d] = value(2 * s.kv_heads * d + h * dv + i - 2 * d);
    }
  }
  float qn = s.q_scale, kn = 1.0f;
  if (s.unit_eps > 0.0f) {
    qn *= 1.0f / sqrtf(block_sum(qq, scratch) + s.unit_eps);
    kn = 1.0f / sqrtf(block_sum(kk, scratch) + s.unit_eps);
  }
  __syncthreads();
  const float rate = s.decay_kind == DECAY_SOFTPLUS ? expf(s.a_log[h]) : 0.0f;
  for (int i = threadIdx.x; i < d + dv; i += blockDim.x) {
    if (i < d) {
      const float b = s.decay_bias != nullptr ? s.decay_bias[h * d + i] : 0.0f;
      const float z = low_rank_dot<T>(static_cast<const T*>(p.a2) + static_cast<size_t>(h * d + i) * p.a_rank, low, p.a_rank);
      g[i] = decay_of(z + b, s, rate);
      q[i] *= qn;
      k[i] *= kn;
    } else {
      const int e = i - d;
      if (p.gate_kind == 0)
        gate[e] = sigmoid_of(low_rank_dot<T>(static_cast<const T*>(p.g2) + static_cast<size_t>(h * dv + e) * p.g_rank,
                                             low + p.a_rank, p.g_rank));
      else
        gate[e] = silu_of(to_f32<T>(xr[p.g_column + h * dv + e]));
    }
  }
  __syncthreads();
  float4 u = rg < RG ? *reinterpret_cast<const float4*>(v + 4 * cg) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  if constexpr (DELTA) {
    float4 dot = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
    for (int i = 0; i < MAXR; ++i) {
      const int e = rg + i * RG;
      if (rg < RG && e < d) {
        const float ge = g[e], ke = k[e];
        S[i].x *= ge; S[i].y *= ge; S[i].z *= ge; S[i].w *= ge;
        dot.x = fmaf(S[i].x, ke, dot.x); dot.y = fmaf(S[i].y, ke, dot.y);
        dot.z = fmaf(S[i].z, ke, dot.z); dot.w = fmaf(S[i].w, ke, dot.w);
      }
    }
    if (rg < RG) *reinterpret_cast<float4*>(part + rg * dv + 4 * cg) = dot;
    __syncthreads();
    if (rg < RG) {
      float4 past = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
      for (int i = 0; i < RG; ++i) {
        const float4 a = *reinterpret_cast<const float4*>(part + i * dv + 4 * cg);
        past.x += a.x; past.y += a.y; past.z += a.z; past.w += a.w;
      }
      const float b = sigmoid_of(to_f32<T>(xr[s.beta_column + h]));
      u = make_float4(b * (u.x - past.x), b * (u.y - past.y), b * (u.z - past.z), b * (u.w - past.w));
    }
    __syncthreads();                                 // `part` is free again
  }
  float4 acc = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
  for (int i = 0; i < MAXR; ++i) {
    const int e = rg + i * RG;
    if (rg < RG && e < d) {
      const float ke = k[e], qe = q[e];
      if constexpr (DELTA) {
        S[i].x = fmaf(ke, u.x, S[i].x); S[i].y = fmaf(ke, u.y, S[i].y);
        S[i].z = fmaf(ke, u.z, S[i].z); S[i].w = fmaf(ke, u.w, S[i].w);
      } else {
        const float ge = g[e];
        S[i].x = fmaf(ge, S[i].x, ke * u.x); S[i].y = fmaf(ge, S[i].y, ke * u.y);
        S[i].z = fmaf(ge, S[i].z, ke * u.z); S[i].w = fmaf(ge, S[i].w, ke * u.w);
      }
      acc.x = fmaf(S[i].x, qe, acc.x); acc.y = fmaf(S[i].y, qe, acc.y);
      acc.z = fmaf(S[i].z, qe, acc.z); acc.w = fmaf(S[i].w, qe, acc.w);
      *reinterpret_cast<float4*>(st + static_cast<size_t>(e) * dv + 4 * cg) = S[i];
    }
  }
  if (rg < RG) *reinterpret_cast<float4*>(part + rg * dv + 4 * cg) = acc;
  __syncthreads();
  float ss = 0.0f;
  for (int e = threadIdx.x; e < dv; e += blockDim.x) {
    float y = 0.0f;
    for (int i = 0; i < RG; ++i) y += part[i * dv + e];
    v[e] = y;                                        // o of this head
    ss = fmaf(y, y, ss);
  }
  ss = block_sum(ss, scratch);
  const float f = 1.0f / sqrtf(ss / static_cast<float>(dv) + p.eps);
  for (int e = threadIdx.x; e < dv; e += blockDim.x)
    out[static_cast<size_t>(t) * s.heads * dv + h * dv + e] = from_f32<T>(v[e] * f * p.norm_w[e] * gate[e]);
}

// ------------------------------------------------------------------ C interface
template <typename T>
static TapsInput<T> conv_input(const void* x, int in_stride, const float* conv_w, int taps, int channels, float* conv_state,
                               const int* row_of_token, const int* cu_q, const int* prefix_len, const int* state_slots) {
  TapsInput<T> in = {};
  in.x = static_cast<const T*>(x);
  in.in_stride = in_stride;
  in.w = conv_w;
  in.taps = taps;
  in.channels = channels;
  in.state = conv_state;
  in.row_of_token = row_of_token;
  in.cu_q = cu_q;
  in.prefix_len = prefix_len;
  in.state_slots = state_slots;
  return in;
}

static bool shape_ok(const LinearStateShape& s) {
  return s.heads > 0 && s.heads <= 65535 && s.kv_heads > 0 && s.heads % s.kv_heads == 0 && s.d > 0 && s.d <= 512 && s.dv > 0 &&
         (s.dv + LS_COLS - 1) / LS_COLS <= 65535 && (s.decay_kind == DECAY_LOGISTIC || (s.decay_kind == DECAY_SOFTPLUS && s.a_log != nullptr));
}

B200_EXPORT int b200_linear_state_shape_size() { return static_cast<int>(sizeof(LinearStateShape)); }
B200_EXPORT int b200_state_decode_params_size() { return static_cast<int>(sizeof(StateDecodeParams)); }

// x [tokens, in_stride]: q, k, v side by side from column 0 (and the beta columns); conv_w [channels of q, k, v; taps]
// or null; z [tokens, heads * d] float.
B200_EXPORT int b200_state_prepare(const void* x, int dtype, int in_stride, const float* conv_w, int taps, float* conv_state,
                                   const int* row_of_token, const int* cu_q, const int* prefix_len, const int* state_slots,
                                   const LinearStateShape* shape, const float* z, float* qf, float* kf, float* vf, float* gf,
                                   float* beta, int tokens, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  const LinearStateShape s = *shape;
  const int channels = 2 * s.kv_heads * s.d + s.heads * s.dv;
  if (!shape_ok(s) || in_stride < channels || taps > TAPS_MAX || (conv_w != nullptr && taps > 1 && conv_state == nullptr))
    return B200_BAD_SIZE;
  const dim3 grid(tokens, (2 * s.kv_heads + 2 * s.heads + LS_PREP_WARPS - 1) / LS_PREP_WARPS);
  if (grid.y > 65535) return B200_BAD_SIZE;
  if (dtype == B200_F32)
    state_prepare_kernel<float><<<grid, LS_PREP_WARPS * 32, 0, stream>>>(
        conv_input<float>(x, in_stride, conv_w, taps, channels, conv_state, row_of_token, cu_q, prefix_len, state_slots), s,
        z, qf, kf, vf, gf, beta);
  else if (dtype == B200_BF16)
    state_prepare_kernel<__nv_bfloat16><<<grid, LS_PREP_WARPS * 32, 0, stream>>>(
        conv_input<__nv_bfloat16>(x, in_stride, conv_w, taps, channels, conv_state, row_of_token, cu_q, prefix_len, state_slots),
        s, z, qf, kf, vf, gf, beta);
  else
    return B200_BAD_DTYPE;
  return b200_check_launch();
}

// beta null: without the delta rule.
B200_EXPORT int b200_state_scan(const float* qf, const float* kf, const float* vf, const float* gf, const float* beta, float* o,
                                float* state, const int* cu_q, const int* prefix_len, const int* state_slots, int num_rows,
                                int heads, int kv_heads, int d, int dv, cudaStream_t stream) {
  if (num_rows <= 0) return 0;
  if (heads <= 0 || heads > 65535 || kv_heads <= 0 || heads % kv_heads || d <= 0 || d > 512 || dv <= 0 ||
      (dv + LS_COLS - 1) / LS_COLS > 65535)
    return B200_BAD_SIZE;
  const int blocks = (d + 31) / 32;
#define LS_CASE(N)                                                                                                    \
  if (blocks <= N)                                                                                                    \
    return launch_state_scan<4 * N>(qf, kf, vf, gf, beta, o, state, cu_q, prefix_len, state_slots, num_rows, heads,   \
                                    kv_heads, d, dv, stream)
  LS_CASE(1);
  LS_CASE(2);
  LS_CASE(3);
  LS_CASE(4);
  LS_CASE(6);
  LS_CASE(8);
  LS_CASE(16);
#undef LS_CASE
  return B200_BAD_SIZE;
}

template <typename T, int MAXR, int THREADS>
static int launch_state_decode(const TapsInput<T>& in, const LinearStateShape& s, const StateDecodeParams& p, void* out,
                               float* state, int rows, size_t smem, cudaStream_t stream) {
  auto kernel = s.beta_column >= 0 ? state_decode_kernel<T, MAXR, true, THREADS> : state_decode_kernel<T, MAXR, false, THREADS>;
  return b200_launch(kernel, dim3(rows, s.heads), dim3(THREADS), smem, stream, 0, in, s, p, static_cast<T*>(out), state);
}

// Rows of one token each (token t is row t).  B200_BAD_SIZE: the sizes do not fit this kernel (dv a multiple of 4, at
// most 20 rows of the state a thread); the caller takes the other two.  Without own_conv the rows' convolution states are
// NOT brought up to date here (a channel of q or k is read by several heads): a kernel behind this one does that.
B200_EXPORT int b200_state_decode(const void* x, int dtype, int in_stride, const float* conv_w, int taps, float* conv_state,
                                  const int* row_of_token, const int* cu_q, const int* prefix_len, const int* state_slots,
                                  const LinearStateShape* shape, const StateDecodeParams* params, void* out, float* state,
                                  int rows, cudaStream_t stream) {
  if (rows <= 0) return 0;
  const LinearStateShape s = *shape;
  const StateDecodeParams p = *params;
  const int channels = 2 * s.kv_heads * s.d + s.heads * s.dv;
  if (!shape_ok(s) || in_stride < channels || taps > TAPS_MAX || (conv_w != nullptr && taps > 1 && conv_state == nullptr) ||
      s.dv % 4 != 0 || s.d % 4 != 0 || s.dv > 1024 || (p.own_conv && s.heads != s.kv_heads) || p.a_rank < 0 || p.g_rank < 0 || reinterpret_cast<uintptr_t>(state) % 16 != 0)
    return B200_BAD_SIZE;
  const int cg = s.dv / 4;
  int threads = 256;
  if (cg > threads || (s.d + threads / cg - 1) / (threads / cg) > 16) threads = 512;
  if (cg > threads) return B200_BAD_SIZE;
  const int rg = threads / cg, per = (s.d + rg - 1) / rg;
  const size_t smem = (3 * static_cast<size_t>(s.d) + 2 * s.dv + ((p.a_rank + p.g_rank + 3) & ~3) + static_cast<size_t>(rg) * s.dv) * sizeof(float);
  if (per > 20 || smem > 48 * 1024) return B200_BAD_SIZE;
#define LS_DECODE(T)                                                                                                    \
  do {                                                                                                                  \
    const TapsInput<T> in = conv_input<T>(x, in_stride, conv_w, taps, channels, conv_state, row_of_token, cu_q, prefix_len, \
                                          state_slots);                                                                 \
    if (threads == 512) return launch_state_decode<T, 20, 512>(in, s, p, out, state, rows, smem, stream);               \
    if (per <= 4) return launch_state_decode<T, 4, 256>(in, s, p, out, state, rows, smem, stream);                      \
    if (per <= 8) return launch_state_decode<T, 8, 256>(in, s, p, out, state, rows, smem, stream);                      \
    return launch_state_decode<T, 16, 256>(in, s, p, out, state, rows, smem, stream);                                   \
  } while (0)
  if (dtype == B200_F32) LS_DECODE(float);
  if (dtype == B200_BF16) LS_DECODE(__nv_bfloat16);
#undef LS_DECODE
  return B200_BAD_DTYPE;
}
