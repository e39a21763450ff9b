// Linear attention whose state decays per key channel or per head, with or without the delta rule, the state of every
// request in float32.  Per head, with S [d, dv] and the decay g [d] of a token acting on the rows of S (one number a head:
// the same g for every row):
//
//   plain   S <- diag(g) S + k v^T                                                             o = S^T q
//   delta   S <- diag(g) S;   u = beta (v - S^T k);   S <- S + k u^T                           o = S^T q
//
// What enters it comes out of a packed projection row x (q heads, k heads, v heads, then whatever else):
//   q, k, v   optionally through a short causal convolution over time (its last inputs are per-request state) and an
//             activation; q and k optionally made unit vectors (x / sqrt(sum x^2 + eps)); q times q_scale
//   g         from z [heads * d] (float) and a bias:   LOGISTIC  sigmoid(z + bias)^(1 / tau)
//                                                     SOFTPLUS  exp(-exp(a_log_h) softplus(z + bias))
//             with one decay a head: z is a column of x a head (decay_column) and the bias has one entry a head
//   beta      sigmoid of one column a head of x
// heads may be a multiple of the q/k heads: head h uses q and k of head h / (heads / kv_heads).
//
//   state_prepare   the four inputs of every token in float (qf, kf [tokens, kv_heads * d], vf [tokens, heads * dv],
//                   gf [tokens, heads * d] (one decay a head: [tokens, heads]), beta [tokens, heads])
//   state_scan      (state_scan.cu) the recurrence, token by token in the sequence's order whatever the step's cut
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
  int decay_column;            // column of x with one pre-activation a head, or -1: one a key channel (z)
  float inv_tau;               // LOGISTIC
  const float* decay_bias;     // [heads * d] ([heads] with decay_column) or null
  const float* a_log;          // [heads], SOFTPLUS
};

__device__ __forceinline__ float silu_of(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float sigmoid_of(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_of(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }

// The decay of one key channel from its pre-activation (bias included) and exp(a_log) of its head.
__device__ __forceinline__ float decay_of(float z, const LinearStateShape& s, float rate) {
  return s.decay_kind == DECAY_LOGISTIC ? expf(-softplus_of(-z) * s.inv_tau) : expf(-rate * softplus_of(z));
}

// The decay of head h where there is one a head; xr: the token's packed row.
template <typename T>
__device__ __forceinline__ float head_decay(const T* __restrict__ xr, const LinearStateShape& s, int h, float rate) {
  const float b = s.decay_bias != nullptr ? s.decay_bias[h] : 0.0f;
  return decay_of(to_f32<T>(xr[s.decay_column + h]) + b, s, rate);
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
    if (s.decay_column >= 0) {
      if (lane == 0) gf[static_cast<size_t>(t) * s.heads + h] = head_decay<T>(xr, s, h, rate);
    } else {
      const size_t base = static_cast<size_t>(t) * s.heads * s.d + static_cast<size_t>(h) * s.d;
      for (int e = lane; e < s.d; e += 32) {
        const float b = s.decay_bias != nullptr ? s.decay_bias[h * s.d + e] : 0.0f;
        gf[base + e] = decay_of(z[base + e] + b, s, rate);
      }
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

// The same with four channels a thread and LS_PREP_TOKENS consecutive tokens a warp, for head sizes and rows of whole
// 16-byte pieces (d a multiple of 4 up to 128): a channel's taps stay in registers and its last inputs move along with the
// tokens, so that a token costs one load of its projection.  grid (token groups, units / 4).
constexpr int LS_PREP_TOKENS = 8;

template <typename T, int TAPS>            // TAPS 0: no convolution
__global__ void __launch_bounds__(LS_PREP_WARPS * 32)
state_prepare_vec_kernel(TapsInput<T> in, LinearStateShape s, const float* __restrict__ z, float* __restrict__ qf,
                         float* __restrict__ kf, float* __restrict__ vf, float* __restrict__ gf, float* __restrict__ beta,
                         int tokens) {
  const int t0 = blockIdx.x * LS_PREP_TOKENS, t1 = min(t0 + LS_PREP_TOKENS, tokens);
  const int lane = threadIdx.x & 31;
  const int unit = blockIdx.y * LS_PREP_WARPS + (threadIdx.x >> 5);
  if (unit >= 2 * s.kv_heads + 2 * s.heads) return;
  if (unit >= 2 * s.kv_heads + s.heads) {                            // a head's decays
    const int h = unit - 2 * s.kv_heads - s.heads;
    const float rate = s.decay_kind == DECAY_SOFTPLUS ? expf(s.a_log[h]) : 0.0f;
    const int e = 4 * lane;
    if (s.decay_column >= 0) {
      if (t0 + lane < t1)
        gf[static_cast<size_t>(t0 + lane) * s.heads + h] =
            head_decay<T>(in.x + static_cast<size_t>(t0 + lane) * in.in_stride, s, h, rate);
    } else if (e < s.d) {
      float4 b = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
      if (s.decay_bias != nullptr) b = *reinterpret_cast<const float4*>(s.decay_bias + h * s.d + e);
#pragma unroll 4
      for (int t = t0; t < t1; ++t) {
        const size_t at = static_cast<size_t>(t) * s.heads * s.d + h * s.d + e;
        const float4 v = *reinterpret_cast<const float4*>(z + at);
        *reinterpret_cast<float4*>(gf + at) = make_float4(decay_of(v.x + b.x, s, rate), decay_of(v.y + b.y, s, rate),
                                                          decay_of(v.z + b.z, s, rate), decay_of(v.w + b.w, s, rate));
      }
    }
    if (s.beta_column >= 0 && t0 + lane < t1)
      beta[static_cast<size_t>(t0 + lane) * s.heads + h] =
          sigmoid_of(to_f32<T>(in.x[static_cast<size_t>(t0 + lane) * in.in_stride + s.beta_column + h]));
    return;
  }
  const bool is_v = unit >= 2 * s.kv_heads, is_k = !is_v && unit >= s.kv_heads;
  const int h = is_v ? unit - 2 * s.kv_heads : is_k ? unit - s.kv_heads : unit;
  const int size = is_v ? s.dv : s.d;
  const int c0 = is_v ? 2 * s.kv_heads * s.d + h * s.dv : (is_k ? s.kv_heads * s.d : 0) + h * s.d;
  const int out_stride = is_v ? s.heads * s.dv : s.kv_heads * s.d;
  float* out = (is_v ? vf : is_k ? kf : qf) + static_cast<size_t>(h) * size;
  const bool unit_norm = !is_v && s.unit_eps > 0.0f;
  const float f = (is_v || is_k) ? 1.0f : s.q_scale;
  constexpr int HIST = TAPS > 1 ? TAPS - 1 : 0;
  for (int e0 = 0; e0 < size; e0 += 128) {                           // (once for q and k)
    const int e = e0 + 4 * lane;
    const bool on = e < size;
    const int c = c0 + (on ? e : 0);
    float w[4][TAPS > 0 ? TAPS : 1];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < TAPS; ++j) w[i][j] = in.w[static_cast<size_t>(c + i) * TAPS + j];
    float past[HIST > 0 ? HIST : 1][4];                              // oldest first
    for (int t = t0; t < t1; ++t) {
      if constexpr (HIST > 0) {
        const int r = in.row_of_token[t];
        if (t == t0 || t == in.cu_q[r]) {                            // the inputs before this token, from x, the state or nowhere
          const TapsRow row = taps_row(in, t);
#pragma unroll
          for (int j = 0; j < HIST; ++j)
#pragma unroll
            for (int i = 0; i < 4; ++i) past[j][i] = taps_past(in, row, t, c + i, HIST - j);
        }
      }
      float now[4], y[4];
      load_floats<T, 4>(in.x + static_cast<size_t>(t) * in.in_stride + c, now);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        if constexpr (TAPS > 0) {
          y[i] = 0.0f;
#pragma unroll
          for (int j = 0; j < HIST; ++j) y[i] = fmaf(w[i][j], past[j][i], y[i]);
          y[i] = fmaf(w[i][TAPS - 1], now[i], y[i]);
        } else {
          y[i] = now[i];
        }
        if (s.silu) y[i] = silu_of(y[i]);
      }
      if constexpr (HIST > 0) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
#pragma unroll
          for (int j = 0; j + 1 < HIST; ++j) past[j][i] = past[j + 1][i];
          past[HIST - 1][i] = now[i];
        }
      }
      float g = f;
      if (unit_norm) {
        float ss = 0.0f;
#pragma unroll
        for (int i = 0; i < 4; ++i) ss = on ? fmaf(y[i], y[i], ss) : 0.0f;
        g *= 1.0f / sqrtf(warp_sum(ss) + s.unit_eps);
      }
      if (on)
        *reinterpret_cast<float4*>(out + static_cast<size_t>(t) * out_stride + e) = make_float4(y[0] * g, y[1] * g, y[2] * g, y[3] * g);
    }
  }
}

// ------------------------------------------------------------------ a step whose rows bring one token each
// grid (rows, heads).  Thread (rg, cg): four neighbouring columns 4 cg .. of the state on the rows rg, rg + RG, ...
// The state is the kernel's traffic (d * dv floats in and out); everything else about the token (convolution,
// activation, unit vectors, the two low-rank products behind decay and gate, norm, gate) is computed in between.
//   decay pre-activation   z_e = a2[h d + e] . x[a_column ..] (rank a_rank), float sums over the rounded row
//                          (with decay_column: one decay a head, a_rank 0)
//   gate                   kind 0: sigmoid(g2[h dv + e] . x[g_column ..]) (rank g_rank);  kind 1: silu(x[g_column + h dv + e])
//   out[t][h dv + e] = o / sqrt(mean(o^2) + eps) * norm_w[e] * gate,   rounded once
// The launch may overlap the tail of the kernel before it (the packed projection).  What the kernel fetches before it
// waits for that one is not written by this step's kernels: weights, the step's index arrays, and the states that the
// step before left, which ended before this step's first kernel began (a step begins with a kernel, the embedding, that
// does not overlap what is before it).
struct StateDecodeParams {
  const void *a2, *g2;
  int a_column, a_rank, g_column, g_rank, gate_kind;
  const float* norm_w;
  float eps;
  int own_conv;                // every channel has one reader (as many q/k heads as heads): it brings the row's convolution
                               // state up to date itself
  int stage;                   // the head's rows of a2 and g2 go through shared memory (ranks of whole 16-byte pieces)
};

// w . v over `rank` elements, eight at a time where a row is whole 16-byte pieces
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

// Bytes of shared memory that a staged row takes: 16 more than its own, so that neighbouring rows begin in other banks.
template <typename T>
__host__ __device__ constexpr int staged_row(int rank) { return rank * static_cast<int>(sizeof(T)) + 16; }

template <typename T, int MAXR, bool DELTA, int THREADS>
__global__ void __launch_bounds__(THREADS, THREADS == 256 ? 2 : 1)
state_decode_kernel(TapsInput<T> in, LinearStateShape s, StateDecodeParams p, T* __restrict__ out, float* __restrict__ state) {
  pdl_launch_dependents();                          // the kernel after this one may be scheduled; it waits before it reads
  extern __shared__ __align__(16) float smem[];
  __shared__ float sums[2][THREADS / 32];
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
  char* rows_a = reinterpret_cast<char*>(part + RG * dv);
  char* rows_g = rows_a + d * staged_row<T>(p.a_rank);
  const int rg = threadIdx.x / CG, cg = threadIdx.x - rg * CG;
  const int slot = in.state_slots[t];
  const bool has_past = in.prefix_len[t] > 0;
  const T* a2 = static_cast<const T*>(p.a2) + static_cast<size_t>(h) * d * p.a_rank;
  const T* g2 = static_cast<const T*>(p.g2) + static_cast<size_t>(h) * dv * p.g_rank;
  float* st = state + (static_cast<size_t>(slot) * s.heads + h) * d * dv;
  float4 S[MAXR];
#pragma unroll
  for (int i = 0; i < MAXR; ++i) {
    const int e = rg + i * RG;
    S[i] = (has_past && rg < RG && e < d) ? *reinterpret_cast<const float4*>(st + static_cast<size_t>(e) * dv + 4 * cg)
                                          : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  }
  if (p.stage) {
    const int pa = p.a_rank * sizeof(T) / 16, pg = p.gate_kind == 0 ? p.g_rank * static_cast<int>(sizeof(T)) / 16 : 0;
    for (int i = threadIdx.x; i < d * pa; i += THREADS) {
      const int e = i / pa, c = i - e * pa;
      cp_async16(rows_a + e * staged_row<T>(p.a_rank) + 16 * c, reinterpret_cast<const char*>(a2) + 16 * static_cast<size_t>(i), true);
    }
    for (int i = threadIdx.x; i < dv * pg; i += THREADS) {
      const int e = i / pg, c = i - e * pg;
      cp_async16(rows_g + e * staged_row<T>(p.g_rank) + 16 * c, reinterpret_cast<const char*>(g2) + 16 * static_cast<size_t>(i), true);
    }
    cp_async_commit();
  }
  pdl_wait();                                        // the packed projection comes from the kernel before
  const T* xr = in.x + static_cast<size_t>(t) * in.in_stride;
  for (int i = threadIdx.x; i < p.a_rank + (p.gate_kind == 0 ? p.g_rank : 0); i += THREADS)
    low[i] = to_f32<T>(xr[i < p.a_rank ? p.a_column + i : p.g_column + i - p.a_rank]);
  TapsRow row;
  row.local = 0;
  row.has_past = has_past;
  row.state = in.w != nullptr ? in.state + static_cast<size_t>(slot) * (in.taps - 1) * in.channels : nullptr;
  const bool conv = in.w != nullptr;
  auto value = [&](int c) {
    float y = conv ? taps_value(in, row, t, c, false) : to_f32<T>(xr[c]);
    if (p.own_conv && in.taps > 1) {                 // this thread is the channel's only reader and has read it
      float* past = in.state + static_cast<size_t>(slot) * (in.taps - 1) * in.channels + c;
      for (int j = 0; j + 2 < in.taps; ++j) past[static_cast<size_t>(j) * in.channels] = has_past ? past[static_cast<size_t>(j + 1) * in.channels] : 0.0f;
      past[static_cast<size_t>(in.taps - 2) * in.channels] = to_f32<T>(xr[c]);
    }
    if (s.silu) y = silu_of(y);
    return y;
  };
  float qq = 0.0f, kk = 0.0f;
#pragma unroll 2
  for (int i = threadIdx.x; i < 2 * d + dv; i += THREADS) {
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
  qq = warp_sum(qq);
  kk = warp_sum(kk);
  if ((threadIdx.x & 31) == 0) { sums[0][threadIdx.x >> 5] = qq; sums[1][threadIdx.x >> 5] = kk; }
  if (p.stage) cp_async_wait<0>();
  __syncthreads();
  float qn = s.q_scale, kn = 1.0f;
  if (s.unit_eps > 0.0f) {
    qq = kk = 0.0f;
#pragma unroll
    for (int w = 0; w < THREADS / 32; ++w) { qq += sums[0][w]; kk += sums[1][w]; }
    qn *= 1.0f / sqrtf(qq + s.unit_eps);
    kn = 1.0f / sqrtf(kk + s.unit_eps);
  }
  const float rate = s.decay_kind == DECAY_SOFTPLUS ? expf(s.a_log[h]) : 0.0f;
  const float whole = s.decay_column >= 0 ? head_decay<T>(xr, s, h, rate) : 0.0f;
  for (int i = threadIdx.x; i < d + dv; i += THREADS) {
    if (i < d && s.decay_column >= 0) {
      g[i] = whole;
      q[i] *= qn;
      k[i] *= kn;
    } else if (i < d) {
      const float b = s.decay_bias != nullptr ? s.decay_bias[h * d + i] : 0.0f;
      const T* w = p.stage ? reinterpret_cast<const T*>(rows_a + i * staged_row<T>(p.a_rank)) : a2 + static_cast<size_t>(i) * p.a_rank;
      g[i] = decay_of(low_rank_dot<T>(w, low, p.a_rank) + b, s, rate);
      q[i] *= qn;
      k[i] *= kn;
    } else {
      const int e = i - d;
      if (p.gate_kind == 0) {
        const T* w = p.stage ? reinterpret_cast<const T*>(rows_g + e * staged_row<T>(p.g_rank)) : g2 + static_cast<size_t>(e) * p.g_rank;
        gate[e] = sigmoid_of(low_rank_dot<T>(w, low + p.a_rank, p.g_rank)) * p.norm_w[e];
      } else {
        gate[e] = silu_of(to_f32<T>(xr[p.g_column + h * dv + e])) * p.norm_w[e];
      }
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
    out[static_cast<size_t>(t) * s.heads * dv + h * dv + e] = from_f32<T>(v[e] * f * gate[e]);
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
         (s.dv + 15) / 16 <= 65535 && (s.decay_kind == DECAY_LOGISTIC || (s.decay_kind == DECAY_SOFTPLUS && s.a_log != nullptr));
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
  const bool vec = s.d % 4 == 0 && s.d <= 128 && s.dv % 4 == 0 && in_stride % 8 == 0 && reinterpret_cast<uintptr_t>(x) % 16 == 0 &&
                   (conv_w == nullptr || taps <= 4);
  if (vec) {
    const dim3 vgrid((tokens + LS_PREP_TOKENS - 1) / LS_PREP_TOKENS, grid.y);
#define LS_PREP(T, N)                                                                                                    \
  state_prepare_vec_kernel<T, N><<<vgrid, LS_PREP_WARPS * 32, 0, stream>>>(                                               \
      conv_input<T>(x, in_stride, conv_w, taps, channels, conv_state, row_of_token, cu_q, prefix_len, state_slots), s, z, \
      qf, kf, vf, gf, beta, tokens)
#define LS_PREP_TAPS(T)                          \
  do {                                           \
    switch (conv_w == nullptr ? 0 : taps) {      \
      case 0: LS_PREP(T, 0); break;              \
      case 1: LS_PREP(T, 1); break;              \
      case 2: LS_PREP(T, 2); break;              \
      case 3: LS_PREP(T, 3); break;              \
      default: LS_PREP(T, 4); break;             \
    }                                            \
  } while (0)
    if (dtype == B200_F32) LS_PREP_TAPS(float);
    else if (dtype == B200_BF16) LS_PREP_TAPS(__nv_bfloat16);
    else return B200_BAD_DTYPE;
#undef LS_PREP_TAPS
#undef LS_PREP
    return b200_check_launch();
  }
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

template <typename T, int MAXR, int THREADS>
static int launch_state_decode(const TapsInput<T>& in, const LinearStateShape& s, const StateDecodeParams& p, void* out,
                               float* state, int rows, size_t smem, cudaStream_t stream) {
  auto kernel = s.beta_column >= 0 ? state_decode_kernel<T, MAXR, true, THREADS> : state_decode_kernel<T, MAXR, false, THREADS>;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return static_cast<int>(e);
  }
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
  StateDecodeParams p = *params;
  const int channels = 2 * s.kv_heads * s.d + s.heads * s.dv;
  if (!shape_ok(s) || in_stride < channels || taps > TAPS_MAX || (conv_w != nullptr && taps > 1 && conv_state == nullptr) ||
      s.dv % 4 != 0 || s.d % 4 != 0 || s.dv > 1024 || (p.own_conv && s.heads != s.kv_heads) || p.a_rank < 0 || p.g_rank < 0 || reinterpret_cast<uintptr_t>(state) % 16 != 0)
    return B200_BAD_SIZE;
  const int cg = s.dv / 4;
  int threads = 256;
  if (cg > threads || (s.d + threads / cg - 1) / (threads / cg) > 16) threads = 512;
  if (cg > threads) return B200_BAD_SIZE;
  const int rg = threads / cg, per = (s.d + rg - 1) / rg;
  const size_t plain = (3 * static_cast<size_t>(s.d) + 2 * s.dv + ((p.a_rank + p.g_rank + 3) & ~3) + static_cast<size_t>(rg) * s.dv) * sizeof(float);
  if (per > 20 || plain > 48 * 1024) return B200_BAD_SIZE;
  // the low-rank factors' rows of a head through shared memory, if they are whole pieces and two blocks still fit an SM
  const size_t item = dtype == B200_F32 ? 4 : 2;
  const size_t staged = s.d * (p.a_rank * item + 16) + (p.gate_kind == 0 ? s.dv * (p.g_rank * item + 16) : 0);
  p.stage = p.a_rank + p.g_rank > 0 && p.a_rank % 8 == 0 && (p.gate_kind != 0 || p.g_rank % 8 == 0) && plain + staged <= 100 * 1024 &&
            (reinterpret_cast<uintptr_t>(p.a2) | reinterpret_cast<uintptr_t>(p.g2)) % 16 == 0;
  const size_t smem = plain + (p.stage ? staged : 0);
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
