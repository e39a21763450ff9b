// The recurrence of linear_state.cu over rows of any length, token by token in the sequence's order whatever the step's cut.
// Per head, with S [d, dv] in float32 and the decay g of a token (one number a key channel, acting on S's rows, or one a
// head):
//
//   plain   S <- diag(g) S + k v^T                                                             o = S^T q
//   delta   S <- diag(g) S;   u = beta (v - S^T k);   S <- S + k u^T                           o = S^T q
//
// The inputs of every token in float come from state_prepare there: qf, kf [tokens, kv_heads * d], vf [tokens, heads * dv],
// gf [tokens, heads * d] (one decay a head: [tokens, heads]), beta [tokens, heads].
#include "common.cuh"

// The scan with one decay a head is a build of its own, for head sizes up to 32 STATE_HEAD_BLOCKS (0: the build whose scan
// has decays per key channel, for every head size).
#ifndef STATE_HEAD_BLOCKS
#define STATE_HEAD_BLOCKS 0
#endif

// ------------------------------------------------------------------ the recurrence, token by token
// grid (rows, heads, column tiles of 16 CPT).  A block of four warps owns 16 CPT columns of one head's state; CPT neighbouring
// columns belong to eight neighbouring lanes, lane l of them holding the rows 32 n + 4 l .. + 3 in registers (DI =
// 4 ceil(d / 32) a column).  Two columns a thread fetch a token's q, k and decays from shared memory, whose bandwidth a
// scan runs into, half as often; one a thread spreads a small grid over more warps.
// A column's products with k and q are sums over its eight lanes (three shuffles), so a token needs no barrier.  Groups of
// tokens come through a ring of buffers in shared memory (the copies of the next groups are in flight beside the
// recurrence); eight tokens are unrolled, so that a token's read-out overlaps the next token's update.
constexpr int LS_TOKENS = 8;                               // tokens that are unrolled
constexpr int ls_group(int di) { return di <= 16 ? 16 : 8; }      // tokens of a buffer
constexpr int ls_stages(int di) { return di <= 16 ? 3 : 4; }
constexpr int LS_LANES = 8;
constexpr int LS_THREADS = 128;

__device__ __forceinline__ float over_lanes(float v) {
  v += __shfl_xor_sync(0xffffffffu, v, 4);
  v += __shfl_xor_sync(0xffffffffu, v, 2);
  v += __shfl_xor_sync(0xffffffffu, v, 1);
  return v;
}

// Eight values a lane, summed over the eight lanes: lane l gets the sum of value l.  The same additions as over_lanes
// makes, in seven shuffles.
__device__ __forceinline__ float eight_over_lanes(const float (&v)[8], int l) {
  float a[4], b[2];
#pragma unroll
  for (int i = 0; i < 4; ++i) a[i] = ((l & 4) ? v[i + 4] : v[i]) + __shfl_xor_sync(0xffffffffu, (l & 4) ? v[i] : v[i + 4], 4);
#pragma unroll
  for (int i = 0; i < 2; ++i) b[i] = ((l & 2) ? a[i + 2] : a[i]) + __shfl_xor_sync(0xffffffffu, (l & 2) ? a[i] : a[i + 2], 2);
  return ((l & 1) ? b[1] : b[0]) + __shfl_xor_sync(0xffffffffu, (l & 1) ? b[0] : b[1], 1);
}

// A token's inputs on this lane's rows.  HEADG: one decay a head, a single number behind the step.
template <int DI, int CPT, bool HEADG>
struct LaneInputs {
  static constexpr int VECS = HEADG ? 2 : 3;          // vectors of dp floats in a token's buffer: q, k and channel decays
  float q[DI], k[DI], g[HEADG ? 1 : DI], v[CPT], beta;

  // tk: the token's buffer (q, k, g of dp floats each, COLS values, the step); pieces of a lane are 32 floats apart
  __device__ __forceinline__ void load(const float* tk, int dp, int l, int cj, int cols, bool delta) {
    const float4* q4 = reinterpret_cast<const float4*>(tk) + l;
    const float4* k4 = reinterpret_cast<const float4*>(tk + dp) + l;
    const float4* g4 = reinterpret_cast<const float4*>(tk + 2 * dp) + l;
#pragma unroll
    for (int i = 0; i < DI / 4; ++i) {
      const float4 b = k4[8 * i], c = q4[8 * i];
      if constexpr (!HEADG) {
        const float4 a = g4[8 * i];
        g[4 * i] = a.x; g[4 * i + 1] = a.y; g[4 * i + 2] = a.z; g[4 * i + 3] = a.w;
      }
      k[4 * i] = b.x; k[4 * i + 1] = b.y; k[4 * i + 2] = b.z; k[4 * i + 3] = b.w;
      q[4 * i] = c.x; q[4 * i + 1] = c.y; q[4 * i + 2] = c.z; q[4 * i + 3] = c.w;
    }
    if constexpr (HEADG) g[0] = tk[VECS * dp + cols + 1];
#pragma unroll
    for (int j = 0; j < CPT; ++j) v[j] = tk[VECS * dp + cj + j];
    beta = delta ? tk[VECS * dp + cols] : 0.0f;
  }
  __device__ __forceinline__ float decay(int i) const { return g[HEADG ? 0 : i]; }
};

// One token; out: this lane's parts of the read-outs of its columns.
template <int DI, int CPT, bool DELTA, bool HEADG>
__device__ __forceinline__ void state_token(float (&S)[CPT][DI], const LaneInputs<DI, CPT, HEADG>& x, float (&out)[CPT]) {
  float u[CPT];
  if constexpr (DELTA) {
    float dot[CPT][4] = {};
#pragma unroll
    for (int i = 0; i < DI; ++i)
#pragma unroll
      for (int j = 0; j < CPT; ++j) {
        S[j][i] *= x.decay(i);
        dot[j][i & 3] = fmaf(S[j][i], x.k[i], dot[j][i & 3]);
      }
#pragma unroll
    for (int j = 0; j < CPT; ++j) u[j] = x.beta * (x.v[j] - over_lanes((dot[j][0] + dot[j][1]) + (dot[j][2] + dot[j][3])));
  }
  float acc[CPT][4] = {};
#pragma unroll
  for (int i = 0; i < DI; ++i)
#pragma unroll
    for (int j = 0; j < CPT; ++j) {
      if constexpr (DELTA) S[j][i] = fmaf(x.k[i], u[j], S[j][i]);
      else S[j][i] = fmaf(x.decay(i), S[j][i], x.k[i] * x.v[j]);
      acc[j][i & 3] = fmaf(S[j][i], x.q[i], acc[j][i & 3]);
    }
#pragma unroll
  for (int j = 0; j < CPT; ++j) out[j] = (acc[j][0] + acc[j][1]) + (acc[j][2] + acc[j][3]);
}

// The delta rule over a group of LS_TOKENS tokens, what a token reads of the past being begun one token ahead, so that
// its sum over the lanes is on its way while the token before it updates the state and is read out.  With D = diag(g_t) S
// (the state of token t before its update) and the next token's k' and g':
//     S_t^T (g' k') = D^T (g' k') + u_t (k_t . (g' k'))
// and neither sum needs u_t.  The group's first token is read directly.
template <int DI, int CPT, bool HEADG>
__device__ __forceinline__ void delta_group(float (&S)[CPT][DI], const float* cur, int tok, int dp, int l, int cj, int cols,
                                            float (&part)[CPT][LS_TOKENS]) {
  LaneInputs<DI, CPT, HEADG> x[3];                          // this token's, the next one's, and the one's after that on their way
  x[0].load(cur, dp, l, cj, cols, true);
  x[1].load(cur + tok, dp, l, cj, cols, true);
  float past[CPT], mix = 0.0f, u[CPT] = {};
#pragma unroll
  for (int tb = 0; tb < LS_TOKENS; ++tb) {
    const LaneInputs<DI, CPT, HEADG>&now = x[tb % 3], &next = x[(tb + 1) % 3];
    if (tb + 2 < LS_TOKENS) x[(tb + 2) % 3].load(cur + (tb + 2) * tok, dp, l, cj, cols, true);
#pragma unroll
    for (int i = 0; i < DI; ++i)
#pragma unroll
      for (int j = 0; j < CPT; ++j) S[j][i] *= now.decay(i);
    if (tb == 0) {
#pragma unroll
      for (int j = 0; j < CPT; ++j) {
        float dot[4] = {};
#pragma unroll
        for (int i = 0; i < DI; ++i) dot[i & 3] = fmaf(S[j][i], now.k[i], dot[i & 3]);
        past[j] = over_lanes((dot[0] + dot[1]) + (dot[2] + dot[3]));
      }
    }
    float ahead[CPT], ahead_mix = 0.0f;
    if (tb + 1 < LS_TOKENS) {
      float dot[CPT][4] = {}, m[4] = {};
#pragma unroll
      for (int i = 0; i < DI; ++i) {
        const float kg = next.k[i] * next.decay(i);
        m[i & 3] = fmaf(kg, now.k[i], m[i & 3]);
#pragma unroll
        for (int j = 0; j < CPT; ++j) dot[j][i & 3] = fmaf(kg, S[j][i], dot[j][i & 3]);
      }
#pragma unroll
      for (int j = 0; j < CPT; ++j) ahead[j] = over_lanes((dot[j][0] + dot[j][1]) + (dot[j][2] + dot[j][3]));
      ahead_mix = over_lanes((m[0] + m[1]) + (m[2] + m[3]));
    }
#pragma unroll
    for (int j = 0; j < CPT; ++j) u[j] = now.beta * (now.v[j] - fmaf(mix, u[j], past[j]));
#pragma unroll
    for (int j = 0; j < CPT; ++j) {
      float acc[4] = {};
#pragma unroll
      for (int i = 0; i < DI; ++i) {
        S[j][i] = fmaf(now.k[i], u[j], S[j][i]);
        acc[i & 3] = fmaf(S[j][i], now.q[i], acc[i & 3]);
      }
      part[j][tb] = (acc[0] + acc[1]) + (acc[2] + acc[3]);
      past[j] = ahead[j];
    }
    mix = ahead_mix;
  }
}

template <int DI, bool DELTA, int CPT, bool HEADG>
__global__ void __launch_bounds__(LS_THREADS, DI <= 16 ? 3 : 1)
state_scan_kernel(const float* __restrict__ qf, const float* __restrict__ kf, const float* __restrict__ vf,
                  const float* __restrict__ gf, const float* __restrict__ beta, float* __restrict__ o,
                  float* __restrict__ state, const int* __restrict__ cu_q, const int* __restrict__ prefix_len,
                  const int* __restrict__ state_slots, int heads, int kv_heads, int d, int dv) {
  constexpr int DP = DI * LS_LANES;                                  // d, rounded up to a multiple of 32
  constexpr int THREADS = LS_THREADS, COLS = THREADS / LS_LANES * CPT;
  constexpr int VECS = LaneInputs<DI, CPT, HEADG>::VECS;
  constexpr int TOK = VECS * DP + COLS + 4;                          // q, k, channel decays, v, beta (and a head's decay) of one token
  constexpr int GROUP = ls_group(DI), STAGES = ls_stages(DI);
  extern __shared__ __align__(16) float smem[];                      // [STAGES][GROUP][TOK]
  const int r = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * COLS;
  const int hk = h / (heads / kv_heads);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int l = lane & (LS_LANES - 1);
  const int cj = (warp * 4 + (lane >> 3)) * CPT;                  // the first of this thread's columns inside the tile
  const int col = col0 + cj;
  const int first = cu_q[r], n = cu_q[r + 1] - first;
  float* st = state + (static_cast<size_t>(state_slots[r]) * heads + h) * d * dv;
  const bool has_past = prefix_len[r] > 0;

  float S[CPT][DI];
#pragma unroll
  for (int i = 0; i < DI; ++i) {
    const int e = (i >> 2) * 32 + l * 4 + (i & 3);
#pragma unroll
    for (int j = 0; j < CPT; ++j)
      S[j][i] = (has_past && col + j < dv && e < d) ? st[static_cast<size_t>(e) * dv + col + j] : 0.0f;
  }
  const bool wide = d % 4 == 0 && dv % 4 == 0;                       // rows of whole 16-byte pieces
  const int vcols = min(COLS, dv - col0);
  if (d != DP || vcols != COLS) {                                    // columns beyond d and dv stay zero in every buffer
    for (int i = threadIdx.x; i < STAGES * GROUP * TOK; i += THREADS) smem[i] = 0.0f;
    __syncthreads();
  }
  // Every thread copies the same pieces of every SLOTS-th token: PIECES pairs of an address in the token's inputs (which
  // moves on by a fixed stride a token) and one in the token's buffer.  16-byte pieces where rows are whole ones, else floats.
  constexpr int MOST = VECS * DP / 4 + COLS / 4;                     // pieces of a token
  constexpr int SLOTS = MOST <= THREADS / 4 ? 4 : MOST <= THREADS / 2 ? 2 : 1;
  constexpr int LINE = THREADS / SLOTS, PIECES = (MOST + LINE - 1) / LINE;
  const int line = threadIdx.x % LINE, slot = threadIdx.x / LINE;
  const int unit = wide ? 4 : 1;
  const int dq = d / unit, per = VECS * dq + vcols / unit;
  auto piece = [&](int p, const float*& src, int& stride, int& to) {
    const int part = p < dq ? 0 : p < 2 * dq ? 1 : p < VECS * dq ? 2 : VECS;      // which vector of the token's buffer
    const int kind = part == VECS ? 3 : part;
    const int at = unit * (p - part * dq);
    const int row_heads = kind < 2 ? kv_heads : heads, row_head = kind < 2 ? hk : h, size = kind == 3 ? dv : d;
    stride = row_heads * size;
    src = (kind == 0 ? qf : kind == 1 ? kf : kind == 2 ? gf : vf) + static_cast<size_t>(first) * stride + row_head * size +
          (kind == 3 ? col0 : 0) + at;
    to = part * DP + at;
  };
  const float* src[PIECES];
  int stride[PIECES], to[PIECES];
#pragma unroll
  for (int i = 0; i < PIECES; ++i) {
    src[i] = nullptr;
    stride[i] = to[i] = 0;
    if (wide && line + i * LINE < per) piece(line + i * LINE, src[i], stride[i], to[i]);
  }
  auto fetch = [&](int base, int buf) {                              // called for one group after the other
    float* dst = smem + buf * GROUP * TOK;
    const int nt = min(GROUP, n - base);
    if (wide) {
#pragma unroll
      for (int i = 0; i < PIECES; ++i) {
        if (src[i] == nullptr) continue;
        const float* s = src[i] + static_cast<size_t>(base + slot) * stride[i];
        float* d = dst + slot * TOK + to[i];
#pragma unroll
        for (int tb = 0; tb < GROUP; tb += SLOTS) {
          if (tb + slot < nt) cp_async16(d + tb * TOK, s, true);
          s += SLOTS * stride[i];
        }
      }
    } else {
      for (int p = threadIdx.x; p < per; p += THREADS) {
        const float* s;
        int step, at;
        piece(p, s, step, at);
        for (int tb = 0; tb < nt; ++tb) dst[tb * TOK + at] = s[static_cast<size_t>(base + tb) * step];
      }
    }
    if (DELTA && static_cast<int>(threadIdx.x) < nt)
      cp_async4(dst + threadIdx.x * TOK + VECS * DP + COLS, beta + static_cast<size_t>(first + base + threadIdx.x) * heads + h);
    if (HEADG && static_cast<int>(threadIdx.x) < nt)
      cp_async4(dst + threadIdx.x * TOK + VECS * DP + COLS + 1, gf + static_cast<size_t>(first + base + threadIdx.x) * heads + h);
  };
#pragma unroll
  for (int s = 0; s < STAGES - 1; ++s) {
    if (s * GROUP < n) fetch(s * GROUP, s);
    cp_async_commit();
  }
  int buf = 0;
  for (int base = 0; base < n; base += GROUP) {
    cp_async_wait<STAGES - 2>();
    __syncthreads();                                                 // this group is there, the buffer before it is free
    {
      const int ahead = base + (STAGES - 1) * GROUP;
      if (ahead < n) fetch(ahead, buf == 0 ? STAGES - 1 : buf - 1);
      cp_async_commit();
    }
#pragma unroll 1
    for (int half = 0; half < GROUP && base + half < n; half += LS_TOKENS) {
      const int nt = min(LS_TOKENS, n - base - half);
      const float* cur = smem + (buf * GROUP + half) * TOK;
      float* dst = o + (static_cast<size_t>(first + base + half) * heads + h) * dv + col;
      const size_t step = static_cast<size_t>(heads) * dv;
      if (nt == LS_TOKENS) {
        // the next token's inputs are on their way to registers while this one's sums go over the lanes (where they fit)
        constexpr int AHEAD = DI <= 16 ? 2 : 1;
        float part[CPT][LS_TOKENS];
        if constexpr (DELTA && AHEAD == 2) {
          delta_group<DI, CPT, HEADG>(S, cur, TOK, DP, l, cj, COLS, part);
        } else {
          LaneInputs<DI, CPT, HEADG> x[AHEAD];
          if constexpr (AHEAD == 2) x[0].load(cur, DP, l, cj, COLS, DELTA);
#pragma unroll
          for (int tb = 0; tb < LS_TOKENS; ++tb) {
            if constexpr (AHEAD == 2) {
              if (tb + 1 < LS_TOKENS) x[(tb + 1) & 1].load(cur + (tb + 1) * TOK, DP, l, cj, COLS, DELTA);
            } else {
              x[0].load(cur + tb * TOK, DP, l, cj, COLS, DELTA);
            }
            float out[CPT];
            state_token<DI, CPT, DELTA, HEADG>(S, x[AHEAD == 2 ? tb & 1 : 0], out);
#pragma unroll
            for (int j = 0; j < CPT; ++j) part[j][tb] = out[j];
          }
        }
#pragma unroll
        for (int j = 0; j < CPT; ++j) {
          const float mine = eight_over_lanes(part[j], l);             // lane l: token l
          if (col + j < dv) dst[l * step + j] = mine;
        }
      } else {
        for (int tb = 0; tb < nt; ++tb) {
          LaneInputs<DI, CPT, HEADG> x;
          x.load(cur + tb * TOK, DP, l, cj, COLS, DELTA);
          float out[CPT];
          state_token<DI, CPT, DELTA, HEADG>(S, x, out);
#pragma unroll
          for (int j = 0; j < CPT; ++j) {
            const float mine = over_lanes(out[j]);
            if (l == 0 && col + j < dv) dst[tb * step + j] = mine;
          }
        }
      }
    }
    buf = buf + 1 == STAGES ? 0 : buf + 1;
  }
#pragma unroll
  for (int i = 0; i < DI; ++i) {
    const int e = (i >> 2) * 32 + l * 4 + (i & 3);
#pragma unroll
    for (int j = 0; j < CPT; ++j)
      if (col + j < dv && e < d) st[static_cast<size_t>(e) * dv + col + j] = S[j][i];
  }
}

template <int DI, int CPT, bool HEADG>
static int launch_state_scan(const float* qf, const float* kf, const float* vf, const float* gf, const float* beta, float* o,
                             float* state, const int* cu_q, const int* prefix_len, const int* state_slots, int num_rows,
                             int heads, int kv_heads, int d, int dv, cudaStream_t stream) {
  constexpr int COLS = LS_THREADS / LS_LANES * CPT;
  const size_t smem = ls_stages(DI) * ls_group(DI) * ((HEADG ? 2 : 3) * DI * LS_LANES + COLS + 4) * sizeof(float);
  const dim3 grid(num_rows, heads, (dv + COLS - 1) / COLS);
  auto kernel = beta != nullptr ? state_scan_kernel<DI, true, CPT, HEADG> : state_scan_kernel<DI, false, CPT, HEADG>;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return static_cast<int>(e);
  }
  kernel<<<grid, LS_THREADS, smem, stream>>>(qf, kf, vf, gf, beta, o, state, cu_q, prefix_len, state_slots, heads, kv_heads,
                                                  d, dv);
  return b200_check_launch();
}

// beta null: without the delta rule.  head_decay: gf has one decay a head ([num tokens, heads]).
B200_EXPORT int b200_state_scan(const float* qf, const float* kf, const float* vf, const float* gf, const float* beta, float* o,
                                float* state, const int* cu_q, const int* prefix_len, const int* state_slots, int num_rows,
                                int heads, int kv_heads, int d, int dv, int head_decay, cudaStream_t stream) {
  if (num_rows <= 0) return 0;
  if (heads <= 0 || heads > 65535 || kv_heads <= 0 || heads % kv_heads || d <= 0 || d > 512 || dv <= 0 ||
      (dv + 15) / 16 > 65535)
    return B200_BAD_SIZE;
  if ((head_decay != 0) != (STATE_HEAD_BLOCKS > 0)) return B200_BAD_SIZE;      // another build's scan
  const int blocks = (d + 31) / 32;
  // One column a thread while that leaves a scheduler (148 SMs of four) one warp at most, else two.
  const bool narrow = static_cast<long long>(num_rows) * heads * ((dv + 3) / 4) <= 4 * 148;
#if STATE_HEAD_BLOCKS
  if (blocks > STATE_HEAD_BLOCKS) return B200_BAD_SIZE;
#define LS_CASE_C(C)                                                                                                  \
  return launch_state_scan<4 * STATE_HEAD_BLOCKS, C, true>(qf, kf, vf, gf, beta, o, state, cu_q, prefix_len,           \
                                                           state_slots, num_rows, heads, kv_heads, d, dv, stream)
  if (narrow) LS_CASE_C(1);
  LS_CASE_C(2);
#undef LS_CASE_C
#else
#define LS_CASE_C(N, C)                                                                                            \
  return launch_state_scan<4 * N, C, false>(qf, kf, vf, gf, beta, o, state, cu_q, prefix_len, state_slots, num_rows,   \
                                            heads, kv_heads, d, dv, stream)
#define LS_CASE(N)                     \
  if (blocks <= N) {                   \
    if (narrow) LS_CASE_C(N, 1);       \
    LS_CASE_C(N, 2);                   \
  }
  LS_CASE(1)
  LS_CASE(2)
  LS_CASE(3)
  LS_CASE(4)
  LS_CASE(6)
  LS_CASE(8)
  LS_CASE(16)
#undef LS_CASE
#undef LS_CASE_C
  return B200_BAD_SIZE;
#endif
}
