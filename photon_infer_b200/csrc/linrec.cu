// Recurrent mixers whose state is one matrix per head, S [N][dv] in 32-bit, that decays by ONE number per head and
// token (modes 0 and 1) or by a number per row (mode 2) and takes a rank-one update:
//
//   S_t = keep_t S_(t-1) + take_t k_t v_t^T,      o_t = S_t^T q_t                        (per head)
//
// Three mixers are this recurrence with different gates.
//
//   state-space (mode 0):  k = B_t, q = C_t (of the head's group), v = x_t;  dt = softplus(dt_raw + dt_bias[h]);
//                          keep = exp(-exp(A_log[h]) dt), take = dt;  y_t = o_t + D[h] x_t.
//   matrix memory (mode 1): log gates i = cap tanh((i_raw + b_i[h]) / cap), f = logsigmoid(cap tanh((f_raw + b_f[h]) / cap));
//                          a running maximum m (from 0): m_t = max(f + m_(t-1), i); keep = exp(f + m_(t-1) - m_t),
//                          take = exp(i - m_t); a vector n_t = keep n_(t-1) + take k_t rides along as one more
//                          column of S (with v = 1);  y_t = o_t / (max(|n_t . q_t|, exp(-m_t)) + 1e-6).
//   forget-and-write (mode 2): a gate per row f = l + (1 - l) sigmoid(z + b) keeps and 1 - f writes, so that a row of the
//                          state is a running mean of the values: S_t = S_(t-1) + k_t (v_t^T - S_(t-1)) with the write gate
//                          k = (1 - l) / (1 + exp(z + b)), formed without the cancellation in 1 - f;  y_t = o_t.  q enters
//                          as silu(q).
//
//   photon_conv_silu        y = silu(bias + causal convolution over `taps` tokens per channel); the taps before the
//                           step's first token of a request come from the request's state.
//   photon_conv_state       the last taps - 1 input rows of every request of the step go into its state.
//   photon_linrec           the recurrence over the tokens of a step, for all requests and heads.
//   photon_linrec_gates     mode 2: silu(q) and the write gates of all tokens side by side, for long portions, whose blocks
//                           would otherwise form them once per sixteen columns (few tokens: photon_linrec does it itself).
//
// A request's state is one float row per layer; S [H][N][dv] comes first, then (mode 1) n [H][N] and m [H]; the
// convolution's rows live at an offset the caller gives.  A state slot of -1 starts from zeros and stores nothing.
// Every token's arithmetic is the same chain whatever the step brought before it, and the cut of a head's columns
// into blocks changes no column's arithmetic, so a request's numbers depend neither on how it was cut into steps nor
// on the batch.
#include "common.cuh"
#include <math.h>

// ---------------------------------------------------------------- short causal convolution
template <typename TI>
__global__ void __launch_bounds__(128)
conv_silu_kernel(const TI* __restrict__ x, long x_stride, const float* __restrict__ taps_w, const float* __restrict__ bias,
                 int taps, const int* __restrict__ token_seq, const int* __restrict__ cu_tokens,
                 const int* __restrict__ state_slots, const float* __restrict__ state, long state_stride, long conv_offset,
                 int num_slots, float* __restrict__ y, int C, int* err) {
  const int t = blockIdx.y;
  const int c = blockIdx.x * 128 + threadIdx.x;
  if (c >= C) return;
  const int s = token_seq[t];
  const int p = t - cu_tokens[s];                     // index of the token among the request's tokens of this step
  int slot = state_slots[s];
  if (slot >= num_slots) {
    if (c == 0) report_error(err, PHOTON_DEV_BAD_SLOT, t, slot, num_slots);
    slot = -1;
  }
  const float* old = slot >= 0 ? state + (size_t)slot * state_stride + conv_offset : nullptr;   // [taps - 1][C], oldest first
  float a = bias ? bias[c] : 0.f;
  for (int j = 0; j < taps; ++j) {
    const int back = taps - 1 - j;                    // tap j weighs the token `back` places before this one
    float xv;
    if (back <= p) xv = to_f32(x[(size_t)(t - back) * x_stride + c]);
    else xv = old ? old[(size_t)(taps - 1 - (back - p)) * C + c] : 0.f;
    a = fmaf(taps_w[(size_t)c * taps + j], xv, a);
  }
  y[(size_t)t * C + c] = a / (1.0f + expf(-a));
}

// x [T][>= C] of x_dtype (row stride x_stride), taps_w float [C][taps] (the last column weighs the current token), bias
// float [C] or null, y float [T][C].  state float [num_slots][state_stride]; the request's last taps - 1 input rows lie at
// conv_offset, oldest first.
PHOTON_API int photon_conv_silu(const void* x, long x_stride, int x_dtype, const float* taps_w, const float* bias, int taps,
                                const int* token_seq, const int* cu_tokens, const int* state_slots, const float* state,
                                long state_stride, long conv_offset, int num_slots, float* y, int T, int C, int* err,
                                cudaStream_t stream) {
  if (T <= 0) return 0;
  if (C <= 0 || taps < 1 || x == nullptr || y == nullptr) return PHOTON_ERR_ARGUMENT;
  if (T > 65535) return PHOTON_ERR_UNSUPPORTED;
  dim3 grid((C + 127) / 128, T);
  if (x_dtype == PHOTON_BF16)
    conv_silu_kernel<bf16><<<grid, 128, 0, stream>>>((const bf16*)x, x_stride, taps_w, bias, taps, token_seq, cu_tokens, state_slots,
                                                     state, state_stride, conv_offset, num_slots, y, C, err);
  else
    conv_silu_kernel<float><<<grid, 128, 0, stream>>>((const float*)x, x_stride, taps_w, bias, taps, token_seq, cu_tokens, state_slots,
                                                      state, state_stride, conv_offset, num_slots, y, C, err);
  return launch_status();
}

// The new rows of a request: the last taps - 1 of (its old rows, then the step's input rows).  A thread owns one channel
// of one request and reads all it needs before it writes, so the rows may move in place.
template <typename TI>
__global__ void __launch_bounds__(128)
conv_state_kernel(const TI* __restrict__ x, long x_stride, int taps, const int* __restrict__ cu_tokens,
                  const int* __restrict__ state_slots, float* __restrict__ state, long state_stride, long conv_offset,
                  int num_slots, int C) {
  const int s = blockIdx.y;
  const int c = blockIdx.x * 128 + threadIdx.x;
  if (c >= C) return;
  const int slot = state_slots[s];
  if (slot < 0 || slot >= num_slots) return;
  const int t0 = cu_tokens[s], n = cu_tokens[s + 1] - t0;
  const int keep = taps - 1;
  float* rows = state + (size_t)slot * state_stride + conv_offset;
  constexpr int MAXK = 16;
  float tmp[MAXK];
  for (int r = 0; r < keep; ++r) {
    const int src = r + n;                            // index in (old rows, new rows)
    tmp[r] = src < keep ? rows[(size_t)src * C + c] : to_f32(x[(size_t)(t0 + src - keep) * x_stride + c]);
  }
  for (int r = 0; r < keep; ++r) rows[(size_t)r * C + c] = tmp[r];
}

PHOTON_API int photon_conv_state(const void* x, long x_stride, int x_dtype, int taps, const int* cu_tokens,
                                 const int* state_slots, float* state, long state_stride, long conv_offset, int num_slots,
                                 int S, int C, cudaStream_t stream) {
  if (S <= 0 || taps <= 1) return 0;
  if (taps - 1 > 16) return PHOTON_ERR_UNSUPPORTED;
  if (C <= 0 || S > 65535) return PHOTON_ERR_ARGUMENT;
  dim3 grid((C + 127) / 128, S);
  if (x_dtype == PHOTON_BF16)
    conv_state_kernel<bf16><<<grid, 128, 0, stream>>>((const bf16*)x, x_stride, taps, cu_tokens, state_slots, state, state_stride,
                                                      conv_offset, num_slots, C);
  else
    conv_state_kernel<float><<<grid, 128, 0, stream>>>((const float*)x, x_stride, taps, cu_tokens, state_slots, state, state_stride,
                                                       conv_offset, num_slots, C);
  return launch_status();
}

// ---------------------------------------------------------------- the recurrence
// A block owns LR_COLS neighbouring columns of one (request, head): 8 lanes share a column, lane i of them holding rows
// i RPL .. i RPL + RPL - 1 of it in registers (RPL a multiple of 4, N <= 8 RPL).  The step's tokens of the request come in
// chunks of LR_CHUNK: their keys, queries, the block's share of their values and their raw gates arrive by cp.async in
// one of two stages of shared memory while the chunk before is walked; one warp turns the raw gates into keep and take
// (the running maximum in token order); then the walk over the chunk needs no barrier and no shuffle: per token RPL
// multiply-adds for the update and RPL for the read-out (operands fetched 16 bytes at a time); the eight lanes' shares of
// a column's read-out meet when the chunk is written out.  In mode 1 the block's last column is the vector n (its value
// is 1), so every block knows n . q for its own columns.
#define LR_CHUNK 16
#define LR_COLS 16
#define LR_THREADS 128

__device__ __forceinline__ float lr_softplus(float x) { return x > 20.f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float lr_logsigmoid(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ void lr_cp4(float* dst, const float* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src));
}
__device__ __forceinline__ void lr_cp16(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src));
}
__device__ __forceinline__ void lr_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int K> __device__ __forceinline__ void lr_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(K) : "memory"); }

// Mode 2's inputs.
__device__ __forceinline__ float lr_silu(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ float lr_write_gate(float z, float bias, float lower) { return (1.0f - lower) / (1.0f + expf(z + bias)); }

// A thread owns four neighbouring channels of LR_GATE_TOK tokens (V 1: one channel).
#define LR_GATE_TOK 4
template <int V>
__global__ void __launch_bounds__(256)
linrec_gates_kernel(const float* __restrict__ q, long q_stride, const float* __restrict__ z, long z_stride,
                    const float* __restrict__ bias, const float* __restrict__ lower, float* __restrict__ q_out,
                    float* __restrict__ k_out, long out_stride, int T, int C) {
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
  if (c >= C) return;
  float b[V], l[V], x[V];
#pragma unroll
  for (int e = 0; e < V; ++e) { b[e] = bias[c + e]; l[e] = lower[c + e]; }
  auto load = [&](const float* p) {
    if constexpr (V == 4) { const float4 r = *reinterpret_cast<const float4*>(p); x[0] = r.x; x[1] = r.y; x[2] = r.z; x[3] = r.w; }
    else x[0] = *p;
  };
  auto store = [&](float* p) {
    if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(x[0], x[1], x[2], x[3]);
    else *p = x[0];
  };
#pragma unroll
  for (int u = 0; u < LR_GATE_TOK; ++u) {
    const int t = blockIdx.y * LR_GATE_TOK + u;
    if (t >= T) return;
    load(q + (size_t)t * q_stride + c);
#pragma unroll
    for (int e = 0; e < V; ++e) x[e] = lr_silu(x[e]);
    store(q_out + (size_t)t * out_stride + c);
    load(z + (size_t)t * z_stride + c);
#pragma unroll
    for (int e = 0; e < V; ++e) x[e] = lr_write_gate(x[e], b[e], l[e]);
    store(k_out + (size_t)t * out_stride + c);
  }
}

// q, z float [T][C] views, bias and lower float [C]; q_out = silu(q), k_out = (1 - lower) sigmoid(-(z + bias)).
PHOTON_API int photon_linrec_gates(const float* q, long q_stride, const float* z, long z_stride, const float* bias,
                                   const float* lower, float* q_out, float* k_out, long out_stride, int T, int C,
                                   cudaStream_t stream) {
  if (T <= 0 || C <= 0) return 0;
  const int rows = (T + LR_GATE_TOK - 1) / LR_GATE_TOK;
  if (rows > 65535) return PHOTON_ERR_UNSUPPORTED;
  const bool vec = C % 4 == 0 && q_stride % 4 == 0 && z_stride % 4 == 0 && out_stride % 4 == 0 && ((uintptr_t)q & 15) == 0 &&
                   ((uintptr_t)z & 15) == 0 && ((uintptr_t)q_out & 15) == 0 && ((uintptr_t)k_out & 15) == 0;
  if (vec)
    linrec_gates_kernel<4><<<dim3((C + 1023) / 1024, rows), 256, 0, stream>>>(q, q_stride, z, z_stride, bias, lower, q_out, k_out, out_stride, T, C);
  else
    linrec_gates_kernel<1><<<dim3((C + 255) / 256, rows), 256, 0, stream>>>(q, q_stride, z, z_stride, bias, lower, q_out, k_out, out_stride, T, C);
  return launch_status();
}

// Eight shares of one sum, added in a fixed order.
__device__ __forceinline__ float lr_sum8(const float* p) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  return ((a.x + a.y) + (a.z + a.w)) + ((b.x + b.y) + (b.z + b.w));
}

template <int MODE, int RPL>
__global__ void __launch_bounds__(LR_THREADS)
linrec_kernel(const float* __restrict__ q, long q_stride, const float* __restrict__ k, long k_stride,
              const float* __restrict__ v, long v_stride, const float* __restrict__ ga, const float* __restrict__ gb,
              long g_stride, const float* __restrict__ p0, const float* __restrict__ p1, const float* __restrict__ p2,
              float cap, float q_scale, const int* __restrict__ cu_tokens, const int* __restrict__ state_slots,
              float* __restrict__ state, long state_stride, int num_slots, float* __restrict__ out, long out_stride,
              int H, int qk_heads, int N, int dv, int vec, int* err) {
  constexpr int NPS = 8 * (RPL + 4);                   // a staged row: 8 lanes' rows, each lane's share 16 bytes further on
  constexpr int REAL = MODE == 1 ? LR_COLS - 1 : LR_COLS;   // columns of S per block
  extern __shared__ __align__(16) float lr_smem[];
  float* ks = lr_smem;                                 // [2][CHUNK][NPS]
  float* qs = ks + 2 * LR_CHUNK * NPS;                 // [2][CHUNK][NPS]
  float* vs = qs + 2 * LR_CHUNK * NPS;                 // [2][CHUNK][COLS]
  float* raw = vs + 2 * LR_CHUNK * LR_COLS;            // [2][2][CHUNK]: the raw gates
  __shared__ __align__(16) float os[LR_CHUNK][LR_COLS][8];
  __shared__ float keep_s[LR_CHUNK], take_s[LR_CHUNK], floor_s[LR_CHUNK];
  __shared__ float m_run;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int sub = lane & 7;                            // this lane's place among the 8 lanes of its column
  const int col = warp * 4 + (lane >> 3);              // column within the block
  const int h = blockIdx.y, s = blockIdx.z;
  const int c0 = blockIdx.x * REAL;
  const bool is_n = MODE == 1 && col == LR_COLS - 1;   // the column that carries n
  const int c = c0 + col;                              // column of S
  const bool live = is_n || (col < REAL && c < dv);
  const int hq = h / (H / qk_heads);
  int slot = state_slots[s];
  if (slot >= num_slots) {
    if (tid == 0 && blockIdx.x == 0 && h == 0) report_error(err, PHOTON_DEV_BAD_SLOT, s, slot, num_slots);
    slot = -1;
  }
  float* st = slot >= 0 ? state + (size_t)slot * state_stride : nullptr;
  float* S_h = st ? st + (size_t)h * N * dv : nullptr;
  float* n_h = (st && MODE == 1) ? st + (size_t)H * N * dv + (size_t)h * N : nullptr;
  float* m_h = (st && MODE == 1) ? st + (size_t)H * N * dv + (size_t)H * N + h : nullptr;

  float S[RPL];
#pragma unroll
  for (int i = 0; i < RPL; ++i) {
    const int r = sub * RPL + i;
    float x = 0.f;
    if (st && live && r < N) x = is_n ? n_h[r] : S_h[(size_t)r * dv + c];
    S[i] = x;
  }
  if (tid == 0) m_run = (MODE == 1 && m_h) ? *m_h : 0.f;
  // what no copy writes stays as it is set here: rows beyond N, columns beyond the head, the value 1 of the n column
  for (int i = tid; i < 2 * LR_CHUNK * NPS; i += LR_THREADS) { ks[i] = 0.f; qs[i] = 0.f; }
  for (int i = tid; i < 2 * LR_CHUNK * LR_COLS; i += LR_THREADS) vs[i] = (MODE == 1 && (i % LR_COLS) == LR_COLS - 1) ? 1.f : 0.f;
  for (int i = tid; i < 4 * LR_CHUNK; i += LR_THREADS) raw[i] = 0.f;
  __syncthreads();
  const int t0 = cu_tokens[s], t1 = cu_tokens[s + 1];
  const float a_h = MODE == 0 ? expf(p0[h]) : 0.f;     // the head's decay rate

  auto issue = [&](int base, int stage) {
    const int cnt = min(LR_CHUNK, t1 - base);
    float* kd = ks + (size_t)stage * LR_CHUNK * NPS;
    float* qd = qs + (size_t)stage * LR_CHUNK * NPS;
    if (vec) {
      const int per = N / 4;                           // 16-byte pieces of a row; a piece never straddles two lanes' shares
      for (int i = tid; i < cnt * per; i += LR_THREADS) {
        const int tt = i / per, r = (i - tt * per) * 4;
        const int at = tt * NPS + r + (r / RPL) * 4;
        lr_cp16(kd + at, k + (size_t)(base + tt) * k_stride + (size_t)hq * N + r);
        lr_cp16(qd + at, q + (size_t)(base + tt) * q_stride + (size_t)hq * N + r);
      }
    } else {
      for (int i = tid; i < cnt * N; i += LR_THREADS) {
        const int tt = i / N, r = i - tt * N;
        const int at = tt * NPS + r + (r / RPL) * 4;
        lr_cp4(kd + at, k + (size_t)(base + tt) * k_stride + (size_t)hq * N + r);
        lr_cp4(qd + at, q + (size_t)(base + tt) * q_stride + (size_t)hq * N + r);
      }
    }
    const int ncol = min(REAL, dv - c0);
    float* vd = vs + (size_t)stage * LR_CHUNK * LR_COLS;
    for (int i = tid; i < cnt * ncol; i += LR_THREADS) {
      const int tt = i / ncol, cc = i - tt * ncol;
      lr_cp4(vd + tt * LR_COLS + cc, v + (size_t)(base + tt) * v_stride + (size_t)h * dv + c0 + cc);
    }
    float* rd = raw + (size_t)stage * 2 * LR_CHUNK;
    if (tid < cnt) lr_cp4(rd + tid, ga + (size_t)(base + tid) * g_stride + h);
    else if (MODE == 1 && tid >= 32 && tid < 32 + cnt) lr_cp4(rd + LR_CHUNK + tid - 32, gb + (size_t)(base + tid - 32) * g_stride + h);
    lr_commit();
  };

  if (t0 < t1) issue(t0, 0);
  int stage = 0;
  for (int base = t0; base < t1; base += LR_CHUNK, stage ^= 1) {
    const int cnt = min(LR_CHUNK, t1 - base);
    __syncthreads();                                   // the chunk before is written out: the other stage is free
    if (base + LR_CHUNK < t1) { issue(base + LR_CHUNK, stage ^ 1); lr_wait<1>(); } else lr_wait<0>();
    __syncthreads();                                   // this chunk has landed for every thread
    const float* kd = ks + (size_t)stage * LR_CHUNK * NPS;
    const float* qd = qs + (size_t)stage * LR_CHUNK * NPS;
    const float* vd = vs + (size_t)stage * LR_CHUNK * LR_COLS;
    const float* rd = raw + (size_t)stage * 2 * LR_CHUNK;
    if (MODE == 0) {
      if (tid < cnt) {
        const float dt = lr_softplus(rd[tid] + p1[h]);
        keep_s[tid] = expf(-a_h * dt);
        take_s[tid] = dt;
      }
    } else if (warp == 0) {
      float gi = 0.f, gf = 0.f;
      if (lane < cnt) {
        gi = cap * tanhf((rd[lane] + p0[h]) / cap);                          // log input gate
        gf = lr_logsigmoid(cap * tanhf((rd[LR_CHUNK + lane] + p1[h]) / cap));  // log forget gate
      }
      float m = m_run, fm_mine = 0.f, mn_mine = 0.f;
      for (int tt = 0; tt < cnt; ++tt) {               // the running maximum, in token order (every lane walks it)
        const float fi = __shfl_sync(0xffffffffu, gi, tt), ff = __shfl_sync(0xffffffffu, gf, tt);
        const float fm = ff + m;
        const float mn = fmaxf(fm, fi);
        if (lane == tt) { fm_mine = fm; mn_mine = mn; }
        m = mn;
      }
      if (lane < cnt) { keep_s[lane] = expf(fm_mine - mn_mine); take_s[lane] = expf(gi - mn_mine); floor_s[lane] = expf(-mn_mine); }
      if (lane == 0) m_run = m;
    }
    __syncthreads();
    const float* kl = kd + sub * (RPL + 4);
    const float* ql = qd + sub * (RPL + 4);
#pragma unroll 4
    for (int tt = 0; tt < cnt; ++tt) {
      const float keep = keep_s[tt];
      const float w = take_s[tt] * vd[tt * LR_COLS + col];
      float a0 = 0.f, a1 = 0.f, a2 = 0.f, a3 = 0.f;
#pragma unroll
      for (int j = 0; j < RPL / 4; ++j) {
        const float4 k4 = *reinterpret_cast<const float4*>(kl + tt * NPS + 4 * j);
        const float4 q4 = *reinterpret_cast<const float4*>(ql + tt * NPS + 4 * j);
        S[4 * j + 0] = fmaf(k4.x, w, keep * S[4 * j + 0]);
        S[4 * j + 1] = fmaf(k4.y, w, keep * S[4 * j + 1]);
        S[4 * j + 2] = fmaf(k4.z, w, keep * S[4 * j + 2]);
        S[4 * j + 3] = fmaf(k4.w, w, keep * S[4 * j + 3]);
        a0 = fmaf(S[4 * j + 0], q4.x, a0);
        a1 = fmaf(S[4 * j + 1], q4.y, a1);
        a2 = fmaf(S[4 * j + 2], q4.z, a2);
        a3 = fmaf(S[4 * j + 3], q4.w, a3);
      }
      os[tt][col][sub] = (a0 + a1) + (a2 + a3);         // the eight lanes' shares of a column meet after the walk
    }
    __syncthreads();
    for (int i = tid; i < cnt * REAL; i += LR_THREADS) {
      const int tt = i / REAL, cc = i - tt * REAL;
      if (c0 + cc >= dv) continue;
      float y = lr_sum8(os[tt][cc]) * q_scale;         // the queries' factor, taken out of the sums
      if (MODE == 0) y = fmaf(p2[h], vd[tt * LR_COLS + cc], y);
      else y = y / (fmaxf(fabsf(lr_sum8(os[tt][LR_COLS - 1]) * q_scale), floor_s[tt]) + 1e-6f);
      out[(size_t)(base + tt) * out_stride + (size_t)h * dv + c0 + cc] = y;
    }
  }
  if (st && live) {
    if (!is_n) {
#pragma unroll
      for (int i = 0; i < RPL; ++i) { const int r = sub * RPL + i; if (r < N) S_h[(size_t)r * dv + c] = S[i]; }
    } else if (blockIdx.x == 0) {
#pragma unroll
      for (int i = 0; i < RPL; ++i) { const int r = sub * RPL + i; if (r < N) n_h[r] = S[i]; }
    }
  }
  __syncthreads();
  if (MODE == 1 && m_h && tid == 0 && blockIdx.x == 0) *m_h = m_run;
}

template <int MODE, int RPL>
static int linrec_go(dim3 grid, cudaStream_t stream, const float* q, long q_stride, const float* k, long k_stride, const float* v,
                     long v_stride, const float* ga, const float* gb, long g_stride, const float* p0, const float* p1,
                     const float* p2, float cap, float q_scale, const int* cu_tokens, const int* state_slots, float* state,
                     long state_stride, int num_slots, float* out, long out_stride, int H, int qk_heads, int N, int dv, int vec,
                     int* err) {
  const size_t smem = ((size_t)4 * LR_CHUNK * 8 * (RPL + 4) + 2 * LR_CHUNK * LR_COLS + 4 * LR_CHUNK) * sizeof(float);
  if (smem > 36 * 1024) {                              // with the 9 KB of static arrays this passes the default limit
    cudaError_t e = cudaFuncSetAttribute(linrec_kernel<MODE, RPL>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  linrec_kernel<MODE, RPL><<<grid, LR_THREADS, smem, stream>>>(q, q_stride, k, k_stride, v, v_stride, ga, gb, g_stride, p0, p1, p2, cap,
      q_scale, cu_tokens, state_slots, state, state_stride, num_slots, out, out_stride, H, qk_heads, N, dv, vec, err);
  return launch_status();
}

template <int MODE>
static int linrec_launch(int rpl, dim3 grid, cudaStream_t stream, const float* q, long q_stride, const float* k, long k_stride,
                         const float* v, long v_stride, const float* ga, const float* gb, long g_stride, const float* p0,
                         const float* p1, const float* p2, float cap, float q_scale, const int* cu_tokens,
                         const int* state_slots, float* state, long state_stride, int num_slots, float* out, long out_stride,
                         int H, int qk_heads, int N, int dv, int* err) {
  // 16-byte copies of keys and queries when every row piece is aligned
  const int vec = (N % 4 == 0 && q_stride % 4 == 0 && k_stride % 4 == 0 && ((uintptr_t)q & 15) == 0 && ((uintptr_t)k & 15) == 0) ? 1 : 0;
#define LR_GO(R) return linrec_go<MODE, R>(grid, stream, q, q_stride, k, k_stride, v, v_stride, ga, gb, g_stride, p0, p1, p2, cap, q_scale, \
      cu_tokens, state_slots, state, state_stride, num_slots, out, out_stride, H, qk_heads, N, dv, vec, err)
  if (rpl <= 4) LR_GO(4);
  if (rpl <= 8) LR_GO(8);
  if (rpl <= 12) LR_GO(12);
  if (rpl <= 16) LR_GO(16);
  if (rpl <= 24) LR_GO(24);
  if (rpl <= 32) LR_GO(32);
  if (rpl <= 48) LR_GO(48);
  if (rpl <= 64) LR_GO(64);
  return PHOTON_ERR_UNSUPPORTED;
}

// ---------------------------------------------------------------- a gate per row (mode 2)
// A lane owns R rows x 4 columns of one (request, head)'s state, as pairs of neighbouring rows for the packed 32-bit
// instructions of sm_100 (a pair is two IEEE operations); L lanes share the columns, lane i of them holding the rows
// (j L + i) 4 .. + 3, j < R / 4 (N <= L R).  A block of four warps owns 16 * 32 / L neighbouring columns.  Per token a pair takes
// d = v - S, S += k d, o += q S; the lanes' shares of the read-outs meet by shuffles in one tree over the lanes, so every
// token's arithmetic is the same chain wherever its step starts.  (Two columns a lane and eight warps take the same time for
// one request of 2,048 tokens and 16 heads of 128 x 128, and a tenth more for 32 heads.)
#define LRR_C 4                 // columns of a lane: 2 or 4
#define LRR_THREADS (512 / LRR_C)
typedef unsigned long long lr_pair;
struct alignas(LRR_C * 4) LrCols { float x[LRR_C]; };   // the lane's columns of one row
__device__ __forceinline__ lr_pair lr_dup(float x) { lr_pair d; asm("mov.b64 %0, {%1, %1};" : "=l"(d) : "f"(x)); return d; }
__device__ __forceinline__ lr_pair lr_mul2(lr_pair a, lr_pair b) { lr_pair d; asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b)); return d; }
__device__ __forceinline__ lr_pair lr_fma2(lr_pair a, lr_pair b, lr_pair c) {
  lr_pair d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ float lr_sum2(lr_pair a) {
  float x, y;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(x), "=f"(y) : "l"(a));
  return x + y;
}
__device__ __forceinline__ lr_pair lr_make(float x, float y) { lr_pair d; asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(x), "f"(y)); return d; }
__device__ __forceinline__ void lr_split(lr_pair a, float& x, float& y) { asm("mov.b64 {%0, %1}, %2;" : "=f"(x), "=f"(y) : "l"(a)); }

// The lanes' shares of NV sums meet over the distances D, D / 2 .. 1: while a lane holds several sums it keeps half of them (the
// upper half where the distance's bit of its number is set) and hands over the others.
template <int D, int NV, int M>
__device__ __forceinline__ void lr_meet(float (&val)[M], int sub) {
  if constexpr (D > 0) {
    if constexpr (NV > 1) {
      const bool up = sub & D;
#pragma unroll
      for (int i = 0; i < NV / 2; ++i) {
        const float own = up ? val[i + NV / 2] : val[i], other = up ? val[i] : val[i + NV / 2];
        val[i] = own + __shfl_xor_sync(0xffffffffu, other, D);
      }
      lr_meet<D / 2, NV / 2>(val, sub);
    } else {
      val[0] += __shfl_xor_sync(0xffffffffu, val[0], D);
      lr_meet<D / 2, 1>(val, sub);
    }
  }
}

template <int L, int R>
__global__ void __launch_bounds__(LRR_THREADS)
linrec_rows_kernel(const float* __restrict__ q, long q_stride, const float* __restrict__ k, long k_stride,
                   const float* __restrict__ v, long v_stride, const float* __restrict__ bias, const float* __restrict__ lower,
                   float q_scale, const int* __restrict__ cu_tokens, const int* __restrict__ state_slots, float* __restrict__ state,
                   long state_stride, int num_slots, float* __restrict__ out, long out_stride, int H, int qk_heads, int N, int dv,
                   int vec, int* err) {
  constexpr int NP = L * R;                            // rows, padded
  constexpr int BC = 16 * (32 / L);                    // columns of a block
  constexpr int TG = R == 4 ? 4 : (R == 8 ? 2 : 1);    // tokens at a time
  extern __shared__ __align__(16) float lr_smem[];
  float* ks = lr_smem;                                 // [2][CHUNK][NP]
  float* qs = ks + 2 * LR_CHUNK * NP;                  // [2][CHUNK][NP]
  float* vs = qs + 2 * LR_CHUNK * NP;                  // [2][CHUNK][BC]
  float* os = vs + 2 * LR_CHUNK * BC;                  // [CHUNK][BC]
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int sub = lane & (L - 1);
  const int col = (warp * (32 / L) + lane / L) * LRR_C;    // the lane's first column within the block
  const int h = blockIdx.y, s = blockIdx.z;
  const int c0 = blockIdx.x * BC;
  const int ncol = min(BC, dv - c0);
  const int hq = h / (H / qk_heads);
  int slot = state_slots[s];
  if (slot >= num_slots) {
    if (tid == 0 && blockIdx.x == 0 && h == 0) report_error(err, PHOTON_DEV_BAD_SLOT, s, slot, num_slots);
    slot = -1;
  }
  float* S_h = slot >= 0 ? state + (size_t)slot * state_stride + (size_t)h * N * dv : nullptr;
  const bool wide = vec && c0 + col + LRR_C <= dv;     // all of the lane's columns at a time
  lr_pair S[R / 2][LRR_C];
#pragma unroll
  for (int j = 0; j < R / 2; ++j) {
    float x[2][LRR_C];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = ((j >> 1) * L + sub) * 4 + (j & 1) * 2 + e;
      const float* src = S_h + (size_t)r * dv + c0 + col;
#pragma unroll
      for (int c = 0; c < LRR_C; ++c) x[e][c] = 0.f;
      if (S_h && r < N) {
        if (wide) {
          const LrCols f = *reinterpret_cast<const LrCols*>(src);
#pragma unroll
          for (int c = 0; c < LRR_C; ++c) x[e][c] = f.x[c];
        } else {
#pragma unroll
          for (int c = 0; c < LRR_C; ++c) if (c0 + col + c < dv) x[e][c] = src[c];
        }
      }
    }
#pragma unroll
    for (int c = 0; c < LRR_C; ++c) S[j][c] = lr_make(x[0][c], x[1][c]);
  }
  // what no copy writes: rows beyond N, columns beyond the head
  if (N < NP) for (int i = tid; i < 4 * LR_CHUNK * NP; i += LRR_THREADS) ks[i] = 0.f;
  if (ncol < BC) for (int i = tid; i < 2 * LR_CHUNK * BC; i += LRR_THREADS) vs[i] = 0.f;
  if (N < NP || ncol < BC) __syncthreads();
  const int t0 = cu_tokens[s], t1 = cu_tokens[s + 1];

  // walks the pieces tid, tid + LRR_THREADS .. of `rows` rows of `per` pieces each
  auto pieces = [&](int rows, int per, auto fn) {
    const int dt = LRR_THREADS / per, dr = LRR_THREADS - dt * per;
    int tt = tid / per, r = tid - tt * per;
    for (; tt < rows; tt += dt) {
      fn(tt, r);
      r += dr;
      if (r >= per) { r -= per; ++tt; }
    }
  };
  auto issue = [&](int base, int stage) {
    const int cnt = min(LR_CHUNK, t1 - base);
    float* kd = ks + (size_t)stage * LR_CHUNK * NP;
    float* qd = qs + (size_t)stage * LR_CHUNK * NP;
    float* vd = vs + (size_t)stage * LR_CHUNK * BC;
    const float* kg = k + (size_t)base * k_stride + (size_t)hq * N;
    const float* qg = q + (size_t)base * q_stride + (size_t)hq * N;
    const float* vg = v + (size_t)base * v_stride + (size_t)h * dv + c0;
    if (vec) {
      pieces(cnt, N / 4, [&](int tt, int r) {
        lr_cp16(kd + tt * NP + r * 4, kg + tt * k_stride + r * 4);
        lr_cp16(qd + tt * NP + r * 4, qg + tt * q_stride + r * 4);
      });
      pieces(cnt, ncol / 4, [&](int tt, int c) { lr_cp16(vd + tt * BC + c * 4, vg + tt * v_stride + c * 4); });
    } else {
      pieces(cnt, N, [&](int tt, int r) {
        lr_cp4(kd + tt * NP + r, kg + tt * k_stride + r);
        lr_cp4(qd + tt * NP + r, qg + tt * q_stride + r);
      });
      pieces(cnt, ncol, [&](int tt, int c) { lr_cp4(vd + tt * BC + c, vg + tt * v_stride + c); });
    }
    lr_commit();
  };

  const lr_pair minus = lr_dup(-1.0f);
  // where the first of the sums that this lane is left with stands in a group's rows of os
  int oslot;
  {
    int first = 0, n = LRR_C * TG;
#pragma unroll
    for (int d = L / 2; d > 0; d >>= 1) {
      n = n > 1 ? n / 2 : 0;
      if (sub & d) first += n;
    }
    oslot = first / LRR_C * BC + col + first % LRR_C;
  }
  if (t0 < t1) issue(t0, 0);
  int stage = 0;
  for (int base = t0; base < t1; base += LR_CHUNK, stage ^= 1) {
    const int cnt = min(LR_CHUNK, t1 - base);
    __syncthreads();                                   // the chunk before is written out: the other stage is free
    if (base + LR_CHUNK < t1) { issue(base + LR_CHUNK, stage ^ 1); lr_wait<1>(); } else lr_wait<0>();
    __syncthreads();                                   // this chunk has landed for every thread
    float* kd = ks + (size_t)stage * LR_CHUNK * NP;
    float* qd = qs + (size_t)stage * LR_CHUNK * NP;
    float* vd = vs + (size_t)stage * LR_CHUNK * BC;
    if (bias != nullptr) {                             // q and k arrived as projected
      pieces(cnt, N, [&](int tt, int r) {
        const int at = tt * NP + r;
        qd[at] = lr_silu(qd[at]);
        kd[at] = lr_write_gate(kd[at], bias[(size_t)hq * N + r], lower[(size_t)hq * N + r]);
      });
    }
    if (cnt % TG != 0) {                               // the last tokens' group is filled up: a gate of 0 writes nothing
      const int fill = TG - cnt % TG;
      for (int i = tid; i < fill * NP; i += LRR_THREADS) { kd[cnt * NP + i] = 0.f; qd[cnt * NP + i] = 0.f; }
      for (int i = tid; i < fill * BC; i += LRR_THREADS) vd[cnt * BC + i] = 0.f;
    }
    if (bias != nullptr || cnt % TG != 0) __syncthreads();
    // TG tokens at a time, their read-outs' shares in val
    auto compute = [&](int t, float (&val)[LRR_C * TG]) {
      ulonglong2 k2[TG][R / 4], q2[TG][R / 4];
      LrCols v2[TG];
#pragma unroll
      for (int u = 0; u < TG; ++u) {
        v2[u] = *reinterpret_cast<const LrCols*>(vd + (t + u) * BC + col);
#pragma unroll
        for (int j = 0; j < R / 4; ++j) {
          k2[u][j] = *reinterpret_cast<const ulonglong2*>(kd + (t + u) * NP + (j * L + sub) * 4);
          q2[u][j] = *reinterpret_cast<const ulonglong2*>(qd + (t + u) * NP + (j * L + sub) * 4);
        }
      }
#pragma unroll
      for (int u = 0; u < TG; ++u) {
        lr_pair o[LRR_C], vv[LRR_C];
#pragma unroll
        for (int c = 0; c < LRR_C; ++c) vv[c] = lr_dup(v2[u].x[c]);
#pragma unroll
        for (int j = 0; j < R / 4; ++j) {
#pragma unroll
          for (int c = 0; c < LRR_C; ++c) {
            S[2 * j][c] = lr_fma2(k2[u][j].x, lr_fma2(S[2 * j][c], minus, vv[c]), S[2 * j][c]);       // v - S, one rounding
            S[2 * j + 1][c] = lr_fma2(k2[u][j].y, lr_fma2(S[2 * j + 1][c], minus, vv[c]), S[2 * j + 1][c]);
            o[c] = j == 0 ? lr_mul2(q2[u][j].x, S[0][c]) : lr_fma2(q2[u][j].x, S[2 * j][c], o[c]);
            o[c] = lr_fma2(q2[u][j].y, S[2 * j + 1][c], o[c]);
          }
        }
#pragma unroll
        for (int c = 0; c < LRR_C; ++c) val[LRR_C * u + c] = lr_sum2(o[c]);
      }
    };
    auto meet = [&](int t, float (&val)[LRR_C * TG]) {
      lr_meet<L / 2, LRR_C * TG>(val, sub);
      constexpr int LEFT = LRR_C * TG > L ? LRR_C * TG / L : 1;  // sums a lane is left with
      constexpr int SPARE = LRR_C * TG < L ? L / (LRR_C * TG) : 1;   // lanes that end up with the same sum
      if ((sub & (SPARE - 1)) == 0) {
#pragma unroll
        for (int i = 0; i < LEFT; ++i) os[t * BC + oslot + i / LRR_C * BC + i % LRR_C] = val[i];
      }
    };
    if (cnt == LR_CHUNK) {
      // straight-line code: the shuffles of one group of tokens run beside the arithmetic of the next
      float val[LR_CHUNK / TG][LRR_C * TG];
      compute(0, val[0]);
#pragma unroll
      for (int g = 1; g < LR_CHUNK / TG; ++g) {
        compute(g * TG, val[g]);
        meet((g - 1) * TG, val[g - 1]);
      }
      meet(LR_CHUNK - TG, val[LR_CHUNK / TG - 1]);
    } else {
      for (int t = 0; t < cnt; t += TG) {
        float val[LRR_C * TG];
        compute(t, val);
        meet(t, val);
      }
    }
    __syncthreads();
    float* og = out + (size_t)base * out_stride + (size_t)h * dv + c0;
    pieces(cnt, ncol, [&](int tt, int c) { og[tt * out_stride + c] = os[tt * BC + c] * q_scale; });
  }
  if (S_h) {
#pragma unroll
    for (int j = 0; j < R / 2; ++j) {
      float x[2][LRR_C];
#pragma unroll
      for (int c = 0; c < LRR_C; ++c) lr_split(S[j][c], x[0][c], x[1][c]);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int r = ((j >> 1) * L + sub) * 4 + (j & 1) * 2 + e;
        float* dst = S_h + (size_t)r * dv + c0 + col;
        if (r < N) {
          if (wide) {
            LrCols f;
#pragma unroll
            for (int c = 0; c < LRR_C; ++c) f.x[c] = x[e][c];
            *reinterpret_cast<LrCols*>(dst) = f;
          } else {
#pragma unroll
            for (int c = 0; c < LRR_C; ++c) if (c0 + col + c < dv) dst[c] = x[e][c];
          }
        }
      }
    }
  }
}

template <int L, int R>
static int linrec_rows_go(cudaStream_t stream, const float* q, long q_stride, const float* k, long k_stride, const float* v, long v_stride,
                          const float* bias, const float* lower, float q_scale, const int* cu_tokens, const int* state_slots,
                          float* state, long state_stride, int num_slots, float* out, long out_stride, int S, int H, int qk_heads,
                          int N, int dv, int* err) {
  constexpr int BC = 16 * (32 / L);
  const int vec = N % 4 == 0 && dv % 4 == 0 && q_stride % 4 == 0 && k_stride % 4 == 0 && v_stride % 4 == 0 && state_stride % 4 == 0 &&
                  ((uintptr_t)q & 15) == 0 && ((uintptr_t)k & 15) == 0 && ((uintptr_t)v & 15) == 0 && ((uintptr_t)state & 15) == 0;
  const size_t smem = ((size_t)4 * LR_CHUNK * L * R + 3 * LR_CHUNK * BC) * sizeof(float);
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(linrec_rows_kernel<L, R>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  linrec_rows_kernel<L, R><<<dim3((dv + BC - 1) / BC, H, S), LRR_THREADS, smem, stream>>>(q, q_stride, k, k_stride, v, v_stride, bias, lower,
      q_scale, cu_tokens, state_slots, state, state_stride, num_slots, out, out_stride, H, qk_heads, N, dv, vec, err);
  return launch_status();
}

// q, k: float [T][qk_heads * N] views (row strides in elements); v float [T][H * dv]; ga, gb: float [T][H] views with row
// stride g_stride, the raw gate inputs (mode 0: ga = dt_raw, gb unused; mode 1: ga = i_raw, gb = f_raw).  p0, p1, p2: float
// [H] (mode 0: A_log, dt_bias, D; mode 1: the input gate's bias, the forget gate's bias, unused).  cap: the gates' bound
// (mode 1).  Mode 2: k holds the raw gates z, p0 and p1 float [qk_heads * N] their biases and lower bounds; p0 null: q and k
// hold silu(q) and the write gates already (photon_linrec_gates); ga, gb are not read.  q_scale multiplies the queries.  out float [T][H * dv] (row stride out_stride).  Head h reads query/key head
// h / (H / qk_heads).  state: float [num_slots][state_stride], see the top of the file.
PHOTON_API int photon_linrec(int mode, const float* q, long q_stride, const float* k, long k_stride, const float* v,
                             long v_stride, const float* ga, const float* gb, long g_stride, const float* p0, const float* p1,
                             const float* p2, float cap, float q_scale, const int* cu_tokens, const int* state_slots,
                             float* state, long state_stride, int num_slots, float* out, long out_stride, int S, int H,
                             int qk_heads, int N, int dv, int* err, cudaStream_t stream) {
  if (S <= 0) return 0;
  if (mode < 0 || mode > 2 || (mode == 2 && (p0 == nullptr) != (p1 == nullptr))) return PHOTON_ERR_ARGUMENT;
  if (H <= 0 || qk_heads <= 0 || H % qk_heads || N <= 0 || dv <= 0) return PHOTON_ERR_ARGUMENT;
  if (mode == 1 && !(cap > 0.f)) return PHOTON_ERR_ARGUMENT;
  if (N > 512 || H > 65535 || S > 65535) return PHOTON_ERR_UNSUPPORTED;
  if (mode == 2) {
#define LR_ROWS(L, R) return linrec_rows_go<L, R>(stream, q, q_stride, k, k_stride, v, v_stride, p0, p1, q_scale, cu_tokens, state_slots, \
      state, state_stride, num_slots, out, out_stride, S, H, qk_heads, N, dv, err)
    if (N <= 32) LR_ROWS(8, 4);
    if (N <= 64) LR_ROWS(16, 4);
    if (N <= 128) LR_ROWS(32, 4);
    if (N <= 256) LR_ROWS(32, 8);
    LR_ROWS(32, 16);
  }
  const int rpl = (N + 7) / 8;
  const int real = mode == 1 ? LR_COLS - 1 : LR_COLS;
  dim3 grid((dv + real - 1) / real, H, S);
  if (mode == 0)
    return linrec_launch<0>(rpl, grid, stream, q, q_stride, k, k_stride, v, v_stride, ga, gb, g_stride, p0, p1, p2, cap, q_scale,
                            cu_tokens, state_slots, state, state_stride, num_slots, out, out_stride, H, qk_heads, N, dv, err);
  return linrec_launch<1>(rpl, grid, stream, q, q_stride, k, k_stride, v, v_stride, ga, gb, g_stride, p0, p1, p2, cap, q_scale,
                          cu_tokens, state_slots, state, state_stride, num_slots, out, out_stride, H, qk_heads, N, dv, err);
}
