// Kernels of attention over a cached latent: every token stores ONE row [c ; k_r] of kv_rank + rot numbers,
// the normed latent c and a rotated key part k_r shared by all heads.  A head's unrotated key is W_uk c and
// its value W_uv c; neither is ever formed.  With q_abs = W_uk^T q_unrotated the score of a head is
// (q_abs . c + q_r . k_r) * scale, the weighted sum of the latents is taken per head, and W_uv is applied to
// that sum.  The attention itself is photon_paged_attention with one key/value head whose values are the head
// of the key rows; this file holds what comes before and after it:
//
//   photon_latent_prep      one pass over the fused down-projection row of a token: RMS norm of the query
//                           latent, RMS norm of the key/value latent, rotation of the shared key part, and the
//                           row's write into the paged cache;
//   photon_latent_q_rope    the rotated part of every head's query, copied behind the absorbed part;
//   photon_head_linear      out[t, h, :] = W[h] x[t, h, :] for all heads in one launch (the absorption of W_uk
//                           into the queries and the application of W_uv to the attention result).
//
// Rotation: the first rot_dims numbers of the rotated part, feature i paired with i + rot_dims / 2 (or, interleaved,
// feature 2i with 2i + 1), angle position * inv_freq[i] in 32-bit; features beyond rot_dims pass unchanged.  All
// arithmetic is 32-bit.
#include "common.cuh"
#include <math.h>

// Number i of a rotated part x whose token stands at position p.
template <typename T>
__device__ __forceinline__ float rotated(const T* x, int i, int rot_dims, int interleaved, float p,
                                         const float* __restrict__ inv_freq) {
  if (i >= rot_dims) return to_f32(x[i]);
  const int half = rot_dims / 2;
  const bool second = interleaved ? (i & 1) : (i >= half);
  const int pair = interleaved ? (i >> 1) : (second ? i - half : i);
  const int mate = interleaved ? (i ^ 1) : (second ? i - half : i + half);
  float sn, cs;
  sincosf(p * inv_freq[pair], &sn, &cs);
  return second ? to_f32(x[i]) * cs + to_f32(x[mate]) * sn : to_f32(x[i]) * cs - to_f32(x[mate]) * sn;
}

// ---------------------------------------------------------------- norms, rotation, cache write
template <typename T>
__global__ void latent_prep_kernel(const T* __restrict__ down, long down_stride, int q_rank, int kv_rank, int rot,
                                   int rot_dims, int interleaved, const void* __restrict__ qw, int qw_bf16,
                                   const void* __restrict__ kw, int kw_bf16, float eps,
                                   const int* __restrict__ positions, const float* __restrict__ inv_freq,
                                   const int* __restrict__ slot_mapping, T* __restrict__ cq, long cq_stride,
                                   T* __restrict__ cache, long num_slots, int* err) {
  __shared__ float red[64];
  const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarp = blockDim.x >> 5;
  const T* row = down + (size_t)t * down_stride;
  const T* kv = row + q_rank;
  // the sums of squares of both latents in one pass and one reduction, whose order depends on the block's size alone
  float sq = 0.f, sk = 0.f;
#pragma unroll 4
  for (int i = threadIdx.x; i < q_rank; i += blockDim.x) { const float v = to_f32(row[i]); sq += v * v; }
  if (cache != nullptr) {
#pragma unroll 4
    for (int i = threadIdx.x; i < kv_rank; i += blockDim.x) { const float v = to_f32(kv[i]); sk += v * v; }
  }
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if (lane == 0) { red[warp] = sq; red[32 + warp] = sk; }
  __syncthreads();
  sq = warp_sum(lane < nwarp ? red[lane] : 0.f);
  sk = warp_sum(lane < nwarp ? red[32 + lane] : 0.f);
  // query latent
  const float qinv = 1.0f / sqrtf(sq / (float)q_rank + eps);
#pragma unroll 4
  for (int i = threadIdx.x; i < q_rank; i += blockDim.x)
    cq[(size_t)t * cq_stride + i] = from_f32<T>(to_f32(row[i]) * qinv * load_w(qw, qw_bf16, i));
  if (cache == nullptr) return;                         // the layer reads rows that another one has stored
  // key/value latent
  const float kinv = 1.0f / sqrtf(sk / (float)kv_rank + eps);
  const int slot = slot_mapping[t];
  if (slot < 0) return;                                 // a padding row: nothing is stored
  if (slot >= num_slots) {
    if (threadIdx.x == 0) report_error(err, PHOTON_DEV_BAD_SLOT, t, slot, (int)num_slots);
    return;
  }
  T* dst = cache + (size_t)slot * (kv_rank + rot);
#pragma unroll 4
  for (int i = threadIdx.x; i < kv_rank; i += blockDim.x)
    dst[i] = from_f32<T>(to_f32(kv[i]) * kinv * load_w(kw, kw_bf16, i));
  const T* kr = kv + kv_rank;
  const float p = (float)positions[t];
  for (int i = threadIdx.x; i < rot; i += blockDim.x)
    dst[kv_rank + i] = from_f32<T>(rotated(kr, i, rot_dims, interleaved, p, inv_freq));
}

// down [T][q_rank + kv_rank + rot] (row stride in elements): the fused down-projections of a token.
// cq [T][q_rank]: the normed query latent.  cache: [num_slots][kv_rank + rot], the pages of one layer; null: only the
// query latent is formed (the row then needs no key/value part, kv_norm_w and slot_mapping are not read).
PHOTON_API int photon_latent_prep(const void* down, long down_stride, int dtype, int q_rank, int kv_rank, int rot,
                                  int rot_dims, int interleaved, const void* q_norm_w, int q_norm_dtype, const void* kv_norm_w,
                                  int kv_norm_dtype, float eps, const int* positions, const float* inv_freq,
                                  const int* slot_mapping, void* cq, long cq_stride, void* cache, long num_slots,
                                  int T_, int* err, cudaStream_t stream) {
  if (T_ <= 0) return 0;
  if (q_rank <= 0 || kv_rank <= 0 || rot < 0 || rot_dims < 0 || rot_dims > rot || (rot_dims & 1)) return PHOTON_ERR_ARGUMENT;
  const int threads = 256;
  if (dtype == PHOTON_BF16)
    latent_prep_kernel<bf16><<<T_, threads, 0, stream>>>((const bf16*)down, down_stride, q_rank, kv_rank, rot, rot_dims,
        interleaved, q_norm_w, q_norm_dtype == PHOTON_BF16, kv_norm_w, kv_norm_dtype == PHOTON_BF16, eps, positions, inv_freq,
        slot_mapping, (bf16*)cq, cq_stride, (bf16*)cache, num_slots, err);
  else
    latent_prep_kernel<float><<<T_, threads, 0, stream>>>((const float*)down, down_stride, q_rank, kv_rank, rot, rot_dims,
        interleaved, q_norm_w, q_norm_dtype == PHOTON_BF16, kv_norm_w, kv_norm_dtype == PHOTON_BF16, eps, positions, inv_freq,
        slot_mapping, (float*)cq, cq_stride, (float*)cache, num_slots, err);
  return launch_status();
}

// ---------------------------------------------------------------- rotated query parts
// q [T][heads][dim + rot] -> out [T][heads][out_head] at offset out_off: the last rot numbers of every head, rotated.
template <typename T>
__global__ void latent_q_rope_kernel(const T* __restrict__ q, long q_stride, int heads, int dim, int rot, int rot_dims,
                                     int interleaved, const int* __restrict__ positions, const float* __restrict__ inv_freq,
                                     T* __restrict__ out, long out_stride, int out_head, int out_off) {
  const int t = blockIdx.x;
  const float p = (float)positions[t];
  for (int idx = threadIdx.x; idx < heads * rot; idx += blockDim.x) {
    const int h = idx / rot, i = idx - h * rot;
    const T* src = q + (size_t)t * q_stride + (size_t)h * (dim + rot) + dim;
    out[(size_t)t * out_stride + (size_t)h * out_head + out_off + i] =
        from_f32<T>(rotated(src, i, rot_dims, interleaved, p, inv_freq));
  }
}

PHOTON_API int photon_latent_q_rope(const void* q, long q_stride, int dtype, int heads, int dim, int rot, int rot_dims,
                                    int interleaved, const int* positions, const float* inv_freq, void* out, long out_stride,
                                    int out_head, int out_off, int T_, cudaStream_t stream) {
  if (T_ <= 0 || rot <= 0) return 0;
  if (rot_dims < 0 || rot_dims > rot || (rot_dims & 1)) return PHOTON_ERR_ARGUMENT;
  if (dtype == PHOTON_BF16)
    latent_q_rope_kernel<bf16><<<T_, 128, 0, stream>>>((const bf16*)q, q_stride, heads, dim, rot, rot_dims, interleaved, positions,
                                                      inv_freq, (bf16*)out, out_stride, out_head, out_off);
  else
    latent_q_rope_kernel<float><<<T_, 128, 0, stream>>>((const float*)q, q_stride, heads, dim, rot, rot_dims, interleaved, positions,
                                                       inv_freq, (float*)out, out_stride, out_head, out_off);
  return launch_status();
}

// ---------------------------------------------------------------- one product per head
// out[t, h, n] = sum_k x[t, h, k] * W[h, n, k], accumulated in 32-bit as one chain of K fused multiply-adds in
// ascending k (a row's result depends on nothing but the row).  Tiles of 64 tokens x 64 features per block.
#define HL_BM 64
#define HL_BN 64
#define HL_BK 16

template <typename T>
__global__ void __launch_bounds__(256)
head_linear_kernel(const T* __restrict__ x, long x_row, long x_head, const T* __restrict__ W, T* __restrict__ out,
                   long o_row, long o_head, int M, int N, int K, const T* __restrict__ gate, long gate_row, int gate_heads) {
  __shared__ float As[HL_BK][HL_BM + 4];
  __shared__ float Ws[HL_BK][HL_BN + 4];
  const int h = blockIdx.z;
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  const int m0 = blockIdx.y * HL_BM, n0 = blockIdx.x * HL_BN;
  const T* A = x + (size_t)h * x_head;
  const T* Wh = W + (size_t)h * N * K;
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  for (int k0 = 0; k0 < K; k0 += HL_BK) {
#pragma unroll
    for (int r = 0; r < 4; ++r) {
      const int idx = tid + r * 256;
      const int row = idx >> 4, kk = idx & 15;
      const int gm = m0 + row, gn = n0 + row, gk = k0 + kk;
      As[kk][row] = (gm < M && gk < K) ? to_f32(A[(size_t)gm * x_row + gk]) : 0.f;
      Ws[kk][row] = (gn < N && gk < K) ? to_f32(Wh[(size_t)gn * K + gk]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < HL_BK; ++kk) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) a[i] = As[kk][ty * 4 + i];
#pragma unroll
      for (int j = 0; j < 4; ++j) b[j] = Ws[kk][tx * 4 + j];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int gm = m0 + ty * 4 + i;
    if (gm >= M) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int gn = n0 + tx * 4 + j;
      if (gn < N) {
        const float g = gate ? 1.0f + expf(-to_f32(gate[(size_t)gm * gate_row + (gate_heads ? h : (size_t)h * N + gn)])) : 1.0f;
        out[(size_t)gm * o_row + (size_t)h * o_head + gn] = from_f32<T>(gate ? acc[i][j] / g : acc[i][j]);
      }
    }
  }
}

// Few bfloat16 rows (decode steps): W[h] is streamed once, 16 bytes per lane and load, straight into the A fragments of
// mma m16n8k16 (16 features of W against 8 rows of x; HLS_GROUPS groups of 8 rows).  The products run over k in an order
// that suits the loads: lane (g, c) holds k = 32 b + 8 c .. + 7 of feature row g and of x's row g alike, the first four of
// them in one product and the last four in the next.  A block's warps share 16 * (4 / ksplit) features; with ksplit > 1
// they cut k between them and add up in shared memory, in the order of the warps.
// ROPE: the blocks behind the features' copy the rotated query parts of their head (latent_q_rope_kernel).
struct HeadRope {
  const bf16* q; long q_stride;                        // [M][heads][dim + rot]
  const int* positions; const float* inv_freq;
  bf16* out; long out_stride; int out_head, out_off;   // [M][heads][out_head]
  int dim, rot, rot_dims, interleaved;
};

__device__ __forceinline__ void mma_bf16_16816(float* c, uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

#define HLS_ROWS 16
template <int GROUPS>
__global__ void __launch_bounds__(128)
head_linear_skinny_kernel(const bf16* __restrict__ x, long x_row, long x_head, const bf16* __restrict__ W,
                          bf16* __restrict__ out, long o_row, long o_head, int M, int N, int K,
                          const bf16* __restrict__ gate, long gate_row, int gate_heads, int ksplit, int feature_blocks, HeadRope R) {
  __shared__ float part[4][16][GROUPS * 8];
  const int h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if ((int)blockIdx.x >= feature_blocks) {
    for (int idx = threadIdx.x; idx < M * R.rot; idx += blockDim.x) {
      const int m = idx / R.rot, i = idx - m * R.rot;
      const bf16* src = R.q + (size_t)m * R.q_stride + (size_t)h * (R.dim + R.rot) + R.dim;
      R.out[(size_t)m * R.out_stride + (size_t)h * R.out_head + R.out_off + i] =
          __float2bfloat16_rn(rotated(src, i, R.rot_dims, R.interleaved, (float)R.positions[m], R.inv_freq));
    }
    return;
  }
  const int g = lane >> 2, c = lane & 3;
  const int tiles = 4 / ksplit;                              // feature tiles of a block
  const int n0 = (blockIdx.x * tiles + warp / ksplit) * 16;
  const int ks = warp % ksplit;
  const int blocks = (K + 31) / 32, per = (blocks + ksplit - 1) / ksplit;
  const int b0 = ks * per, b1 = min(blocks, b0 + per);
  const bf16* w0 = W + ((size_t)h * N + n0 + g) * K;
  const bf16* w1 = w0 + (size_t)8 * K;
  const bool ok0 = n0 + g < N, ok1 = n0 + g + 8 < N;
  float acc[GROUPS][4];
#pragma unroll
  for (int j = 0; j < GROUPS; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[j][e] = 0.f;
  const uint4 zero = make_uint4(0, 0, 0, 0);
#pragma unroll 4
  for (int b = b0; b < b1; ++b) {
    const int k = b * 32 + c * 8;
    const bool in = k < K;                                   // K is a multiple of 8
    const uint4 a = in && ok0 ? *reinterpret_cast<const uint4*>(w0 + k) : zero;
    const uint4 d = in && ok1 ? *reinterpret_cast<const uint4*>(w1 + k) : zero;
#pragma unroll
    for (int j = 0; j < GROUPS; ++j) {
      const int m = j * 8 + g;
      const uint4 xv = in && m < M ? *reinterpret_cast<const uint4*>(x + (size_t)m * x_row + (size_t)h * x_head + k) : zero;
      mma_bf16_16816(acc[j], a.x, d.x, a.y, d.y, xv.x, xv.y);
      mma_bf16_16816(acc[j], a.z, d.z, a.w, d.w, xv.z, xv.w);
    }
  }
  // acc[j]: features g and g + 8 of rows j * 8 + 2 c, + 1
#pragma unroll
  for (int j = 0; j < GROUPS; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) part[warp][g + (e >> 1) * 8][j * 8 + 2 * c + (e & 1)] = acc[j][e];
  __syncthreads();
  for (int idx = threadIdx.x; idx < tiles * 16 * M; idx += blockDim.x) {
    const int f = idx & 15, m = (idx >> 4) % M, tile = (idx >> 4) / M;
    const int n = (blockIdx.x * tiles + tile) * 16 + f;
    if (n >= N) continue;
    float v = 0.f;
    for (int u = 0; u < ksplit; ++u) v += part[tile * ksplit + u][f][m];
    if (gate) v /= 1.0f + expf(-__bfloat162float(gate[(size_t)m * gate_row + (gate_heads ? h : (size_t)h * N + n)]));
    out[(size_t)m * o_row + (size_t)h * o_head + n] = __float2bfloat16_rn(v);
  }
}

static int head_linear_skinny_launch(const void* x, long x_row, long x_head, const void* W, void* out, long o_row, long o_head,
                                     int M, int heads, int N, int K, const void* gate, long gate_row, int gate_heads, const HeadRope* rope,
                                     cudaStream_t stream) {
  // few features: cut k over the warps of a block, so that there are blocks for most SMs
  int ksplit = 1;
  while (ksplit < 4 && K >= 128 * ksplit && (long)heads * ((N + 64 / ksplit - 1) / (64 / ksplit)) < 2 * photon_sm_count()) ksplit *= 2;
  const int feature_blocks = (N + 64 / ksplit - 1) / (64 / ksplit);
  const dim3 grid(feature_blocks + (rope ? 1 : 0), heads);
  HeadRope r = {};
  if (rope) r = *rope;
  if (M <= 8)
    head_linear_skinny_kernel<1><<<grid, 128, 0, stream>>>((const bf16*)x, x_row, x_head, (const bf16*)W, (bf16*)out, o_row, o_head, M,
                                                         N, K, (const bf16*)gate, gate_row, gate_heads, ksplit, feature_blocks, r);
  else
    head_linear_skinny_kernel<2><<<grid, 128, 0, stream>>>((const bf16*)x, x_row, x_head, (const bf16*)W, (bf16*)out, o_row, o_head, M,
                                                         N, K, (const bf16*)gate, gate_row, gate_heads, ksplit, feature_blocks, r);
  return launch_status();
}

static bool head_linear_skinny_ok(const void* x, long x_row, long x_head, const void* W, int dtype, int M, int heads, int K) {
  return dtype == PHOTON_BF16 && M <= HLS_ROWS && K % 8 == 0 && x_row % 8 == 0 && x_head % 8 == 0 && (uintptr_t)x % 16 == 0 &&
         (uintptr_t)W % 16 == 0 && heads <= 65535;
}

// A decode step's queries into the latent space in one launch: out[m, h, :N] = W[h] q[m, h, :dim] and, behind it at
// out_off, the rotated last rot numbers of the head.  q [M][heads][dim + rot], out [M][heads][out_head], at most 16 rows
// of bfloat16, dim a multiple of 8 (else PHOTON_ERR_UNSUPPORTED: the two separate entry points take every size).
PHOTON_API int photon_latent_absorb(const void* q, long q_stride, int dtype, const void* W, int M, int heads, int dim, int rot,
                                    int rot_dims, int interleaved, const int* positions, const float* inv_freq, int N, void* out,
                                    long out_stride, int out_head, int out_off, cudaStream_t stream) {
  if (M <= 0 || heads <= 0 || N <= 0) return 0;
  if (dim <= 0 || rot <= 0 || rot_dims < 0 || rot_dims > rot || (rot_dims & 1)) return PHOTON_ERR_ARGUMENT;
  if (!head_linear_skinny_ok(q, q_stride, dim + rot, W, dtype, M, heads, dim)) return PHOTON_ERR_UNSUPPORTED;
  const HeadRope r = {(const bf16*)q, q_stride, positions, inv_freq, (bf16*)out, out_stride, out_head, out_off, dim, rot, rot_dims, interleaved};
  return head_linear_skinny_launch(q, q_stride, dim + rot, W, out, out_stride, out_head, M, heads, N, dim, nullptr, 0, 0, &r, stream);
}

// x [M][heads][K] and out [M][heads][N] with row and head strides in elements; W [heads][N][K] contiguous.  gate (may be
// null; the type of x, [M][heads * N] with row stride gate_row): every output is multiplied by sigmoid(gate) before it
// is rounded.  gate_heads != 0: gate is [M][heads], one number for all outputs of a head.
PHOTON_API int photon_head_linear(const void* x, long x_row, long x_head, const void* W, void* out, long o_row,
                                  long o_head, int dtype, int M, int heads, int N, int K, const void* gate, long gate_row,
                                  int gate_heads, cudaStream_t stream) {
  if (M <= 0 || heads <= 0 || N <= 0) return 0;
  if (K <= 0) return PHOTON_ERR_ARGUMENT;
  if (head_linear_skinny_ok(x, x_row, x_head, W, dtype, M, heads, K))
    return head_linear_skinny_launch(x, x_row, x_head, W, out, o_row, o_head, M, heads, N, K, gate, gate_row, gate_heads, nullptr, stream);
  dim3 grid((N + HL_BN - 1) / HL_BN, (M + HL_BM - 1) / HL_BM, heads);
  if (grid.y > 65535 || grid.z > 65535) return PHOTON_ERR_UNSUPPORTED;
  if (dtype == PHOTON_BF16)
    head_linear_kernel<bf16><<<grid, 256, 0, stream>>>((const bf16*)x, x_row, x_head, (const bf16*)W, (bf16*)out, o_row,
                                                      o_head, M, N, K, (const bf16*)gate, gate_row, gate_heads);
  else
    head_linear_kernel<float><<<grid, 256, 0, stream>>>((const float*)x, x_row, x_head, (const float*)W, (float*)out,
                                                       o_row, o_head, M, N, K, (const float*)gate, gate_row, gate_heads);
  return launch_status();
}

// ---------------------------------------------------------------- a request's cached rows, in order
// out[i, :] = the cached row of position first + i of the request whose pages are `table`, for i < count: its latent
// rows as one dense matrix, the operand of the products that attention over a long prompt portion is made of.
// Positions outside [valid_lo, valid_hi) give zero rows (columns of the products that nothing sees).
template <typename T>
__global__ void gather_rows_kernel(const T* __restrict__ cache, const int* __restrict__ table, int page_size,
                                   int num_pages, int width, int first, int valid_lo, int valid_hi, T* __restrict__ out,
                                   int* err) {
  const int p = first + blockIdx.x;
  T* dst = out + (size_t)blockIdx.x * width;
  const bool valid = p >= valid_lo && p < valid_hi;
  const int page = valid ? table[p / page_size] : -1;
  if (page < 0 || page >= num_pages) {
    if (valid && threadIdx.x == 0) report_error(err, PHOTON_DEV_BAD_PAGE, 0, p, page);
    for (int i = threadIdx.x; i < width; i += blockDim.x) dst[i] = from_f32<T>(0.f);
    return;
  }
  const T* src = cache + ((size_t)page * page_size + p % page_size) * width;
  for (int i = threadIdx.x; i < width; i += blockDim.x) dst[i] = src[i];
}

PHOTON_API int photon_gather_rows(const void* cache, int dtype, const int* table, int page_size, int num_pages,
                                  int width, int first, int count, int valid_lo, int valid_hi, void* out, int* err,
                                  cudaStream_t stream) {
  if (count <= 0) return 0;
  if (page_size <= 0 || width <= 0 || first < 0 || valid_lo < 0) return PHOTON_ERR_ARGUMENT;
  if (dtype == PHOTON_BF16)
    gather_rows_kernel<bf16><<<count, 128, 0, stream>>>((const bf16*)cache, table, page_size, num_pages, width, first, valid_lo, valid_hi, (bf16*)out, err);
  else
    gather_rows_kernel<float><<<count, 128, 0, stream>>>((const float*)cache, table, page_size, num_pages, width, first, valid_lo, valid_hi, (float*)out, err);
  return launch_status();
}

// ---------------------------------------------------------------- causal softmax over rows of scores
// scores [rows][ld] float: column c is the key at position first_key + c; row r belongs to the token at position
// first_pos + r / heads, which sees the keys up to its own position and, with window > 0, the last `window` of them.
// probs [rows][ldp] = softmax(scale * scores) over the visible keys, zero elsewhere, up to column `cols`.  sinks [heads]
// (may be null): row r's denominator also holds exp(sinks[r % heads]).  One block per row, 32-bit throughout, rounded once on the way out.
template <typename T>
__global__ void causal_softmax_kernel(const float* __restrict__ scores, long ld, T* __restrict__ probs, long ldp,
                                      int heads, int first_pos, int first_key, int window, int cols, float scale,
                                      const float* __restrict__ sinks) {
  __shared__ float red[32];
  const int r = blockIdx.x;
  const int pos = first_pos + r / heads;
  const int hi = min(cols, pos + 1 - first_key);
  const int lo = window > 0 ? max(0, pos + 1 - window - first_key) : 0;
  const float* s = scores + (size_t)r * ld;
  T* p = probs + (size_t)r * ldp;
  float m = -INFINITY;
  for (int i = lo + threadIdx.x; i < hi; i += blockDim.x) m = fmaxf(m, s[i] * scale);
  m = warp_max(m);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = m;
  __syncthreads();
  m = (threadIdx.x & 31) < (blockDim.x >> 5) ? red[threadIdx.x & 31] : -INFINITY;
  m = warp_max(m);
  float sum = 0.f;
  for (int i = lo + threadIdx.x; i < hi; i += blockDim.x) sum += expf(s[i] * scale - m);
  sum = block_sum(sum, red);
  if (sinks) sum += expf(sinks[r % heads] - m);
  const float inv = 1.0f / sum;
  for (int i = threadIdx.x; i < cols; i += blockDim.x)
    p[i] = from_f32<T>(i >= lo && i < hi ? expf(s[i] * scale - m) * inv : 0.f);
}

PHOTON_API int photon_causal_softmax_rows(const float* scores, long ld, void* probs, long ldp, int dtype, int rows,
                                          int heads, int first_pos, int first_key, int window, int cols, float scale,
                                          const float* sinks, cudaStream_t stream) {
  if (rows <= 0 || cols <= 0) return 0;
  if (heads <= 0 || first_pos < 0 || first_key < 0 || first_key > first_pos) return PHOTON_ERR_ARGUMENT;
  if (dtype == PHOTON_BF16)
    causal_softmax_kernel<bf16><<<rows, 256, 0, stream>>>(scores, ld, (bf16*)probs, ldp, heads, first_pos, first_key, window, cols, scale, sinks);
  else
    causal_softmax_kernel<float><<<rows, 256, 0, stream>>>(scores, ld, (float*)probs, ldp, heads, first_pos, first_key, window, cols, scale, sinks);
  return launch_status();
}

// ---------------------------------------------------------------- decoded tokens on the tensor cores
// All heads of a token attend to the same cached rows, so a decoded token is a (heads x width) by (width x keys)
// product followed by a (heads x keys) by (keys x kv_rank) one.  Block (t, s) takes token t and the s-th 64 keys of
// its request, counted from the block of 64 that holds the first key the token sees (key 0 without a window): the rows come into shared memory once (16-byte loads through the block table) and
// serve every tile of 16 heads; scores = Q C^T with wmma (bfloat16 in, 32-bit accumulate), a softmax over the
// block's keys in 32-bit, P (rounded to bfloat16) times the first kv_rank columns of the same rows.  Every block
// leaves its unnormalised sums [token][head][share][dv] and, behind all of them, the rows' maxima and denominators
// [token][head][share][2]; a second kernel puts the shares of a (token, head) together in their order.
#include <mma.h>
using namespace nvcuda;

#define LD_KEYS 64
#define LD_THREADS 256

// 16 bytes from global to shared memory, asynchronously; zeros where `in` is false.
__device__ __forceinline__ void ld_copy16(void* dst, const void* src, bool in) {
  const int bytes = in ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(bytes) : "memory");
}

__global__ void __launch_bounds__(LD_THREADS)
latent_decode_kernel(const bf16* __restrict__ q, long q_stride, const bf16* __restrict__ cache,
                     const int* __restrict__ block_table, int max_pages, const int* __restrict__ token_seq,
                     const int* __restrict__ positions, int heads, int width, int dv, int page_size, int num_pages,
                     float scale, int window, int splits, float* __restrict__ part, int* err) {
  extern __shared__ __align__(128) unsigned char smem_raw[];
  const int t = blockIdx.x, s = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int ldk = width + 8;                                   // bfloat16 elements; rows of 16 keys stay 32-byte aligned
  bf16* Ks = reinterpret_cast<bf16*>(smem_raw);                // 64 x ldk
  bf16* Qs = Ks + LD_KEYS * ldk;                               // 16 x ldk
  float* Sf = reinterpret_cast<float*>(Qs + 16 * ldk);         // 2 x 16 x 68: both halves of the width
  bf16* Ps = reinterpret_cast<bf16*>(Sf + 2 * 16 * 68);        // 16 x 72
  float* Ot = reinterpret_cast<float*>(Ps + 16 * 72);          // 8 x 16 x 20
  float* ml = part + (size_t)gridDim.x * heads * splits * dv;  // [token][head][share][2]
  const int p = positions[t];
  const int first = window > 0 ? max(0, p + 1 - window) : 0;   // the first key the token sees
  const int k0 = (first / LD_KEYS + s) * LD_KEYS;
  const int nlow = max(0, first - k0);                         // keys of this block that lie before it
  const int nkeys = min(LD_KEYS, p + 1 - k0);                  // keys of this block that the token sees
  if (nkeys <= 0) {                                            // an empty share: the merge skips it
    for (int h = tid; h < heads; h += LD_THREADS) {
      float* dst = ml + (((size_t)t * heads + h) * splits + s) * 2;
      dst[0] = -INFINITY; dst[1] = 0.f;
    }
    return;
  }
  const int* table = block_table + (size_t)token_seq[t] * max_pages;
  const int vecs = width / 8;
  // where each of the block's rows lies, looked up once; the loads of the rows then depend on nothing but this list
  long long* rowbase = reinterpret_cast<long long*>(Ot + 8 * 16 * 20);
  if (tid < LD_KEYS) {
    long long base = -1;
    if (tid >= nlow && tid < nkeys) {
      const int kk = k0 + tid;
      const int page = table[kk / page_size];
      if (page < 0 || page >= num_pages) report_error(err, PHOTON_DEV_BAD_PAGE, t, kk, page);
      else base = ((long long)page * page_size + kk % page_size) * width;
    }
    rowbase[tid] = base;
  }
  __syncthreads();
  for (int i = tid; i < LD_KEYS * vecs; i += LD_THREADS) {     // all copies of a block in flight at once
    const int key = i / vecs, j = (i - key * vecs) * 8;
    const long long base = rowbase[key];
    ld_copy16(Ks + key * ldk + j, cache + (base >= 0 ? base + j : 0), base >= 0);
  }
  for (int h0 = 0; h0 < heads; h0 += 16) {
    __syncthreads();                                           // the last tile of heads is done with Qs
    for (int i = tid; i < 16 * vecs; i += LD_THREADS) {
      const int h = i / vecs, j = (i - h * vecs) * 8;
      const bool in = h0 + h < heads;
      ld_copy16(Qs + h * ldk + j, q + (size_t)t * q_stride + (size_t)(in ? h0 + h : 0) * width + j, in);
    }
    asm volatile("cp.async.wait_all;" ::: "memory");           // the rows (first pass) and the queries are in
    __syncthreads();
    {   // scores of 16 heads x 16 keys per warp, over one half of the width
      const int kt = warp & 3, half = warp >> 2, steps = width / 16, mid = (steps + 1) / 2;
      wmma::fragment<wmma::accumulator, 16, 16, 16, float> acc;
      wmma::fill_fragment(acc, 0.f);
      for (int k = half ? mid : 0; k < (half ? steps : mid); ++k) {
        wmma::fragment<wmma::matrix_a, 16, 16, 16, bf16, wmma::row_major> a;
        wmma::fragment<wmma::matrix_b, 16, 16, 16, bf16, wmma::col_major> b;
        wmma::load_matrix_sync(a, Qs + k * 16, ldk);
        wmma::load_matrix_sync(b, Ks + (size_t)kt * 16 * ldk + k * 16, ldk);
        wmma::mma_sync(acc, a, b, acc);
      }
      wmma::store_matrix_sync(Sf + half * 16 * 68 + kt * 16, acc, 68, wmma::mem_row_major);
    }
    __syncthreads();
    {   // softmax over the block's keys: sixteen lanes a row, four keys a lane
      const int row = tid >> 4, c0 = (tid & 15) * 4;
      float v[4], m = -INFINITY;
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const int i = row * 68 + c0 + u;
        v[u] = c0 + u >= nlow && c0 + u < nkeys ? (Sf[i] + Sf[16 * 68 + i]) * scale : -INFINITY;
        m = fmaxf(m, v[u]);
      }
      for (int d = 1; d < 16; d <<= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, d));
      float l = 0.f;
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const float e = v[u] == -INFINITY ? 0.f : expf(v[u] - m);
        l += e;
        Ps[row * 72 + c0 + u] = __float2bfloat16_rn(e);
      }
      for (int d = 1; d < 16; d <<= 1) l += __shfl_xor_sync(0xffffffffu, l, d);
      if ((tid & 15) == 0 && h0 + row < heads) {
        float* dst = ml + (((size_t)t * heads + h0 + row) * splits + s) * 2;
        dst[0] = m; dst[1] = l;
      }
    }
    __syncthreads();
    for (int nt = warp; nt < dv / 16; nt += LD_THREADS / 32) { // 16 heads x 16 value columns per tile
      wmma::fragment<wmma::accumulator, 16, 16, 16, float> acc;
      wmma::fill_fragment(acc, 0.f);
#pragma unroll
      for (int kk = 0; kk < LD_KEYS; kk += 16) {
        wmma::fragment<wmma::matrix_a, 16, 16, 16, bf16, wmma::row_major> a;
        wmma::fragment<wmma::matrix_b, 16, 16, 16, bf16, wmma::row_major> b;
        wmma::load_matrix_sync(a, Ps + kk, 72);
        wmma::load_matrix_sync(b, Ks + (size_t)kk * ldk + nt * 16, ldk);
        wmma::mma_sync(acc, a, b, acc);
      }
      float* dst = part + (((size_t)t * heads + h0) * splits + s) * dv + nt * 16;
      if (h0 + 16 <= heads) {
        wmma::store_matrix_sync(dst, acc, splits * dv, wmma::mem_row_major);
      } else {                                                 // the last heads fill part of a tile
        float* stage = Ot + warp * 16 * 20;
        wmma::store_matrix_sync(stage, acc, 20, wmma::mem_row_major);
        __syncwarp();
        for (int e = lane; e < 256; e += 32) {
          const int h = e >> 4, c = e & 15;
          if (h0 + h < heads) dst[(size_t)h * splits * dv + c] = stage[h * 20 + c];
        }
        __syncwarp();
      }
    }
  }
}

// One block per (token, head).  A token's shares that hold keys come first, so the sums run over those alone.
#define LM_THREADS 128
__global__ void __launch_bounds__(LM_THREADS)
latent_merge_kernel(const float* __restrict__ part, int splits, int dv, bf16* __restrict__ out, long out_stride, int heads,
                    const float* __restrict__ sinks) {
  __shared__ float wgt[LM_THREADS];
  const int t = blockIdx.x, h = blockIdx.y, lane = threadIdx.x & 31;
  const size_t row = (size_t)t * heads + h;
  const float* ml = part + (size_t)gridDim.x * heads * splits * dv + row * splits * 2;
  const float* src = part + row * splits * dv;
  // every warp forms the maximum, the denominator and the number of shares by itself
  float m = -INFINITY;
  for (int s = lane; s < splits; s += 32) m = fmaxf(m, ml[2 * s]);
  m = warp_max(m);
  float l = 0.f;
  int used = 0;
  for (int s = lane; s < splits; s += 32) {
    const float ms = ml[2 * s];
    if (ms != -INFINITY) { l += ml[2 * s + 1] * expf(ms - m); ++used; }
  }
  l = warp_sum(l);
  if (sinks) l += expf(sinks[h] - m);                          // one more key with this score and no value
  for (int d = 16; d > 0; d >>= 1) used += __shfl_xor_sync(0xffffffffu, used, d);
  const float inv = l > 0.f ? 1.0f / l : 0.f;
  for (int j0 = 0; j0 < dv; j0 += LM_THREADS * 4) {
    const int j = j0 + threadIdx.x * 4;
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int s0 = 0; s0 < used; s0 += LM_THREADS) {
      const int n = min(LM_THREADS, used - s0);
      __syncthreads();
      if ((int)threadIdx.x < n) wgt[threadIdx.x] = expf(ml[2 * (s0 + threadIdx.x)] - m) * inv;
      __syncthreads();
      if (j < dv) {
#pragma unroll 4
        for (int s = 0; s < n; ++s) {
          const float4 v = *reinterpret_cast<const float4*>(src + (size_t)(s0 + s) * dv + j);
          const float w = wgt[s];
          a.x = fmaf(w, v.x, a.x); a.y = fmaf(w, v.y, a.y); a.z = fmaf(w, v.z, a.z); a.w = fmaf(w, v.w, a.w);
        }
      }
    }
    if (j < dv) {
      bf16* dst = out + (size_t)t * out_stride + (size_t)h * dv + j;
      dst[0] = __float2bfloat16_rn(a.x); dst[1] = __float2bfloat16_rn(a.y);
      dst[2] = __float2bfloat16_rn(a.z); dst[3] = __float2bfloat16_rn(a.w);
    }
  }
}

// q [T][heads * width] bfloat16 (row stride in elements), cache [num_pages * page_size][width] bfloat16, out
// [T][heads * dv]: token t at position positions[t] of request token_seq[t] sees the rows 0 .. positions[t], with
// window > 0 the last `window` of them; a row's value is its first dv numbers.  width and dv multiples of 16.  splits >=
// ceil((largest position + 1) / 64), with a window no more than ceil((window - 1) / 64) + 1 are needed;
// part: float [T * heads * splits * (dv + 2)].  sinks (float [heads], may be null): the softmax of head h has one more key
// with the score sinks[h] (not scaled) and no value.
PHOTON_API int photon_latent_decode_attention(const void* q, long q_stride, const void* cache, const int* block_table,
                                              int max_pages, const int* token_seq, const int* positions, int T_,
                                              int heads, int width, int dv, int page_size, int num_pages, float scale,
                                              int window, int splits, float* part, void* out, long out_stride,
                                              const float* sinks, int* err, cudaStream_t stream) {
  if (T_ <= 0) return 0;
  if (heads <= 0 || splits <= 0 || part == nullptr || dv > width) return PHOTON_ERR_ARGUMENT;
  if (width % 16 || dv % 16 || q_stride % 8 || (uintptr_t)q % 16 || (uintptr_t)cache % 16 || (uintptr_t)part % 32 || splits > 65535 || heads > 65535)
    return PHOTON_ERR_UNSUPPORTED;
  const size_t smem = (size_t)(LD_KEYS + 16) * (width + 8) * 2 + 2 * 16 * 68 * 4 + 16 * 72 * 2 + 8 * 16 * 20 * 4 + LD_KEYS * 8;
  if (smem > 220 * 1024) return PHOTON_ERR_UNSUPPORTED;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(latent_decode_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  latent_decode_kernel<<<dim3(T_, splits), LD_THREADS, smem, stream>>>((const bf16*)q, q_stride, (const bf16*)cache, block_table,
      max_pages, token_seq, positions, heads, width, dv, page_size, num_pages, scale, window, splits, part, err);
  int st = launch_status();
  if (st != 0) return st;
  latent_merge_kernel<<<dim3(T_, heads), LM_THREADS, 0, stream>>>(part, splits, dv, (bf16*)out, out_stride, heads, sinks);
  return launch_status();
}
