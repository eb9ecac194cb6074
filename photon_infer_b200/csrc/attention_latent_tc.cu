// Attention of long prompt portions over a latent that has been expanded for the step, on the fifth-generation tensor
// cores (tcgen05, accumulators in tensor memory), bfloat16.
//
// A long portion visits every cached latent many times, so it pays to form the heads' keys W_uk c and values W_uv c of
// the visible rows once (one product, the caller's) and to attend with heads of d + r and v numbers instead of latents
// of hundreds.  The rows of all long requests of a step lie one request behind the other in one matrix, so nothing here
// is paged.  A key is two parts: d numbers of the head's own and r rotated numbers that all heads share; they are never
// joined in memory, and neither are the two parts of a query.
//
// A block owns one head and up to 256 tokens of one request as two tiles of 128 rows, and walks the keys that any of
// them sees in tiles of 128 (a product with N 64 takes the tensor core about as long as one with N 128: tiles of 64 keys
// measured 50 us where these take 38, at 2,048 tokens, 16 heads of 128 + 64 and a window of 1,024):
//   * warp 8 brings both query tiles and then the key tiles and the value tiles in halves (TMA, 128-byte swizzle, zeros
//     beyond d, r, v and the matrix' end) into two rings in shared memory;
//   * one thread of warp 9 issues, for the two query tiles in turn, O += P V (M 128, N 64 * LT_NV, P in tensor memory) and
//     the next S = Q K^T (M 128, N 128), which takes the place of that P;
//   * warps 0-3 and 4-7 own the rows of a query tile each, one row per thread: running maximum and sum in 32-bit, P =
//     exp2(..) as bfloat16 written back over the scores, O rescaled only when a row's maximum has grown by more than
//     2^8.  While one tile's softmax runs, the tensor cores work for the other.
//
// Every wait on an mbarrier is bounded.  When one runs out the block raises an abort flag that all roles poll, records
// PHOTON_DEV_WAIT_TIMEOUT, waits (bounded) for the copies it has in flight, frees its tensor memory and returns.
//
// Compiled per model with -DLT_NU=, -DLT_NR=, -DLT_NV=: 64-wide chunks of d, r and v.
#include "attention_tc.cuh"
#include <math.h>

#ifndef LT_NU
#define LT_NU 1
#endif
#ifndef LT_NR
#define LT_NR 1
#endif
#ifndef LT_NV
#define LT_NV 1
#endif
#define LT_NK (LT_NU + LT_NR)
static_assert(LT_NU >= 1 && LT_NR >= 1 && LT_NK <= 4 && LT_NV >= 1 && LT_NV <= 2, "sizes of the latent prompt attention");

#define LT_ROWS 128                                // rows of a query tile
#define LT_KT 128                                  // keys per tile
#define LT_VH 64                                   // keys per half of a value tile
#define LT_THREADS 320
#define LT_Q_BYTES (LT_ROWS * 128 * LT_NK)         // one query tile
#define LT_K_BYTES (LT_KT * 128 * LT_NK)           // one key tile
#define LT_V_BYTES (LT_VH * 128 * LT_NV)           // half a value tile
#define LT_ROOM (224 * 1024)
#define LT_KST (2 * LT_Q_BYTES + 2 * LT_K_BYTES + 2 * LT_V_BYTES <= LT_ROOM ? 2 : 1)                    // key tiles in the ring
#define LT_VST (2 * LT_Q_BYTES + LT_KST * LT_K_BYTES + 4 * LT_V_BYTES <= LT_ROOM ? 4 : 2)              // halves of value tiles
#define LT_SMEM_BYTES (2 * LT_Q_BYTES + LT_KST * LT_K_BYTES + LT_VST * LT_V_BYTES + 1024 + 256)
static_assert(LT_SMEM_BYTES <= 227 * 1024, "shared memory of a block");
#define LT_TMEM_COLS 512
#define LT_O_COL 256                               // scores: 2 tiles x 128 columns; O: 2 x 128
#define LT_RESCALE_STEP 8.0f
#define LT_MAX_SEQS 64

struct LatentTcSeq {
  int tok0, ntok;                                  // the request's tokens in q and out
  int start;                                       // position of the first of them
  int base, row0;                                  // position of the request's first row in the matrix, and that row
};

struct LatentTcParams {
  bf16* out; long out_stride;                      // [T, heads * v]
  const bf16* gate; long gate_stride;              // may be null: every output times sigmoid(gate)
  int gate_heads;                                  // the gate is one number per head: [T, heads]
  const float* sinks;                              // may be null: [heads], one more key with this score and no value
  int dv, window, tiles_per_seq;
  float scale_log2;
  int* err;
  LatentTcSeq seq[LT_MAX_SEQS];
};

__global__ void __launch_bounds__(LT_THREADS, 1)
attention_latent_tc_kernel(const __grid_constant__ CUtensorMap map_qu, const __grid_constant__ CUtensorMap map_qr,
                           const __grid_constant__ CUtensorMap map_ku, const __grid_constant__ CUtensorMap map_kr,
                           const __grid_constant__ CUtensorMap map_v, const __grid_constant__ LatentTcParams P) {
  const int head = blockIdx.x;
  const int si = blockIdx.y / P.tiles_per_seq;
  const int qtile = P.tiles_per_seq - 1 - (blockIdx.y - si * P.tiles_per_seq);     // most keys first
  const LatentTcSeq q = P.seq[si];
  const int t0 = qtile * 2 * LT_ROWS;              // first token of the block
  if (t0 >= q.ntok) { pdl_wait(); return; }
  const int pos_last = q.start + min(t0 + 2 * LT_ROWS, q.ntok) - 1;
  const int key_lo = (P.window > 0 && q.start + t0 - P.window + 1 > 0) ? q.start + t0 - P.window + 1 : 0;
  const int ntiles = (pos_last - key_lo) / LT_KT + 1;
  const int row_lo = q.row0 + key_lo - q.base;     // matrix row of key key_lo

  extern __shared__ unsigned char lt_dyn[];
  unsigned char* base = reinterpret_cast<unsigned char*>(((uintptr_t)lt_dyn + 1023) & ~(uintptr_t)1023);
  unsigned char* q_s = base;                                           // 2 x query tile
  unsigned char* k_s = q_s + 2 * LT_Q_BYTES;                           // LT_KST key tiles
  unsigned char* v_s = k_s + LT_KST * LT_K_BYTES;                      // LT_VST halves of value tiles
  uint64_t* bars = reinterpret_cast<uint64_t*>(v_s + LT_VST * LT_V_BYTES);
  uint64_t* q_full = bars;
  uint64_t* k_full = bars + 1;                      // [LT_KST] TMA -> MMA
  uint64_t* k_empty = k_full + LT_KST;              // [LT_KST] MMA -> TMA
  uint64_t* v_full = k_empty + LT_KST;              // [LT_VST]
  uint64_t* v_empty = v_full + LT_VST;              // [LT_VST]
  uint64_t* s_full = v_empty + LT_VST;              // [query tile] MMA -> softmax
  uint64_t* p_full = s_full + 2;                    // [query tile] softmax -> MMA (one arrival per warp)
  uint64_t* pv_done = p_full + 2;                   // [query tile] MMA -> softmax: O is up to date
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(pv_done + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    tc_mbar_init(q_full, 1);
    for (int s = 0; s < LT_KST; ++s) { tc_mbar_init(&k_full[s], 1); tc_mbar_init(&k_empty[s], 1); }
    for (int s = 0; s < LT_VST; ++s) { tc_mbar_init(&v_full[s], 1); tc_mbar_init(&v_empty[s], 1); }
    for (int b = 0; b < 2; ++b) { tc_mbar_init(&s_full[b], 1); tc_mbar_init(&p_full[b], 4); tc_mbar_init(&pv_done[b], 1); }
    *abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 9) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(tc_smem(tmem_slot)), "n"(LT_TMEM_COLS) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  pdl_wait();                                       // queries, keys and values come from the kernels before

  if (warp == 8) {
    // ---------------- producer
    if (lane == 0) {
      tc_mbar_expect_tx(q_full, 2 * LT_Q_BYTES);
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        unsigned char* qt = q_s + j * LT_Q_BYTES;
        const int t = q.tok0 + t0 + j * LT_ROWS;
#pragma unroll
        for (int c = 0; c < LT_NU; ++c) tc_tma_load3(qt + c * (LT_ROWS * 128), &map_qu, c * 64, head, t, q_full);
#pragma unroll
        for (int c = 0; c < LT_NR; ++c) tc_tma_load3(qt + (LT_NU + c) * (LT_ROWS * 128), &map_qr, c * 64, head, t, q_full);
      }
      int kn = 0, vn = 0;                           // key tiles and value halves asked for so far
      auto load_k = [&]() -> bool {
        const int s = kn % LT_KST;
        if (!tc_wait(&k_empty[s], ((kn / LT_KST) & 1) ^ 1, abort_flag)) return false;
        unsigned char* dst = k_s + s * LT_K_BYTES;
        const int row = row_lo + kn * LT_KT;
        tc_mbar_expect_tx(&k_full[s], LT_K_BYTES);
#pragma unroll
        for (int c = 0; c < LT_NU; ++c) tc_tma_load3(dst + c * (LT_KT * 128), &map_ku, c * 64, head, row, &k_full[s]);
#pragma unroll
        for (int c = 0; c < LT_NR; ++c) tc_tma_load(dst + (LT_NU + c) * (LT_KT * 128), &map_kr, c * 64, row, &k_full[s]);
        ++kn;
        return true;
      };
      auto load_v = [&]() -> bool {
        const int s = vn % LT_VST;
        if (!tc_wait(&v_empty[s], ((vn / LT_VST) & 1) ^ 1, abort_flag)) return false;
        unsigned char* dst = v_s + s * LT_V_BYTES;
        const int row = row_lo + vn * LT_VH;
        tc_mbar_expect_tx(&v_full[s], LT_V_BYTES);
#pragma unroll
        for (int c = 0; c < LT_NV; ++c) tc_tma_load3(dst + c * (LT_VH * 128), &map_v, c * 64, head, row, &v_full[s]);
        ++vn;
        return true;
      };
      // in the order in which room appears: the scores of tile i free a key tile before the products of tile i free values
      bool ok = true;
      for (int n = 0; n < LT_KST && n < ntiles && ok; ++n) ok = load_k();
      for (int i = 0; i < ntiles && ok; ++i) {
        ok = load_v() && load_v();
        if (ok && kn < ntiles) ok = load_k();
      }
      if (*abort_flag) {
        // copies already issued still write into this block's shared memory: wait for them, bounded
        for (uint32_t w = 0; w < TC_WAIT_LIMIT && !tc_mbar_try(q_full, 0); ++w) {}
        for (int n = (kn > LT_KST ? kn - LT_KST : 0); n < kn; ++n)
          for (uint32_t w = 0; w < TC_WAIT_LIMIT && !tc_mbar_try(&k_full[n % LT_KST], (n / LT_KST) & 1); ++w) {}
        for (int n = (vn > LT_VST ? vn - LT_VST : 0); n < vn; ++n)
          for (uint32_t w = 0; w < TC_WAIT_LIMIT && !tc_mbar_try(&v_full[n % LT_VST], (n / LT_VST) & 1); ++w) {}
      }
    }
  } else if (warp == 9) {
    // ---------------- MMA issuer
    if (lane == 0) {
      const uint32_t idesc_s = tc_idesc(LT_ROWS, LT_KT);
      const uint32_t idesc_o = tc_idesc(LT_ROWS, 64 * LT_NV) | TC_IDESC_B_MN;
      // the scores of key tile i for query tile j; the second query tile is the last to read the keys
      auto issue_scores = [&](int i, int j) -> bool {
        const int s = i % LT_KST;
        if (!tc_wait(&k_full[s], (i / LT_KST) & 1, abort_flag)) return false;
        tc_fence_after();
        const uint32_t q_addr = tc_smem(q_s + j * LT_Q_BYTES), k_addr = tc_smem(k_s + s * LT_K_BYTES);
#pragma unroll
        for (int kk = 0; kk < LT_NK * 4; ++kk)
          tc_mma(tmem_base + j * 128, tc_desc(q_addr + (kk >> 2) * (LT_ROWS * 128) + (kk & 3) * 32),
                 tc_desc(k_addr + (kk >> 2) * (LT_KT * 128) + (kk & 3) * 32), idesc_s, kk > 0 ? 1u : 0u);
        tc_commit(&s_full[j]);
        if (j == 1) tc_commit(&k_empty[s]);
        return true;
      };
      bool ok = tc_wait(q_full, 0, abort_flag);
      if (ok) ok = issue_scores(0, 0) && issue_scores(0, 1);
      for (int i = 0; i < ntiles && ok; ++i) {
        for (int j = 0; j < 2 && ok; ++j) {
          if (!tc_wait(&p_full[j], i & 1, abort_flag)) { ok = false; break; }
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            const int n = 2 * i + half, s = n % LT_VST;
            if (!tc_wait(&v_full[s], (n / LT_VST) & 1, abort_flag)) { ok = false; break; }
            tc_fence_after();
            const uint32_t v_addr = tc_smem(v_s + s * LT_V_BYTES);
#pragma unroll
            for (int kk = 0; kk < LT_VH / 16; ++kk)  // P: 8 columns of packed pairs per 16 keys
              at_mma_ts(tmem_base + LT_O_COL + j * 128, tmem_base + j * 128 + half * 32 + kk * 8,
                        tc_desc_mn(v_addr + kk * 2048, LT_VH * 128, 1024), idesc_o, (n > 0 || kk > 0) ? 1u : 0u);
            if (j == 1) tc_commit(&v_empty[s]);
          }
          if (!ok) break;
          tc_commit(&pv_done[j]);
          // the next scores go where this tile's P was; the tensor core runs the products in the order of issue
          if (i + 1 < ntiles) ok = issue_scores(i + 1, j);
        }
      }
      pdl_launch_dependents();                      // all products of this block are issued
    }
  } else {
    // ---------------- softmax: thread = row of query tile j
    const int j = warp >> 2;
    const int t = t0 + j * LT_ROWS + (threadIdx.x & 127);
    const bool valid = t < q.ntok;
    const int pos = valid ? q.start + t : -1;
    const int lo = (P.window > 0 && pos - P.window + 1 > 0) ? pos - P.window + 1 : 0;
    const uint32_t lane_addr = tmem_base + ((uint32_t)((warp & 3) * 32) << 16);
    const float c = P.scale_log2;
    float m_used = -INFINITY, l = 0.f;
    bool ok = true;
    // the warp goes on or gives up together: tcgen05.ld/st need all of its lanes
    auto wait_all = [&](uint64_t* bar, uint32_t parity) -> bool {
      return __all_sync(0xffffffffu, tc_wait(bar, parity, abort_flag) ? 1 : 0) != 0;
    };
    const uint32_t s_addr = lane_addr + j * 128, o_addr = lane_addr + LT_O_COL + j * 128;
    for (int i = 0; i < ntiles; ++i) {
      if (!wait_all(&s_full[j], i & 1)) { ok = false; break; }
      tc_fence_after();
      const int key_base = key_lo + i * LT_KT;
      uint32_t sv[128];
#pragma unroll
      for (int u = 0; u < 128; u += 32) tc_ld32_issue(s_addr + u, sv + u);
      tc_ld_wait();
      if (!(key_base + LT_KT - 1 <= pos && key_base >= lo)) {
        // keys this row does not see: those before offset a or behind offset b of the tile
        const int a = lo - key_base, b = pos - key_base;
#pragma unroll
        for (int u = 0; u < 128; ++u) sv[u] = (u >= a && u <= b) ? sv[u] : 0xff800000u;       // -inf
      }
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int u = 0; u < 128; u += 8) {
#pragma unroll
        for (int w = 0; w < 4; ++w) mx4[w] = at_max3(mx4[w], __uint_as_float(sv[u + 2 * w]), __uint_as_float(sv[u + 2 * w + 1]));
      }
      const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
      // the maximum in use lags behind the true one by at most LT_RESCALE_STEP
      const float cand = fmaxf(m_used, mx * c);
      float factor = 1.f;
      const bool grow = cand > m_used + LT_RESCALE_STEP;          // also the first finite maximum
      if (grow) { factor = at_exp2(m_used - cand); m_used = cand; l *= factor; }
      const float nsub = (m_used == -INFINITY) ? 0.f : -m_used;
      // P = exp2(score * c - max in use), packed pairs over the scores they came from (32 columns per 64 keys)
      float sum8[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        uint32_t pk[32];
#pragma unroll
        for (int u = 0; u < 64; u += 2) {
          float x0, x1;
          at_fma2(x0, x1, __uint_as_float(sv[half * 64 + u]), __uint_as_float(sv[half * 64 + u + 1]), c, nsub);
          const float p0 = at_exp2(x0), p1 = at_exp2(x1);
          at_add2(sum8[u & 6], sum8[(u & 6) + 1], p0, p1);
          pk[u >> 1] = at_pack(p0, p1);
        }
        tc_st32(s_addr + half * 32, pk);
      }
      l += ((sum8[0] + sum8[1]) + (sum8[2] + sum8[3])) + ((sum8[4] + sum8[5]) + (sum8[6] + sum8[7]));
      if (i > 0 && __any_sync(0xffffffffu, grow)) {
        // O rescale: the products of the tile before must have landed
        if (!wait_all(&pv_done[j], (i - 1) & 1)) { ok = false; break; }
        tc_fence_after();
#pragma unroll 1
        for (int cc = 0; cc < 64 * LT_NV; cc += 32) {
          uint32_t ov[32];
          tc_ld32(o_addr + cc, ov);
#pragma unroll
          for (int u = 0; u < 32; ++u) ov[u] = __float_as_uint(__uint_as_float(ov[u]) * factor);
          tc_st32(o_addr + cc, ov);
        }
      }
      tc_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) tc_mbar_arrive(&p_full[j]);
    }
    if (ok && wait_all(&pv_done[j], (ntiles - 1) & 1)) {
      tc_fence_after();
      if (P.sinks && valid) l += exp2f(fmaf(P.sinks[head], 1.4426950408889634f, -m_used));   // relative to the maximum in use
      float inv = l > 0.f ? 1.f / l : 0.f;
      if (P.gate && P.gate_heads && valid)
        inv = __fdividef(inv, 1.0f + __expf(-__bfloat162float(P.gate[(size_t)(q.tok0 + t) * P.gate_stride + head])));
      bf16* dst = P.out + (size_t)(q.tok0 + t) * P.out_stride + (size_t)head * P.dv;
      const bf16* gt = P.gate && !P.gate_heads ? P.gate + (size_t)(q.tok0 + t) * P.gate_stride + (size_t)head * P.dv : nullptr;
#pragma unroll 1
      for (int cc = 0; cc < 64 * LT_NV; cc += 32) {
        uint32_t ov[32];
        tc_ld32(o_addr + cc, ov);
        if (valid) {
#pragma unroll
          for (int u = 0; u < 32; u += 8) {
            if (cc + u < P.dv) {                    // v is a multiple of 8
              float y[8];
#pragma unroll
              for (int w = 0; w < 8; ++w) y[w] = __uint_as_float(ov[u + w]) * inv;
              if (gt) {
                const uint4 gz = *reinterpret_cast<const uint4*>(gt + cc + u);
                const __nv_bfloat162* gp = reinterpret_cast<const __nv_bfloat162*>(&gz);
#pragma unroll
                for (int w = 0; w < 4; ++w) {
                  const float2 z = __bfloat1622float2(gp[w]);
                  y[2 * w] = __fdividef(y[2 * w], 1.0f + __expf(-z.x));
                  y[2 * w + 1] = __fdividef(y[2 * w + 1], 1.0f + __expf(-z.y));
                }
              }
              *reinterpret_cast<uint4*>(dst + cc + u) = make_uint4(at_pack(y[0], y[1]), at_pack(y[2], y[3]), at_pack(y[4], y[5]), at_pack(y[6], y[7]));
            }
          }
        }
      }
    }
  }
  // ---------------- teardown
  tc_fence_before();
  __syncthreads();
  if (warp == 9) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "n"(LT_TMEM_COLS) : "memory");
  }
  if (threadIdx.x == 0 && *abort_flag) report_error(P.err, PHOTON_DEV_WAIT_TIMEOUT, blockIdx.x, blockIdx.y, 0);
}

// A 3-D map over bf16 [n2][n1][n0] with row strides in elements; boxes of box2 x 1 x 64.
static int lt_map3(CUtensorMap* map, const void* base, long n0, long n1, long n2, long s1, long s2, int box2) {
  EncodeTiledFn fn = encode_fn();
  if (fn == nullptr) return PHOTON_ERR_UNSUPPORTED;
  cuuint64_t dims[3] = {(cuuint64_t)n0, (cuuint64_t)n1, (cuuint64_t)n2};
  cuuint64_t strides[2] = {(cuuint64_t)s1 * 2, (cuuint64_t)s2 * 2};
  cuuint32_t box[3] = {64, 1, (cuuint32_t)box2};
  cuuint32_t estr[3] = {1, 1, 1};
  CUresult r = fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, estr,
                  CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                  CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? 0 : PHOTON_ERR_ARGUMENT;
}

PHOTON_API int photon_attention_latent_tc_chunks(void) { return LT_NU * 100 + LT_NR * 10 + LT_NV; }
PHOTON_API int photon_attention_latent_tc_max_seqs(void) { return LT_MAX_SEQS; }

// q [T][heads][d + r] (row stride q_stride; the d unrotated numbers of every head), q_rot [T][heads][r] contiguous; kv
// [rows][kv_stride]: every row holds heads x d key numbers, then heads x v value numbers; rot_rows: the r shared key numbers of
// every row (row stride rot_stride).  out [T][heads * v]; gate (may be null) [T][heads * v] or, with gate_heads != 0,
// [T][heads] (one number per head, any alignment); sinks (may be null) float [heads].  seqs (host memory): S x (tok0,
// ntok, start, base, row0), see LatentTcSeq; a token at position p sees the rows of positions max(0, p - window + 1) .. p
// (window <= 0: from 0), all of which must be in the matrix.  d, r, v multiples of 8; all pointers and strides 16-byte aligned.
PHOTON_API int photon_attention_latent_tc(const void* q, long q_stride, const void* q_rot, const void* kv, long kv_stride,
                                          const void* rot_rows, long rot_stride, void* out, long out_stride, const void* gate,
                                          long gate_stride, int gate_heads, const float* sinks, const int* seqs, int S, int T,
                                          int rows, int heads, int d, int r, int v, int window, float scale, int* err,
                                          cudaStream_t stream) {
  if (S <= 0 || T <= 0) return 0;
  if (rows <= 0 || heads <= 0 || heads > 65535 || !(scale > 0.f)) return PHOTON_ERR_ARGUMENT;
  if ((d & 7) || (r & 7) || (v & 7) || (d + 63) / 64 != LT_NU || (r + 63) / 64 != LT_NR || (v + 63) / 64 != LT_NV)
    return PHOTON_ERR_UNSUPPORTED;
  if (((uintptr_t)q & 15) || ((uintptr_t)q_rot & 15) || ((uintptr_t)kv & 15) || ((uintptr_t)rot_rows & 15) || ((uintptr_t)out & 15) ||
      (q_stride & 7) || (kv_stride & 7) || (rot_stride & 7) || (out_stride & 7) ||
      (gate && !gate_heads && (((uintptr_t)gate & 15) || (gate_stride & 7))))
    return PHOTON_ERR_ARGUMENT;
  CUtensorMap map_qu, map_qr, map_ku, map_kr, map_v;
  int st = lt_map3(&map_qu, q, d, heads, T, d + r, q_stride, LT_ROWS);
  if (st == 0) st = lt_map3(&map_qr, q_rot, r, heads, T, r, (long)heads * r, LT_ROWS);
  if (st == 0) st = lt_map3(&map_ku, kv, d, heads, rows, d, kv_stride, LT_KT);
  if (st == 0) st = lt_map3(&map_v, (const bf16*)kv + (long)heads * d, v, heads, rows, v, kv_stride, LT_VH);
  if (st == 0) st = make_map(&map_kr, rot_rows, rows, r, rot_stride, LT_KT);
  if (st != 0) return st;
  static bool attr_done = false;
  if (!attr_done) {
    cudaError_t e = cudaFuncSetAttribute(attention_latent_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, LT_SMEM_BYTES);
    if (e != cudaSuccess) return (int)e;
    attr_done = true;
  }
  for (int s0 = 0; s0 < S; s0 += LT_MAX_SEQS) {
    const int n = S - s0 < LT_MAX_SEQS ? S - s0 : LT_MAX_SEQS;
    LatentTcParams P;
    P.out = (bf16*)out; P.out_stride = out_stride; P.gate = (const bf16*)gate; P.gate_stride = gate_stride;
    P.gate_heads = gate_heads; P.sinks = sinks;
    P.dv = v; P.window = window; P.scale_log2 = scale * 1.4426950408889634f; P.err = err;
    int most = 0;
    for (int i = 0; i < n; ++i) {
      const int* e = seqs + (size_t)(s0 + i) * 5;
      P.seq[i].tok0 = e[0]; P.seq[i].ntok = e[1]; P.seq[i].start = e[2]; P.seq[i].base = e[3]; P.seq[i].row0 = e[4];
      const int first = (window > 0 && e[2] - window + 1 > 0) ? e[2] - window + 1 : 0;
      if (e[0] < 0 || e[1] <= 0 || e[0] + e[1] > T || e[2] < 0 || e[3] < 0 || e[3] > first || e[4] < 0 ||
          (long)e[4] + e[2] + e[1] - e[3] > rows)
        return PHOTON_ERR_ARGUMENT;
      if (e[1] > most) most = e[1];
    }
    P.tiles_per_seq = (most + 2 * LT_ROWS - 1) / (2 * LT_ROWS);
    if ((long)n * P.tiles_per_seq > 65535) return PHOTON_ERR_UNSUPPORTED;
    st = launch_pdl(attention_latent_tc_kernel, dim3(heads, n * P.tiles_per_seq), dim3(LT_THREADS), (size_t)LT_SMEM_BYTES, stream,
                    map_qu, map_qr, map_ku, map_kr, map_v, P);
    if (st != 0) return st;
  }
  return 0;
}
