// Parallel residual streams: every token has S rows X_1 .. X_S of H numbers instead of one.  A sublayer reads
// u = sum_s a[s] X_s through its norm, and its output y is written back as X_t <- sum_s M[s][t] X_s + b[t] y, all
// streams at once from the old ones.
//
//   photon_stream_norm   writes what is pending (M, b, y of the sublayer before), reads u with the a of the sublayer
//                        that follows, and norms u, in ONE pass over the token's rows.
//
// The S rows of a token lie one after the other, [T][S][H] float.  A step starts with all streams equal: the kernel
// then reads one row [T][H] in the place of all of them (stream stride 0) and the first write spreads them out.
// All arithmetic is 32-bit; only the normed row is rounded.
#include "common.cuh"

#define HY_MAX_STREAMS 16

template <typename T> struct Four;            // four consecutive numbers as one load or store
template <> struct Four<float> {
  __device__ static void load(const float* p, float* f) { const float4 r = *reinterpret_cast<const float4*>(p); f[0] = r.x; f[1] = r.y; f[2] = r.z; f[3] = r.w; }
  __device__ static void store(float* p, const float* f) { *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]); }
};
template <> struct Four<bf16> {
  __device__ static void load(const bf16* p, float* f) {
    const uint2 r = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
  }
  __device__ static void store(bf16* p, const float* f) {
    __nv_bfloat162 a = __floats2bfloat162_rn(f[0], f[1]), b = __floats2bfloat162_rn(f[2], f[3]);
    uint2 r;
    r.x = *reinterpret_cast<uint32_t*>(&a);
    r.y = *reinterpret_cast<uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = r;
  }
};

// One block per token (or per entry of `rows`).  MS: streams held in registers (S <= MS).  V: numbers per thread and
// step (4 with aligned rows, else 1).  src and dst may be the same buffer: a thread writes only the numbers it read.
template <typename TY, typename TO, int MS, int V>
__global__ void stream_norm_kernel(const float* src, long src_token, long src_stream, float* dst, const TY* y,
                                   const float* __restrict__ mix, const float* __restrict__ wout,
                                   const float* __restrict__ win, int S, int H, const void* __restrict__ w, int w_bf16,
                                   const void* __restrict__ bias, int bias_bf16, int center, float eps, TO* out,
                                   const int* rows) {
  __shared__ float red[32];
  __shared__ float cm[MS * MS], cb[MS], ca[MS];
  extern __shared__ __align__(16) float stash[];               // H floats: u
  for (int i = threadIdx.x; i < S * S; i += blockDim.x) cm[i] = mix ? mix[i] : 0.f;
  for (int i = threadIdx.x; i < S; i += blockDim.x) { cb[i] = wout ? wout[i] : 0.f; ca[i] = win ? win[i] : 1.f; }
  __syncthreads();
  pdl_wait();                                                  // the weights above are not written by earlier kernels
  const int r = rows ? rows[blockIdx.x] : blockIdx.x;
  const float* x = src + (size_t)r * src_token;
  float* xo = dst ? dst + (size_t)r * S * H : nullptr;
  const TY* yr = y ? y + (size_t)r * H : nullptr;
  float sum = 0.f;
  for (int i = threadIdx.x * V; i < H; i += blockDim.x * V) {
    float v[MS][V], u[V];
    float yv[V];
#pragma unroll
    for (int s = 0; s < MS; ++s) {
      if (s < S) {
        const float* p = x + (size_t)s * src_stream + i;
        if (V == 4) Four<float>::load(p, v[s]); else v[s][0] = *p;
      }
    }
#pragma unroll
    for (int e = 0; e < V; ++e) u[e] = 0.f;
    if (yr) {
      if (V == 4) Four<TY>::load(yr + i, yv); else yv[0] = to_f32(yr[i]);
#pragma unroll
      for (int t = 0; t < MS; ++t) {
        if (t < S) {
          float n[V];
#pragma unroll
          for (int e = 0; e < V; ++e) n[e] = cb[t] * yv[e];
#pragma unroll
          for (int s = 0; s < MS; ++s) {
            if (s < S) {
              const float m = cm[s * S + t];
#pragma unroll
              for (int e = 0; e < V; ++e) n[e] = fmaf(m, v[s][e], n[e]);
            }
          }
          if (xo) { if (V == 4) Four<float>::store(xo + (size_t)t * H + i, n); else xo[(size_t)t * H + i] = n[0]; }
#pragma unroll
          for (int e = 0; e < V; ++e) u[e] = fmaf(ca[t], n[e], u[e]);
        }
      }
    } else {
#pragma unroll
      for (int s = 0; s < MS; ++s) {
        if (s < S) {
#pragma unroll
          for (int e = 0; e < V; ++e) u[e] = fmaf(ca[s], v[s][e], u[e]);
        }
      }
    }
    if (V == 4) Four<float>::store(stash + i, u); else stash[i] = u[0];
#pragma unroll
    for (int e = 0; e < V; ++e) sum += center ? u[e] : u[e] * u[e];
  }
  float mean = 0.f, ss;
  sum = block_sum(sum, red);
  if (center) {                                                // a thread reads back what it stored itself
    mean = sum / (float)H;
    ss = 0.f;
    for (int i = threadIdx.x * V; i < H; i += blockDim.x * V) {
#pragma unroll
      for (int e = 0; e < V; ++e) { const float c = stash[i + e] - mean; ss += c * c; }
    }
    ss = block_sum(ss, red);
  } else {
    ss = sum;
  }
  pdl_launch_dependents();
  const float inv = 1.0f / sqrtf(ss / (float)H + eps);
  TO* o = out + (size_t)blockIdx.x * H;
  for (int i = threadIdx.x * V; i < H; i += blockDim.x * V) {
    float q[V];
#pragma unroll
    for (int e = 0; e < V; ++e)
      q[e] = (stash[i + e] - mean) * inv * load_w(w, w_bf16, i + e) + (bias ? load_w(bias, bias_bf16, i + e) : 0.f);
    if (V == 4) Four<TO>::store(o + i, q); else o[i] = from_f32<TO>(q[0]);
  }
}

template <typename TY, typename TO, int MS>
static int stream_norm_launch(const float* src, long src_token, long src_stream, float* dst, const void* y, const float* mix,
                              const float* wout, const float* win, int S, int H, const void* w, int w_bf16, const void* bias,
                              int bias_bf16, int center, float eps, void* out, const int* rows, int n, cudaStream_t stream) {
  const size_t smem = (size_t)H * sizeof(float);
  if (smem > 200 * 1024) return PHOTON_ERR_UNSUPPORTED;
  const bool vec = (H % 4 == 0) && (src_token % 4 == 0) && (src_stream % 4 == 0) && ((uintptr_t)src % 16 == 0) &&
                   ((uintptr_t)dst % 16 == 0) && ((uintptr_t)y % 16 == 0) && ((uintptr_t)out % 16 == 0);
  auto kernel = vec ? stream_norm_kernel<TY, TO, MS, 4> : stream_norm_kernel<TY, TO, MS, 1>;
  if (smem > 40 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  int threads = 64;
  while (threads < 512 && threads * 4 < H) threads <<= 1;      // depends on H only
  return launch_pdl(kernel, dim3(n), dim3(threads), smem, stream, src, src_token, src_stream, dst, (const TY*)y, mix, wout,
                    win, S, H, w, w_bf16, bias, bias_bf16, center, eps, (TO*)out, rows);
}

// src: the streams of token t start at src + t * src_token, stream s lies src_stream behind (0: all streams equal).
// y [T][H] of y_dtype with mix [S][S] ([from][to]) and wout [S]: the pending write (y null: none; dst is then not used).
// dst (may be null: the new streams are not kept): [T][S][H], may be src.  win [S] (null: all ones, the sum of the
// streams): u = sum_s win[s] X_s.  out [n][H] = norm(u) * w + bias: center != 0 a layer norm, else an RMS norm; bias may
// be null.  rows (may be null) [n]: only these tokens are read; nothing is written back (dst must be null).
PHOTON_API int photon_stream_norm(const float* src, long src_token, long src_stream, float* dst, const void* y, int y_dtype,
                                  const float* mix, const float* wout, const float* win, int S, int H, const void* w,
                                  int w_dtype, const void* bias, int bias_dtype, int center, float eps, void* out,
                                  int out_dtype, const int* rows, int n, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (S <= 0 || H <= 0 || (y != nullptr && (mix == nullptr || wout == nullptr)) || (rows != nullptr && dst != nullptr))
    return PHOTON_ERR_ARGUMENT;
  if (S > HY_MAX_STREAMS) return PHOTON_ERR_UNSUPPORTED;
  if (y == nullptr) { dst = nullptr; y_dtype = out_dtype; }
#define HY_GO(TY, TO, MS) return stream_norm_launch<TY, TO, MS>(src, src_token, src_stream, dst, y, mix, wout, win, S, H, w, \
      w_dtype == PHOTON_BF16, bias, bias_dtype == PHOTON_BF16, center, eps, out, rows, n, stream)
#define HY_STREAMS(TY, TO) do { if (S <= 2) HY_GO(TY, TO, 2); if (S <= 3) HY_GO(TY, TO, 3); if (S <= 4) HY_GO(TY, TO, 4); \
      if (S <= 8) HY_GO(TY, TO, 8); HY_GO(TY, TO, 16); } while (0)
  if (y_dtype == PHOTON_BF16 && out_dtype == PHOTON_BF16) HY_STREAMS(bf16, bf16);
  if (y_dtype == PHOTON_F32 && out_dtype == PHOTON_F32) HY_STREAMS(float, float);
  if (y_dtype == PHOTON_F32 && out_dtype == PHOTON_BF16) HY_STREAMS(float, bf16);
  if (y_dtype == PHOTON_BF16 && out_dtype == PHOTON_F32) HY_STREAMS(bf16, float);
  return PHOTON_ERR_ARGUMENT;
}
