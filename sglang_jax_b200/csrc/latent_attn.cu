// Latent attention with any sizes (latent width R, rotary width, heads, head and value widths), in bf16 or fp32, around
// the paged latent cache  [pages, P, row]  (row >= R + rotary lanes):
//
//   latent_prep       one pass over a step's fused projection: RMS-normalises the latent, rotates the shared key part
//                     and the queries' rotary part (interleaved pairs, fp32 angles), writes the cache rows
//   latent_attn_any   absorbed attention of single query tokens on the CUDA cores, everything in fp32: the fp32 mode,
//                     and bf16 sizes that the tensor-core kernels (mla.cu, latent_extend.cu) do not take
//   latent_gather     cache rows of whole sequences -> contiguous latents and key parts (input of the prefill kernel)
//
// Compiled without fast-math substitutions.
#include <math.h>

#include "common.cuh"

namespace sglb {
namespace {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

constexpr int kPrepThreads = 128;

// One CTA per token.  `proj` is the fused projection [T, ld]: query heads at column q_off, [latent | key part] at dkv_off.
template <typename T>
__global__ void __launch_bounds__(kPrepThreads)
latent_prep_kernel(T* __restrict__ proj, long long ld, int q_off, int dkv_off, int H, int dim, int rot, int R,
                   const float* __restrict__ norm_w, float eps, const float* __restrict__ cos_sin,
                   const int* __restrict__ positions, const int* __restrict__ loc, T* __restrict__ cache,
                   int row_elems) {
  __shared__ float red[kPrepThreads / 32];
  pdl_wait();
  const int t = blockIdx.x, tid = threadIdx.x, half = rot / 2;
  T* row = proj + static_cast<long long>(t) * ld;
  const float* cs = cos_sin + static_cast<long long>(positions[t]) * rot;
  T* dst = cache + static_cast<long long>(loc[t]) * row_elems;
  const T* lat = row + dkv_off;
  float ss = 0.f;
  for (int i = tid; i < R; i += kPrepThreads) {
    const float v = to_f(lat[i]);
    ss += v * v;
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int i = 0; i < kPrepThreads / 32; ++i) tot += red[i];
  const float inv = 1.f / sqrtf(tot / R + eps);
  for (int i = tid; i < R; i += kPrepThreads) dst[i] = from_f<T>(to_f(lat[i]) * inv * norm_w[i]);
  for (int i = tid; i < half; i += kPrepThreads) {
    const float u = to_f(lat[R + 2 * i]), v = to_f(lat[R + 2 * i + 1]), c = cs[i], s = cs[half + i];
    dst[R + 2 * i] = from_f<T>(u * c - v * s);
    dst[R + 2 * i + 1] = from_f<T>(v * c + u * s);
  }
  for (int j = tid; j < H * half; j += kPrepThreads) {
    const int h = j / half, i = j - h * half;
    T* q = row + q_off + static_cast<long long>(h) * (dim + rot) + dim + 2 * i;
    const float u = to_f(q[0]), v = to_f(q[1]), c = cs[i], s = cs[half + i];
    q[0] = from_f<T>(u * c - v * s);
    q[1] = from_f<T>(v * c + u * s);
  }
}

// ---------------------------------------------------------------------------------------------
// One CTA per (query token, head): online softmax over tiles of 64 cached tokens.
constexpr int kAnyThreads = 128;
constexpr int kAnyTile = 64;
constexpr int kAnyMaxAcc = 8;                 // latent width up to 8 * 128

template <typename T>
__global__ void __launch_bounds__(kAnyThreads)
latent_attn_any_kernel(const T* __restrict__ q_lat, const T* __restrict__ q_pe, long long pe_token_stride,
                       int pe_head_stride, const T* __restrict__ cache, int row_elems,
                       const int* __restrict__ page_table, int max_pages, int page_size, const int* __restrict__ rows,
                       const int* __restrict__ kv_lens, T* __restrict__ out, int H, int R, int rot, float scale) {
  extern __shared__ float sm[];
  float* qs = sm;                             // [R + rot]
  float* sc = sm + R + rot;                   // [kAnyTile]
  int* slot = reinterpret_cast<int*>(sc + kAnyTile);
  pdl_wait();
  const int n = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int len = kv_lens[n];
  const int* pt = page_table + static_cast<long long>(rows[n]) * max_pages;
  const long long nh = static_cast<long long>(n) * H + h;
  for (int i = tid; i < R; i += kAnyThreads) qs[i] = to_f(q_lat[nh * R + i]);
  for (int i = tid; i < rot; i += kAnyThreads)
    qs[R + i] = to_f(q_pe[n * pe_token_stride + static_cast<long long>(h) * pe_head_stride + i]);
  float acc[kAnyMaxAcc];
#pragma unroll
  for (int i = 0; i < kAnyMaxAcc; ++i) acc[i] = 0.f;
  float m = -INFINITY, l = 0.f;
  const int D = R + rot;
  for (int k0 = 0; k0 < len; k0 += kAnyTile) {
    const int nk = min(kAnyTile, len - k0);
    __syncthreads();                          // qs written / the previous tile's scores and slots read
    if (tid < nk) {
      const int pg = (k0 + tid) / page_size;
      slot[tid] = pt[pg] * page_size + (k0 + tid - pg * page_size);
    }
    __syncthreads();
    for (int j = warp; j < nk; j += kAnyThreads / 32) {
      const T* kr = cache + static_cast<long long>(slot[j]) * row_elems;
      float a = 0.f;
      for (int i = lane; i < D; i += 32) a += qs[i] * to_f(kr[i]);
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) a += __shfl_xor_sync(0xffffffffu, a, o);
      if (lane == 0) sc[j] = a * scale;
    }
    __syncthreads();
    float mx = m;
    for (int j = 0; j < nk; ++j) mx = fmaxf(mx, sc[j]);
    const float corr = expf(m - mx);
    l *= corr;
#pragma unroll
    for (int i = 0; i < kAnyMaxAcc; ++i) acc[i] *= corr;
    for (int j = 0; j < nk; ++j) {
      const float p = expf(sc[j] - mx);
      l += p;
      const T* kr = cache + static_cast<long long>(slot[j]) * row_elems;
#pragma unroll
      for (int i = 0; i < kAnyMaxAcc; ++i) {
        const int d = tid + i * kAnyThreads;
        if (d < R) acc[i] += p * to_f(kr[d]);
      }
    }
    m = mx;
  }
  const float inv = l > 0.f ? 1.f / l : 0.f;
#pragma unroll
  for (int i = 0; i < kAnyMaxAcc; ++i) {
    const int d = tid + i * kAnyThreads;
    if (d < R) out[nh * R + d] = from_f<T>(acc[i] * inv);
  }
}

// ctx row r of sequence b (ctx_start[b] <= r < ctx_start[b + 1]) is the sequence's token r - ctx_start[b].
__global__ void latent_gather_kernel(__nv_bfloat16* __restrict__ lat, __nv_bfloat16* __restrict__ pe,
                                     const __nv_bfloat16* __restrict__ cache, int row_elems,
                                     const int* __restrict__ page_table, int max_pages, int page_size,
                                     const int* __restrict__ rows, const int* __restrict__ ctx_start, int B, int total,
                                     int R, int rot) {
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int r = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (r >= total) return;
  int lo = 0, hi = B - 1;
  while (lo < hi) {                           // last sequence that starts at or before r
    const int mid = (lo + hi + 1) >> 1;
    if (ctx_start[mid] <= r) lo = mid;
    else hi = mid - 1;
  }
  const int pos = r - ctx_start[lo], pg = pos / page_size;
  const int slot = page_table[static_cast<long long>(rows[lo]) * max_pages + pg] * page_size + (pos - pg * page_size);
  const uint4* src = reinterpret_cast<const uint4*>(cache + static_cast<long long>(slot) * row_elems);
  uint4* d0 = reinterpret_cast<uint4*>(lat + static_cast<long long>(r) * R);
  uint4* d1 = reinterpret_cast<uint4*>(pe + static_cast<long long>(r) * rot);
  for (int i = lane; i < (R + rot) / 8; i += 32) {
    if (i < R / 8) d0[i] = src[i];
    else d1[i - R / 8] = src[i];
  }
}

template <typename T>
int attn_any(const void* q_lat, const void* q_pe, long long pe_token_stride, int pe_head_stride, const void* cache,
             int row_elems, const int* page_table, int max_pages, int page_size, const int* rows, const int* kv_lens,
             void* out, int N, int H, int R, int rot, float scale, cudaStream_t s) {
  const size_t smem = (R + rot + 2 * kAnyTile) * sizeof(float);
  launch_pdl(latent_attn_any_kernel<T>, dim3(N, H), dim3(kAnyThreads), smem, s, static_cast<const T*>(q_lat),
             static_cast<const T*>(q_pe), pe_token_stride, pe_head_stride, static_cast<const T*>(cache), row_elems,
             page_table, max_pages, page_size, rows, kv_lens, static_cast<T*>(out), H, R, rot, scale);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace
}  // namespace sglb

extern "C" {

// proj [T, ld] (queries rotated in place), cos_sin fp32 [positions, rot] = [cos | sin], cache rows of `row_elems`.
int sglb_latent_prep(void* proj, long long ld, int q_off, int dkv_off, int T, int H, int dim, int rot, int R,
                     const float* norm_w, float eps, const float* cos_sin, const int* positions, const int* loc,
                     void* cache, int row_elems, int is_f32, cudaStream_t s) {
  using namespace sglb;
  if (T <= 0) return 0;
  if (rot % 2 != 0 || row_elems < R + rot) return -kBadArgument;
  if (is_f32)
    launch_pdl(latent_prep_kernel<float>, dim3(T), dim3(kPrepThreads), 0, s, static_cast<float*>(proj), ld, q_off, dkv_off,
               H, dim, rot, R, norm_w, eps, cos_sin, positions, loc, static_cast<float*>(cache), row_elems);
  else
    launch_pdl(latent_prep_kernel<__nv_bfloat16>, dim3(T), dim3(kPrepThreads), 0, s, static_cast<__nv_bfloat16*>(proj), ld,
               q_off, dkv_off, H, dim, rot, R, norm_w, eps, cos_sin, positions, loc, static_cast<__nv_bfloat16*>(cache),
               row_elems);
  return static_cast<int>(cudaGetLastError());
}

// q_lat [N, H, R]; q_pe addressed by strides; query n sees the first kv_lens[n] tokens of table row rows[n];
// out [N, H, R].
int sglb_latent_attn_any(const void* q_lat, const void* q_pe, long long pe_token_stride, int pe_head_stride,
                         const void* cache, int row_elems, const int* page_table, int max_pages, int page_size,
                         const int* rows, const int* kv_lens, void* out, int N, int H, int R, int rot, float scale,
                         int is_f32, cudaStream_t s) {
  using namespace sglb;
  if (N <= 0) return 0;
  if (R > kAnyMaxAcc * kAnyThreads || R + rot > 8192 || H > 65535) return -kBadArgument;
  return is_f32 ? attn_any<float>(q_lat, q_pe, pe_token_stride, pe_head_stride, cache, row_elems, page_table, max_pages,
                                  page_size, rows, kv_lens, out, N, H, R, rot, scale, s)
                : attn_any<__nv_bfloat16>(q_lat, q_pe, pe_token_stride, pe_head_stride, cache, row_elems, page_table,
                                          max_pages, page_size, rows, kv_lens, out, N, H, R, rot, scale, s);
}

// lat [total, R], pe [total, rot] <- cache rows of B sequences laid end to end at ctx_start (bf16; R and rot multiples
// of 8).
int sglb_latent_gather(void* lat, void* pe, const void* cache, int row_elems, const int* page_table, int max_pages,
                       int page_size, const int* rows, const int* ctx_start, int B, int total, int R, int rot,
                       cudaStream_t s) {
  using namespace sglb;
  if (B <= 0 || total <= 0) return 0;
  if (R % 8 != 0 || rot % 8 != 0 || row_elems % 8 != 0) return -kBadArgument;
  launch_pdl(latent_gather_kernel, dim3((total + 7) / 8), dim3(256), 0, s, static_cast<__nv_bfloat16*>(lat),
             static_cast<__nv_bfloat16*>(pe), static_cast<const __nv_bfloat16*>(cache), row_elems, page_table, max_pages,
             page_size, rows, ctx_start, B, total, R, rot);
  return static_cast<int>(cudaGetLastError());
}

}  // extern "C"
