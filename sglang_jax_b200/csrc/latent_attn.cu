// Latent attention with any sizes (latent width R, rotary width, heads, head and value widths), in bf16 or fp32, around
// the paged latent cache  [pages, P, row]  (row >= R + rotary lanes):
//
//   latent_prep       one pass over a step's fused projection: RMS-normalises the latent, rotates the shared key part
//                     and the queries' rotary part (interleaved pairs, fp32 angles), writes the cache rows; where queries
//                     have a latent of their own, RMS-normalises that instead, and
//   latent_rotate     rotates the queries that come out of it
//   latent_attn_any   absorbed attention of single query tokens on the CUDA cores, everything in fp32: the fp32 mode,
//                     and bf16 sizes that the tensor-core kernels (mla.cu, latent_extend.cu) do not take; window, sink
//   latent_gather     cache rows of whole sequences (or from a token on) -> contiguous latents and key parts (input of the
//                     prefill kernel)
//
// Compiled without fast-math substitutions.
#include <math.h>

#include <type_traits>

#include "common.cuh"

namespace sglb {
namespace {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

constexpr int kPrepThreads = 128;

// Queries that come from a latent: its columns in the projection, its norm's weight, the result [T, rank] (out null: none).
struct QueryLatent {
  int off, rank;
  const float* norm_w;
  void* out;
};

// VEC consecutive values as one access (8 of bf16 or 4 of fp32: 16 bytes; 2: a rotary pair; 1: any alignment)
template <typename T, int VEC> struct Vec { T v[VEC]; };
template <> struct alignas(16) Vec<__nv_bfloat16, 8> { __nv_bfloat16 v[8]; };
template <> struct alignas(16) Vec<float, 4> { float v[4]; };
template <> struct alignas(4) Vec<__nv_bfloat16, 2> { __nv_bfloat16 v[2]; };
template <> struct alignas(8) Vec<float, 2> { float v[2]; };

// A warp's sum of squares of what its lanes read of src
template <typename T, int VEC>
__device__ __forceinline__ float squares(const T* __restrict__ src, int n) {
  float ss = 0.f;
  for (int i = threadIdx.x * VEC; i < n; i += kPrepThreads * VEC) {
    const Vec<T, VEC> a = *reinterpret_cast<const Vec<T, VEC>*>(src + i);
#pragma unroll
    for (int e = 0; e < VEC; ++e) ss += to_f(a.v[e]) * to_f(a.v[e]);
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  return ss;
}

// dst = src * inv * w over n values
template <typename T, int VEC>
__device__ __forceinline__ void scaled_row(const T* __restrict__ src, T* __restrict__ dst, const float* __restrict__ w, int n,
                                           float inv) {
  for (int i = threadIdx.x * VEC; i < n; i += kPrepThreads * VEC) {
    Vec<T, VEC> a = *reinterpret_cast<const Vec<T, VEC>*>(src + i);
#pragma unroll
    for (int e = 0; e < VEC; ++e) a.v[e] = from_f<T>(to_f(a.v[e]) * inv * w[i + e]);
    *reinterpret_cast<Vec<T, VEC>*>(dst + i) = a;
  }
}

// VEC / 2 interleaved pairs from pair i on; cs = [cos | sin] of the position, `half` each
template <typename T, int VEC>
__device__ __forceinline__ void rotate_pairs(const T* src, T* dst, const float* __restrict__ cs, int half, int i) {
  constexpr int N = VEC < 2 ? 2 : VEC;
  Vec<T, N> a;
  if constexpr (VEC < 2) {
    a.v[0] = src[0];
    a.v[1] = src[1];
  } else {
    a = *reinterpret_cast<const Vec<T, N>*>(src);
  }
#pragma unroll
  for (int e = 0; e < N; e += 2) {
    const float u = to_f(a.v[e]), v = to_f(a.v[e + 1]), c = cs[i + e / 2], s = cs[half + i + e / 2];
    a.v[e] = from_f<T>(u * c - v * s);
    a.v[e + 1] = from_f<T>(v * c + u * s);
  }
  if constexpr (VEC < 2) {
    dst[0] = a.v[0];
    dst[1] = a.v[1];
  } else {
    *reinterpret_cast<Vec<T, N>*>(dst) = a;
  }
}

// One CTA per token.  `proj` is the fused projection [T, ld]: query heads at column q_off, [latent | key part] at dkv_off.
template <typename T, int VEC>
__global__ void __launch_bounds__(kPrepThreads)
latent_prep_kernel(T* __restrict__ proj, long long ld, int q_off, int dkv_off, int H, int dim, int rot, int R,
                   const float* __restrict__ norm_w, float eps, const float* __restrict__ cos_sin,
                   const int* __restrict__ positions, const int* __restrict__ loc, T* __restrict__ cache,
                   int row_elems, const QueryLatent ql) {
  __shared__ float red[2][kPrepThreads / 32];
  constexpr int kPairs = VEC < 2 ? 1 : VEC / 2;
  pdl_wait();
  const int t = blockIdx.x, tid = threadIdx.x, half = rot / 2;
  T* row = proj + static_cast<long long>(t) * ld;
  const float* cs = cos_sin + static_cast<long long>(positions[t]) * rot;
  T* dst = cache + static_cast<long long>(loc[t]) * row_elems;
  const T* lat = row + dkv_off;
  for (int i = tid * kPairs; i < half; i += kPrepThreads * kPairs)
    rotate_pairs<T, VEC>(lat + R + 2 * i, dst + R + 2 * i, cs, half, i);
  const float s0 = squares<T, VEC>(lat, R), s1 = ql.out != nullptr ? squares<T, VEC>(row + ql.off, ql.rank) : 0.f;
  if ((tid & 31) == 0) {
    red[0][tid >> 5] = s0;
    red[1][tid >> 5] = s1;
  }
  __syncthreads();
  float tot = 0.f, tot_q = 0.f;
#pragma unroll
  for (int i = 0; i < kPrepThreads / 32; ++i) {
    tot += red[0][i];
    tot_q += red[1][i];
  }
  scaled_row<T, VEC>(lat, dst, norm_w, R, 1.f / sqrtf(tot / R + eps));
  if (ql.out != nullptr) {
    scaled_row<T, VEC>(row + ql.off, static_cast<T*>(ql.out) + static_cast<long long>(t) * ql.rank, ql.norm_w, ql.rank,
                       1.f / sqrtf(tot_q / ql.rank + eps));
    return;
  }
  const int per = half / kPairs;
  for (int j = tid; j < H * per; j += kPrepThreads) {
    const int h = j / per, i = (j - h * per) * kPairs;
    T* q = row + q_off + static_cast<long long>(h) * (dim + rot) + dim + 2 * i;
    rotate_pairs<T, VEC>(q, q, cs, half, i);
  }
}

// Rotates the last `rot` of every head's `dim + rot` lanes in place.
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
latent_rotate_kernel(T* __restrict__ q, long long ld, int H, int dim, int rot, const float* __restrict__ cos_sin,
                     const int* __restrict__ positions) {
  constexpr int kPairs = VEC < 2 ? 1 : VEC / 2;
  pdl_wait();
  const int half = rot / 2, per = half / kPairs;
  const float* cs = cos_sin + static_cast<long long>(positions[blockIdx.x]) * rot;
  T* row = q + blockIdx.x * ld + dim;
  for (int j = threadIdx.x; j < H * per; j += blockDim.x) {
    const int h = j / per, i = (j - h * per) * kPairs;
    T* a = row + static_cast<long long>(h) * (dim + rot) + 2 * i;
    rotate_pairs<T, VEC>(a, a, cs, half, i);
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
                       const int* __restrict__ kv_lens, T* __restrict__ out, int H, int R, int rot, float scale,
                       int window, const float* __restrict__ sink) {
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
  const int D = R + rot, first = window > 0 && len > window ? len - window : 0;
  for (int k0 = first / kAnyTile * kAnyTile; k0 < len; k0 += kAnyTile) {
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
      if (lane == 0) sc[j] = k0 + j >= first ? a * scale : -INFINITY;
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
  float inv = l > 0.f ? 1.f / l : 0.f;
  if (sink != nullptr) {
    const float mx = fmaxf(m, sink[h]), c = expf(m - mx);
    inv = c / (l * c + expf(sink[h] - mx));
  }
#pragma unroll
  for (int i = 0; i < kAnyMaxAcc; ++i) {
    const int d = tid + i * kAnyThreads;
    if (d < R) out[nh * R + d] = from_f<T>(acc[i] * inv);
  }
}

// ctx row r of sequence b (ctx_start[b] <= r < ctx_start[b + 1]) is the sequence's token r - ctx_start[b] + skip[b] (skip null:
// none left out).
__global__ void latent_gather_kernel(__nv_bfloat16* __restrict__ lat, __nv_bfloat16* __restrict__ pe,
                                     const __nv_bfloat16* __restrict__ cache, int row_elems,
                                     const int* __restrict__ page_table, int max_pages, int page_size,
                                     const int* __restrict__ rows, const int* __restrict__ ctx_start,
                                     const int* __restrict__ skip, int B, int total, int R, int rot) {
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
  const int pos = r - ctx_start[lo] + (skip != nullptr ? skip[lo] : 0), pg = pos / page_size;
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
             void* out, int N, int H, int R, int rot, float scale, int window, const float* sink, cudaStream_t s) {
  const size_t smem = (R + rot + 2 * kAnyTile) * sizeof(float);
  launch_pdl(latent_attn_any_kernel<T>, dim3(N, H), dim3(kAnyThreads), smem, s, static_cast<const T*>(q_lat),
             static_cast<const T*>(q_pe), pe_token_stride, pe_head_stride, static_cast<const T*>(cache), row_elems,
             page_table, max_pages, page_size, rows, kv_lens, static_cast<T*>(out), H, R, rot, scale, window, sink);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace
}  // namespace sglb

extern "C" {

// proj [T, ld] (queries rotated in place), cos_sin fp32 [positions, rot] = [cos | sin], cache rows of `row_elems`.  With
// `q_latent` [T, q_rank] the projection holds no queries but their latent at column q_off, which is normalised (q_norm_w) into
// it.
int sglb_latent_prep(void* proj, long long ld, int q_off, int dkv_off, int T, int H, int dim, int rot, int R,
                     const float* norm_w, float eps, const float* cos_sin, const int* positions, const int* loc,
                     void* cache, int row_elems, void* q_latent, int q_rank, const float* q_norm_w, int is_f32,
                     cudaStream_t s) {
  using namespace sglb;
  if (T <= 0) return 0;
  if (rot % 2 != 0 || row_elems < R + rot || (q_latent != nullptr && (q_rank < 1 || q_norm_w == nullptr)))
    return -kBadArgument;
  const QueryLatent ql{q_off, q_rank, q_norm_w, q_latent};
  const int n = is_f32 ? 4 : 8;
  auto whole = [&](long long v) { return v % n == 0; };
  const bool wide = whole(ld) && whole(dkv_off) && whole(R) && whole(rot) && whole(row_elems) && whole(q_off) &&
                    (q_latent != nullptr ? whole(q_rank) : whole(dim)) && reinterpret_cast<uintptr_t>(proj) % 16 == 0;
  auto run = [&](auto kernel, auto* p) {
    using T_ = std::remove_pointer_t<decltype(p)>;
    launch_pdl(kernel, dim3(T), dim3(kPrepThreads), 0, s, p, ld, q_off, dkv_off, H, dim, rot, R, norm_w, eps, cos_sin,
               positions, loc, static_cast<T_*>(cache), row_elems, ql);
  };
  if (is_f32) run(wide ? latent_prep_kernel<float, 4> : latent_prep_kernel<float, 1>, static_cast<float*>(proj));
  else run(wide ? latent_prep_kernel<__nv_bfloat16, 8> : latent_prep_kernel<__nv_bfloat16, 1>,
           static_cast<__nv_bfloat16*>(proj));
  return static_cast<int>(cudaGetLastError());
}

// Head h of token t at q + t * ld + h * (dim + rot), rotated in place.
int sglb_latent_rotate(void* q, long long ld, int T, int H, int dim, int rot, const float* cos_sin, const int* positions,
                       int is_f32, cudaStream_t s) {
  using namespace sglb;
  if (T <= 0 || rot == 0) return 0;
  if (rot % 2 != 0 || H < 1) return -kBadArgument;
  const int n = is_f32 ? 4 : 8;
  const uintptr_t at = reinterpret_cast<uintptr_t>(q);
  const bool wide = ld % n == 0 && dim % n == 0 && rot % n == 0 && at % 16 == 0;
  const bool pairs = ld % 2 == 0 && dim % 2 == 0 && at % 8 == 0;
  auto run = [&](auto kernel, auto* p) {
    launch_pdl(kernel, dim3(T), dim3(256), 0, s, p, ld, H, dim, rot, cos_sin, positions);
  };
  if (is_f32)
    run(wide ? latent_rotate_kernel<float, 4> : (pairs ? latent_rotate_kernel<float, 2> : latent_rotate_kernel<float, 1>),
        static_cast<float*>(q));
  else
    run(wide ? latent_rotate_kernel<__nv_bfloat16, 8>
             : (pairs ? latent_rotate_kernel<__nv_bfloat16, 2> : latent_rotate_kernel<__nv_bfloat16, 1>),
        static_cast<__nv_bfloat16*>(q));
  return static_cast<int>(cudaGetLastError());
}

// q_lat [N, H, R]; q_pe addressed by strides; query n sees the first kv_lens[n] tokens of table row rows[n];
// out [N, H, R].  `window` (0: none): tokens a query sees, its own included; `sink` [H] or null.
int sglb_latent_attn_any(const void* q_lat, const void* q_pe, long long pe_token_stride, int pe_head_stride,
                         const void* cache, int row_elems, const int* page_table, int max_pages, int page_size,
                         const int* rows, const int* kv_lens, void* out, int N, int H, int R, int rot, float scale,
                         int window, const float* sink, int is_f32, cudaStream_t s) {
  using namespace sglb;
  if (N <= 0) return 0;
  if (R > kAnyMaxAcc * kAnyThreads || R + rot > 8192 || H > 65535) return -kBadArgument;
  return is_f32 ? attn_any<float>(q_lat, q_pe, pe_token_stride, pe_head_stride, cache, row_elems, page_table, max_pages,
                                  page_size, rows, kv_lens, out, N, H, R, rot, scale, window, sink, s)
                : attn_any<__nv_bfloat16>(q_lat, q_pe, pe_token_stride, pe_head_stride, cache, row_elems, page_table,
                                          max_pages, page_size, rows, kv_lens, out, N, H, R, rot, scale, window, sink, s);
}

// lat [total, R], pe [total, rot] <- cache rows of B sequences, each from token skip[b] on (null: 0), laid end to end at
// ctx_start (bf16; R and rot multiples of 8).
int sglb_latent_gather(void* lat, void* pe, const void* cache, int row_elems, const int* page_table, int max_pages,
                       int page_size, const int* rows, const int* ctx_start, const int* skip, int B, int total, int R,
                       int rot, cudaStream_t s) {
  using namespace sglb;
  if (B <= 0 || total <= 0) return 0;
  if (R % 8 != 0 || rot % 8 != 0 || row_elems % 8 != 0) return -kBadArgument;
  launch_pdl(latent_gather_kernel, dim3((total + 7) / 8), dim3(256), 0, s, static_cast<__nv_bfloat16*>(lat),
             static_cast<__nv_bfloat16*>(pe), static_cast<const __nv_bfloat16*>(cache), row_elems, page_table, max_pages,
             page_size, rows, ctx_start, skip, B, total, R, rot);
  return static_cast<int>(cudaGetLastError());
}

}  // extern "C"
