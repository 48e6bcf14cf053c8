// Absorbed multi-head latent attention, decode step (DeepSeek-V2/V3, Kimi-K2, GLM-5, Zozopel, Kunudra).
//
// Every head attends over the same latent cache rows  [pages, P, R + rotary lanes]  (R = kv_lora_rank; 512 + 64
// lanes in the DeepSeek family): logits = q_latent . c + q_pe . k_pe, output = softmax . c  (the caller applies
// W_UV).  This is multi-query attention with an (R + rotary)-wide key and an R-wide value that alias the same
// bytes, so one tile of 64 tokens (72 KB at 576 lanes) streamed by TMA serves both products.  A key is a run of
// 64-lane blocks; lanes past its width arrive as zeros.
//
// One CTA handles 16 heads of one sequence and one KV split.  Its four consumer warps split the work
// along different axes in the two products: for S = Q K^T each warp owns 16 of the tile's 64 tokens
// (Q fragments come from shared memory); the scaled logits go through a double-buffered
// shared tile so that every warp sees the whole 16 x 64 row block, computes the (identical) online
// softmax statistics, and then accumulates its own share of the R output lanes of O += P V (NG groups of
// 16 lanes).  No cross-warp merge is needed at the end.  With EXACT the weights enter that product as a sum of
// two bf16 numbers (their rounding and its remainder) instead of being rounded to bf16.  A fifth warp issues the
// TMA copies (page gathers through the device page table).  With a window only the tiles it reaches are read; a sink joins
// the denominator once the splits are together.  All barrier waits are bounded; no multicast is used.
//
// Reference contract: python/sgl_jax/srt/kernels/mla/v2/kernel.py:1338 (oracle mla/v1/ref.py).
#include <cstdlib>
#include <math.h>

#include <unordered_map>

#include "common.cuh"
#include "score_terms.cuh"

namespace sglb {
namespace {

constexpr int TN = 64;                 // tokens per tile
constexpr int kChunkBytes = TN * 128;  // one column block of 64 bf16 (128-byte swizzle rows): 8 KB
constexpr int kMaxStages = 4;
constexpr int kSBytes = 2 * 16 * TN * 4;             // double-buffered logits tile
constexpr int kConsumerWarps = 4;
constexpr int kThreads = (kConsumerWarps + 1) * 32;
// `blocks` column blocks per key: that many per stage, and per 16-head query tile
constexpr int smem_bytes(int blocks, int stages) {
  return stages * blocks * kChunkBytes + blocks * 16 * 128 + kSBytes + 128 + 1024;
}
constexpr int kMaxSmem = 227 * 1024;

struct MlaParams {
  const __nv_bfloat16* q_lat;   // [B, H, R]
  const __nv_bfloat16* q_pe;    // rotary lanes of (b, h) at b * pe_token_stride + h * pe_head_stride
  __nv_bfloat16* out;           // [B, H, R]
  float* part_o;                // [B, H, splits, R]
  float* part_lse;              // [B, H, splits]
  const int* page_table;        // [rows, max_pages]
  const int* req_pool_indices;  // [B]
  const int* seq_lens;          // [B]
  Status* status;
  int B, H, max_pages, page_size, num_splits;
  int R, DK;                    // latent (value) width, key width = R + rotary lanes
  int blocks, stages;           // 64-lane column blocks of a key, tiles in the ring
  long long pe_token_stride;
  int pe_head_stride;
  float scale;
  int window;                   // keys a query sees, its own included; 0: all
  ScoreTerms terms;             // (the sink only)
};

__device__ __forceinline__ void ldsm_x4(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// byte offset of (row, 16-byte chunk) inside a [rows][64 bf16] block with the 128-byte swizzle
__device__ __forceinline__ uint32_t sw_off(int row, int chunk) { return row * 128 + ((chunk ^ (row & 7)) << 4); }

// NG: 16-lane groups of the output per consumer warp, R <= 64 * NG
template <int NG, bool EXACT>
__global__ void __launch_bounds__(kThreads, 1)
mla_decode_kernel(const __grid_constant__ CUtensorMap tmap, const MlaParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int R = p.R, DK = p.DK, nblk = p.blocks, stages = p.stages;
  const int stage_bytes = nblk * kChunkBytes;
  uint8_t* q_sm = smem + stages * stage_bytes;
  float* s_sm = reinterpret_cast<float*>(q_sm + nblk * 16 * 128);
  uint64_t* full_bar = reinterpret_cast<uint64_t*>(reinterpret_cast<uint8_t*>(s_sm) + kSBytes);
  uint64_t* empty_bar = full_bar + kMaxStages;
  volatile int* abort_flag = reinterpret_cast<volatile int*>(empty_bar + kMaxStages);

  const int b = blockIdx.x, hg = blockIdx.y, split = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int seq = p.seq_lens[b];
  const int* pt_row = p.page_table + static_cast<size_t>(p.req_pool_indices[b]) * p.max_pages;
  const int first = p.window > 0 && seq > p.window ? seq - p.window : 0;      // first visible token
  const int n_tiles = (seq + TN - 1) / TN, tb = first / TN;
  const int per = (n_tiles - tb + p.num_splits - 1) / p.num_splits;
  const int t0 = tb + split * per;
  const int t1 = min(t0 + per, n_tiles);

  if (threadIdx.x == 0) {
    for (int s = 0; s < stages; ++s) {
      mbar_init(smem_u32(&full_bar[s]), 1);
      mbar_init(smem_u32(&empty_bar[s]), kConsumerWarps);
    }
    *abort_flag = 0;
    fence_barrier_init();
  }
  __syncthreads();

  if (warp == kConsumerWarps) {
    // ------------------------------------------------------------------ TMA producer
    if (lane == 0) {
      prefetch_tmap(&tmap);
      const uint64_t pol = l2_policy_evict_first();      // every latent row is read once per head group
      int stage = 0;
      uint32_t phase = 0;
      const int run = p.page_size < TN ? p.page_size : TN;
      const int n_runs = TN / run;
      for (int t = t0; t < t1 && !*abort_flag; ++t) {
        if (!mbar_wait(smem_u32(&empty_bar[stage]), phase ^ 1)) {
          report(p.status, kTimeoutEmptyBarrier, b, t);
          *abort_flag = 1;
          break;
        }
        const uint32_t bar = smem_u32(&full_bar[stage]);
        const uint32_t dst0 = smem_u32(smem + stage * stage_bytes);
        mbar_expect_tx(bar, stage_bytes);
        for (int r = 0; r < n_runs; ++r) {
          const int tok = t * TN + r * run;
          int pg = tok / p.page_size;
          if (pg >= p.max_pages) pg = p.max_pages - 1;
          const int row = pt_row[pg] * p.page_size + (tok - pg * p.page_size);
          for (int c = 0; c < nblk; ++c)
            tma_load_2d_hint(dst0 + c * kChunkBytes + r * run * 128, &tmap, bar, c * 64, row, pol);
        }
        if (++stage == stages) {
          stage = 0;
          phase ^= 1;
        }
      }
    }
  } else {
    // ------------------------------------------------------------------ consumers
    const int g = lane >> 2, t4 = lane & 3;
    const int ctid = threadIdx.x;                       // 0..127
    // stage the 16 query rows (zero rows beyond H) into swizzled shared memory
    const bool vec = R % 8 == 0 && DK % 8 == 0 && p.pe_token_stride % 8 == 0 && p.pe_head_stride % 8 == 0 &&
                     reinterpret_cast<uintptr_t>(p.q_pe) % 16 == 0;
    for (int v = ctid; v < 16 * nblk * 8; v += kConsumerWarps * 32) {
      const int r = v / (nblk * 8), c8 = v - r * (nblk * 8);      // row, 16-byte chunk along the key lanes
      const int h = hg * 16 + r;
      uint4 val = make_uint4(0u, 0u, 0u, 0u);
      if (h < p.H && c8 * 8 < DK) {
        const __nv_bfloat16* ql = p.q_lat + (static_cast<size_t>(b) * p.H + h) * R;
        const __nv_bfloat16* qp = p.q_pe + b * p.pe_token_stride + static_cast<long long>(h) * p.pe_head_stride;
        if (vec) {
          val = *reinterpret_cast<const uint4*>(c8 < R / 8 ? ql + c8 * 8 : qp + (c8 * 8 - R));
        } else {
          __align__(16) __nv_bfloat16 e8[8];
#pragma unroll
          for (int e = 0; e < 8; ++e) {
            const int d = c8 * 8 + e;
            e8[e] = d < R ? ql[d] : (d < DK ? qp[d - R] : __float2bfloat16(0.f));
          }
          val = *reinterpret_cast<const uint4*>(e8);
        }
      }
      const int blk = c8 / 8, ch = c8 % 8;
      *reinterpret_cast<uint4*>(q_sm + blk * (16 * 128) + sw_off(r, ch)) = val;
    }
    named_bar_sync(1, kConsumerWarps * 32);

    float o[2 * NG][4];                                  // this warp's 16 * NG output lanes of rows g, g+8
#pragma unroll
    for (int i = 0; i < 2 * NG; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};
    const float scale_log2 = p.scale * kLog2E;
    const uint32_t q_base = smem_u32(q_sm);
    int stage = 0;
    uint32_t phase = 0;
    int sbuf = 0;
    for (int t = t0; t < t1 && !*abort_flag; ++t) {
      if (!mbar_wait(smem_u32(&full_bar[stage]), phase)) {
        report(p.status, kTimeoutFullBarrier, b, t);
        *abort_flag = 1;
        break;
      }
      const uint32_t kv = smem_u32(smem + stage * stage_bytes);
      // ---- S[:, 16w .. 16w+15] = Q K^T over the key lanes
      float s[2][4];
#pragma unroll
      for (int j = 0; j < 2; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.f;
#pragma unroll 4
      for (int kk = 0; kk < nblk * 4; ++kk) {
        const int blk = kk >> 2, c0 = (kk & 3) * 2;
        uint32_t a[4];
        ldsm_x4(q_base + blk * (16 * 128) + sw_off((lane & 7) + (((lane >> 3) & 1) << 3), c0 + (lane >> 4)),
                a[0], a[1], a[2], a[3]);
        const int row = warp * 16 + (lane & 7) + ((lane >> 4) << 3);
        uint32_t b0, b1, b2, b3;
        ldsm_x4(kv + blk * kChunkBytes + sw_off(row, c0 + ((lane >> 3) & 1)), b0, b1, b2, b3);
        mma16816(s[0], a, b0, b1);
        mma16816(s[1], a, b2, b3);
      }
      float* sb = s_sm + sbuf * (16 * TN);
#pragma unroll
      for (int j = 0; j < 2; ++j) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int col = warp * 16 + j * 8 + t4 * 2 + (e & 1);
          const int tok = t * TN + col;
          sb[(g + 8 * (e >> 1)) * TN + col] = tok < seq && tok >= first ? s[j][e] * scale_log2 : -INFINITY;
        }
      }
      named_bar_sync(1, kConsumerWarps * 32);
      // ---- online softmax over the whole 16 x 64 block (every warp computes the same statistics)
      float pr[8][4];                                    // [j][e]: cols 8j + 2*t4 + (e&1), row g + 8*(e>>1)
      float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const float2 lo = *reinterpret_cast<const float2*>(sb + g * TN + j * 8 + t4 * 2);
        const float2 hi = *reinterpret_cast<const float2*>(sb + (g + 8) * TN + j * 8 + t4 * 2);
        pr[j][0] = lo.x; pr[j][1] = lo.y; pr[j][2] = hi.x; pr[j][3] = hi.y;
        mx[0] = fmaxf(mx[0], fmaxf(lo.x, lo.y));
        mx[1] = fmaxf(mx[1], fmaxf(hi.x, hi.y));
      }
      float corr[2], mref[2];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 1));
        mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 2));
        const float mnew = fmaxf(m_run[i], mx[i]);
        mref[i] = mnew == -INFINITY ? 0.f : mnew;
        corr[i] = exp2f(m_run[i] - mref[i]);
        m_run[i] = mnew;
      }
      float rs[2] = {0.f, 0.f};
#pragma unroll
      for (int j = 0; j < 8; ++j) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float pv = exp2f(pr[j][e] - mref[e >> 1]);
          pr[j][e] = pv;
          rs[e >> 1] += pv;
        }
      }
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        rs[i] += __shfl_xor_sync(0xffffffffu, rs[i], 1);
        rs[i] += __shfl_xor_sync(0xffffffffu, rs[i], 2);
        l_run[i] = l_run[i] * corr[i] + rs[i];
      }
#pragma unroll
      for (int n = 0; n < 2 * NG; ++n) {
        o[n][0] *= corr[0]; o[n][1] *= corr[0];
        o[n][2] *= corr[1]; o[n][3] *= corr[1];
      }
      // ---- O[:, 16 NG w .. 16 NG (w + 1) - 1] += P V   (V = the first R lanes of the same rows)
#pragma unroll
      for (int kk = 0; kk < TN / 16; ++kk) {
        uint32_t pa[4];
        pa[0] = pack_bf16(pr[2 * kk][0], pr[2 * kk][1]);
        pa[1] = pack_bf16(pr[2 * kk][2], pr[2 * kk][3]);
        pa[2] = pack_bf16(pr[2 * kk + 1][0], pr[2 * kk + 1][1]);
        pa[3] = pack_bf16(pr[2 * kk + 1][2], pr[2 * kk + 1][3]);
        uint32_t pl[4];
        if constexpr (EXACT) {
          auto rest = [](float a, float b, uint32_t hi) {
            return pack_bf16(a - __uint_as_float(hi << 16), b - __uint_as_float(hi & 0xffff0000u));
          };
          pl[0] = rest(pr[2 * kk][0], pr[2 * kk][1], pa[0]);
          pl[1] = rest(pr[2 * kk][2], pr[2 * kk][3], pa[1]);
          pl[2] = rest(pr[2 * kk + 1][0], pr[2 * kk + 1][1], pa[2]);
          pl[3] = rest(pr[2 * kk + 1][2], pr[2 * kk + 1][3], pa[3]);
        }
#pragma unroll
        for (int np = 0; np < NG; ++np) {
          const int row = kk * 16 + (lane & 7) + (((lane >> 3) & 1) << 3);
          const int dcol = (warp * NG + np) * 16 + ((lane >> 4) << 3);
          uint32_t b0, b1, b2, b3;
          ldsm_x4_t(kv + (dcol >> 6) * kChunkBytes + sw_off(row, (dcol & 63) >> 3), b0, b1, b2, b3);
          mma16816(o[2 * np], pa, b0, b1);
          mma16816(o[2 * np + 1], pa, b2, b3);
          if constexpr (EXACT) {
            mma16816(o[2 * np], pl, b0, b1);
            mma16816(o[2 * np + 1], pl, b2, b3);
          }
        }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(&empty_bar[stage]));
      if (++stage == stages) {
        stage = 0;
        phase ^= 1;
      }
      sbuf ^= 1;
    }
    // ---- write out (rows g and g+8 of this head group, this warp's lanes)
    const int lane0 = warp * 16 * NG + t4 * 2;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int h = hg * 16 + g + 8 * i;
      if (h >= p.H) continue;
      float inv = l_run[i] > 0.f ? 1.f / l_run[i] : 0.f;
      if (p.num_splits == 1 && p.terms.sink != nullptr) {
        const float sink = p.terms.sink_log2(h), m = fmaxf(m_run[i], sink), c = exp2f(m_run[i] - m);
        inv = c / (l_run[i] * c + exp2f(sink - m));
      }
      const size_t bh = static_cast<size_t>(b) * p.H + h;
      if (p.num_splits == 1) {
        __nv_bfloat16* dst = p.out + bh * R;
#pragma unroll
        for (int n = 0; n < 2 * NG; ++n) {
          const int d = lane0 + n * 8;
          const uint32_t v = pack_bf16(o[n][2 * i] * inv, o[n][2 * i + 1] * inv);
          if (R % 2 == 0) {
            if (d < R) *reinterpret_cast<uint32_t*>(dst + d) = v;
          } else {
            if (d < R) dst[d] = __float2bfloat16(o[n][2 * i] * inv);
            if (d + 1 < R) dst[d + 1] = __float2bfloat16(o[n][2 * i + 1] * inv);
          }
        }
      } else {
        float* dst = p.part_o + (bh * p.num_splits + split) * R;
#pragma unroll
        for (int n = 0; n < 2 * NG; ++n) {
          const int d = lane0 + n * 8;
          if (R % 2 == 0) {
            if (d < R) *reinterpret_cast<float2*>(dst + d) = make_float2(o[n][2 * i] * inv, o[n][2 * i + 1] * inv);
          } else {
            if (d < R) dst[d] = o[n][2 * i] * inv;
            if (d + 1 < R) dst[d + 1] = o[n][2 * i + 1] * inv;
          }
        }
        if (warp == 0 && t4 == 0)
          p.part_lse[bh * p.num_splits + split] = l_run[i] > 0.f ? m_run[i] + log2f(l_run[i]) : -INFINITY;
      }
    }
  }
  __syncthreads();
  if (*abort_flag) {
    // give copies that are still in flight time to land before the CTA's shared memory is released
    const uint64_t ts = global_timer_ns();
    while (global_timer_ns() - ts < 200000ull) __nanosleep(1000);
  }
}

__global__ void mla_combine_kernel(const float* __restrict__ part_o, const float* __restrict__ part_lse,
                                   __nv_bfloat16* __restrict__ out, int num_splits, int R, int H, const ScoreTerms terms) {
  const int row = blockIdx.x;   // b * H + h
  const float* lse = part_lse + static_cast<size_t>(row) * num_splits;
  float mmax = -INFINITY;
  for (int s = 0; s < num_splits; ++s) mmax = fmaxf(mmax, lse[s]);
  const float sink = terms.sink_log2(row % H);
  mmax = fmaxf(mmax, sink);
  float wsum = sink == -INFINITY ? 0.f : exp2f(sink - mmax);
  for (int s = 0; s < num_splits; ++s) wsum += (lse[s] == -INFINITY) ? 0.f : exp2f(lse[s] - mmax);
  const float inv = wsum > 0.f ? 1.f / wsum : 0.f;
  for (int d = threadIdx.x; d < R; d += blockDim.x) {
    float acc = 0.f;
    for (int s = 0; s < num_splits; ++s) {
      const float w = (lse[s] == -INFINITY) ? 0.f : exp2f(lse[s] - mmax);
      acc += w * part_o[(static_cast<size_t>(row) * num_splits + s) * R + d];
    }
    out[static_cast<size_t>(row) * R + d] = __float2bfloat16(acc * inv);
  }
}

struct Key {
  const void* p; long long rows; int box, width, stride;
  bool operator==(const Key& o) const {
    return p == o.p && rows == o.rows && box == o.box && width == o.width && stride == o.stride;
  }
};
struct KeyHash {
  size_t operator()(const Key& k) const {
    return std::hash<const void*>()(k.p) ^ (std::hash<long long>()(k.rows) * 1315423911u) ^ (k.box * 2654435761u) ^ (k.width * 40503u) ^
           (k.stride * 97u);
  }
};
std::unordered_map<Key, CUtensorMap, KeyHash> g_maps;

bool get_map(const void* kv, long long rows, int width, int stride, int page_size, CUtensorMap* out) {
  const int box_rows = page_size < TN ? page_size : TN;
  Key key{kv, rows, box_rows, width, stride};
  auto it = g_maps.find(key);
  if (it != g_maps.end()) {
    *out = it->second;
    return true;
  }
  CUtensorMap m;
  if (!encode_tmap_2d(&m, kv, width, rows, static_cast<uint64_t>(stride) * 2, 64, box_rows, 2)) return false;
  if (g_maps.size() > 1024) g_maps.clear();
  g_maps.emplace(key, m);
  *out = m;
  return true;
}

template <int NG, bool EXACT>
cudaError_t launch(const CUtensorMap& tm, const MlaParams& p, int smem, cudaStream_t stream) {
  static int cfg = 0;
  if (cfg < smem) {
    const cudaError_t e = cudaFuncSetAttribute(mla_decode_kernel<NG, EXACT>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                               smem);
    if (e != cudaSuccess) return e;
    cfg = smem;
  }
  mla_decode_kernel<NG, EXACT><<<dim3(p.B, (p.H + 15) / 16, p.num_splits), kThreads, smem, stream>>>(tm, p);
  return cudaGetLastError();
}

template <bool EXACT>
cudaError_t launch_width(const CUtensorMap& tm, const MlaParams& p, int smem, cudaStream_t stream) {
  const int ng = (p.R + 63) / 64;
  if (ng <= 1) return launch<1, EXACT>(tm, p, smem, stream);
  if (ng <= 2) return launch<2, EXACT>(tm, p, smem, stream);
  if (ng <= 4) return launch<4, EXACT>(tm, p, smem, stream);
  return launch<8, EXACT>(tm, p, smem, stream);
}

}  // namespace
}  // namespace sglb

extern "C" {

// Suggested number of KV splits of a launch over B queries with `groups` 16-head groups each: two CTAs per SM, at least
// two tiles per split.
int sglb_mla_num_splits(int B, int groups, int max_seq_len) {
  const int ctas = B * groups, tiles = (max_seq_len + sglb::TN - 1) / sglb::TN;
  int splits = (2 * sglb::sm_count() + ctas - 1) / ctas;
  if (splits > tiles / 2) splits = tiles / 2;
  return splits < 1 ? 1 : (splits > 32 ? 32 : splits);
}

// Absorbed-MLA decode.  `kv_buffer` is the latent cache [num_pages, page_size, row_elems] (bf16, rows of
// kv_lora_rank + rope_dim lanes and padding, row_elems a multiple of 8); `q_lat` [B, H, kv_lora_rank], `q_pe` addressed
// by strides; `out` [B, H, kv_lora_rank].  With `num_splits > 1` the partial buffers `part_o [B, H, splits, R]` and
// `part_lse [B, H, splits]` (fp32) are required.  `exact`: attention weights are not rounded to bf16.  `window` (0: none):
// tokens a query sees, its own included; `sink` [H] or null.
int sglb_mla_decode(const void* q_lat, const void* q_pe, long long pe_token_stride, int pe_head_stride, void* out,
                    const void* kv_buffer, long long num_pages, int row_elems, const int* page_table, int max_pages,
                    const int* req_pool_indices, const int* seq_lens, int B, int H, int kv_lora_rank, int rope_dim,
                    int page_size, float scale, int window, const float* sink, int num_splits, float* part_o,
                    float* part_lse, int exact, cudaStream_t stream) {
  using namespace sglb;
  if (B <= 0) return 0;
  const int dk = kv_lora_rank + rope_dim;
  if (kv_lora_rank < 1 || kv_lora_rank > 512 || rope_dim < 1 || dk > row_elems || row_elems % 8 != 0) return -kBadArgument;
  if (page_size < TN ? (TN % page_size != 0) : (page_size % TN != 0)) return -kBadArgument;
  if (num_splits > 1 && (part_o == nullptr || part_lse == nullptr)) return -kBadArgument;
  MlaParams p{};
  // one block past the key when the output lanes of the widest warp group reach further (they are not stored)
  const int ng = (kv_lora_rank + 63) / 64;
  const int lanes = 64 * (ng <= 2 ? ng : (ng <= 4 ? 4 : 8));
  p.blocks = (dk > lanes ? dk + 63 : lanes + 63) / 64;
  p.stages = 2;
  // more tiles in flight where keys are narrow, two CTAs per SM permitting
  while (p.stages < kMaxStages && smem_bytes(p.blocks, p.stages + 1) <= kMaxSmem / 2) ++p.stages;
  const int smem = smem_bytes(p.blocks, p.stages);
  if (smem > kMaxSmem) return -kBadArgument;
  CUtensorMap tm;
  if (!get_map(kv_buffer, num_pages * page_size, dk, row_elems, page_size, &tm)) return -100;
  p.q_lat = static_cast<const __nv_bfloat16*>(q_lat);
  p.q_pe = static_cast<const __nv_bfloat16*>(q_pe);
  p.pe_token_stride = pe_token_stride;
  p.pe_head_stride = pe_head_stride;
  p.out = static_cast<__nv_bfloat16*>(out);
  p.part_o = part_o;
  p.part_lse = part_lse;
  p.page_table = page_table;
  p.req_pool_indices = req_pool_indices;
  p.seq_lens = seq_lens;
  p.status = device_status();
  p.B = B; p.H = H; p.max_pages = max_pages; p.page_size = page_size;
  p.R = kv_lora_rank; p.DK = dk;
  p.num_splits = num_splits < 1 ? 1 : num_splits;
  p.scale = scale;
  p.window = window;
  p.terms = ScoreTerms{0.f, nullptr, sink};
  cudaError_t e = exact ? launch_width<true>(tm, p, smem, stream) : launch_width<false>(tm, p, smem, stream);
  if (e == cudaSuccess && p.num_splits > 1) {
    mla_combine_kernel<<<B * H, 128, 0, stream>>>(part_o, part_lse, p.out, p.num_splits, kv_lora_rank, H, p.terms);
    e = cudaGetLastError();
  }
  return e == cudaSuccess ? 0 : static_cast<int>(e);
}

}  // extern "C"
