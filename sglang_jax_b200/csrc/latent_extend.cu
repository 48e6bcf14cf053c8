// Causal prefill attention over expanded latents on the 5th-generation tensor cores (bf16 operands, fp32 softmax).
//
// Keys of a head are [unrotated | rotated]: the unrotated lanes and the values come from one [context, heads,
// dim + vdim] buffer that a GEMM computed from the latents, the rotated lanes from one [context, rot] buffer shared by
// all heads.  Queries are read in place from the fused projection.  A sequence's context rows start at ctx_start[b];
// query i of the step sees the first prefix[b] + i + 1 of them, under a window only the last ones of these (then the rows may
// start at token skip[b], a multiple of 64, of the sequence).  A sink joins the softmax's denominator (score_terms.cuh).
//
// One CTA per (256 query rows of one sequence, head): two 128-row tiles that share every K / V tile of 64 keys.  Warp 0
// drives TMA (two-stage ring), warp 1 issues tcgen05.mma, warps 2..5 and 6..9 do the softmax of the two tiles, one
// thread per row:
//
//   S_j = Q K_j^T      128 x 64, two accumulator buffers per tile in tensor memory
//   P_j = exp2(S_j-m)  read with tcgen05.ld, written back over S_j as two bf16 terms (rounding and remainder, so that
//                      the weights keep 16 bits of mantissa in the product) in the A-operand layout
//   O  += P_j V_j      A from tensor memory, V the MN-major B operand in shared memory
//
// While one tile's exponentials run, the tensor pipe works on the other tile.  The running maximum is only raised when
// it grows by more than 2^8.  Lanes past dim / rot / vdim arrive as zeros and whole zero steps are skipped.  All waits
// are bounded; a timeout unwinds through the normal teardown.  No multicast.
#include <math.h>

#include "common.cuh"
#include "score_terms.cuh"
#include "window_mask.cuh"

namespace sglb {
namespace {

constexpr int kTileQ = 128, kTiles = 2, kTileK = 64;
constexpr int kBlkQ = kTileQ * 128;                 // [128 rows][64 bf16], swizzled
constexpr int kBlkK = kTileK * 128;                 // [64 keys][64 bf16]
constexpr int kThreads = 64 + kTiles * 128;
constexpr int kTmemCols = 512;                      // per tile: S 2 x 64 (P in place), O 128
constexpr int kTmemTile = 256, kTmemO = 128;
constexpr float kRescale = 8.f;
constexpr int kMinSmem = 120 * 1024;                // one CTA per SM: it takes all of tensor memory

struct Bars {
  uint64_t q_full, k_full[2], k_empty[2], v_full[2], v_empty[2];
  uint64_t s_full[kTiles][2], p_ready[kTiles][2], pv_done[kTiles][2];
  uint32_t tmem_slot;
  int abort_flag;
};

struct Params {
  __nv_bfloat16* out;            // [T, heads, vdim] by strides
  long long out_token_stride;
  int out_head_stride;
  const int *q_start, *q_len, *prefix, *ctx_start, *skip;   // [B], skip may be null
  Status* status;
  int B, dim, rot, vdim;
  int nb_n, nb_r, nb_v;          // 64-lane blocks of the unrotated / rotated key part and of the values
  float scale;
  Window win;
  ScoreTerms terms;              // (the sink only)
};

__device__ __forceinline__ float ex2_approx(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

__global__ void __launch_bounds__(kThreads, 1)
latent_extend_kernel(const __grid_constant__ CUtensorMap map_qn, const __grid_constant__ CUtensorMap map_qr,
                     const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_kr,
                     const __grid_constant__ CUtensorMap map_v, const Params p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int nb_q = p.nb_n + p.nb_r;
  const int stage_bytes = (nb_q + p.nb_v) * kBlkK;
  uint8_t* q_s = smem;                                            // [tile][block]
  uint8_t* kv_s = smem + kTiles * nb_q * kBlkQ;
  Bars* bars = reinterpret_cast<Bars*>(kv_s + 2 * stage_bytes);
  volatile int* abort_flag = &bars->abort_flag;

  // (sequence, 256-row query tile); long rows of keys first
  int b = 0, tile = -1;
  {
    int acc = 0;
    const int want = gridDim.x - 1 - blockIdx.x;
    for (int i = 0; i < p.B; ++i) {
      const int nt = (p.q_len[i] + kTiles * kTileQ - 1) / (kTiles * kTileQ);
      if (want < acc + nt) {
        b = i;
        tile = want - acc;
        break;
      }
      acc += nt;
    }
    if (tile < 0) return;
  }
  const int head = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int q_len = p.q_len[b], prefix = p.prefix[b], seq = prefix + q_len, ctx0 = p.ctx_start[b] - (p.skip != nullptr ? p.skip[b] : 0);
  const int q0 = tile * kTiles * kTileQ;
  const KeyTiles<kTileK> keys(p.win, prefix + q0, prefix + min(q0 + kTiles * kTileQ, q_len) - 1);
  QueryTile qt[kTiles];
#pragma unroll
  for (int t = 0; t < kTiles; ++t)
    qt[t] = query_tile(p.win, keys, prefix + q0 + t * kTileQ, prefix + min(q0 + (t + 1) * kTileQ, q_len) - 1);
  const int n = max(qt[0].n, qt[1].n);

  if (threadIdx.x == 0) {
    prefetch_tmap(&map_qn);
    prefetch_tmap(&map_qr);
    prefetch_tmap(&map_k);
    prefetch_tmap(&map_kr);
    prefetch_tmap(&map_v);
    mbar_init(smem_u32(&bars->q_full), 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(smem_u32(&bars->k_full[i]), 1);
      mbar_init(smem_u32(&bars->k_empty[i]), 1);
      mbar_init(smem_u32(&bars->v_full[i]), 1);
      mbar_init(smem_u32(&bars->v_empty[i]), 1);
      for (int t = 0; t < kTiles; ++t) {
        mbar_init(smem_u32(&bars->s_full[t][i]), 1);
        mbar_init(smem_u32(&bars->p_ready[t][i]), 4);             // one arrival per softmax warp of the tile
        mbar_init(smem_u32(&bars->pv_done[t][i]), 1);
      }
    }
    bars->abort_flag = 0;
    fence_barrier_init();
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(&bars->tmem_slot), kTmemCols);
    tmem_relinquish();
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem = bars->tmem_slot;

  if (warp == 0) {
    // ------------------------------------------------------------------ TMA producer
    if (lane == 0) {
      const uint32_t qb = smem_u32(&bars->q_full);
      mbar_expect_tx(qb, kTiles * nb_q * kBlkQ);
      for (int t = 0; t < kTiles; ++t) {
        const int row = p.q_start[b] + q0 + t * kTileQ;           // rows past the projection read as zeros
        for (int c = 0; c < nb_q; ++c) {
          const uint32_t dst = smem_u32(q_s + (t * nb_q + c) * kBlkQ);
          if (c < p.nb_n) tma_load_3d(dst, &map_qn, qb, c * 64, head, row);
          else tma_load_3d(dst, &map_qr, qb, (c - p.nb_n) * 64, head, row);
        }
      }
      auto load = [&](int j, bool values) -> bool {
        const int st = j & 1;
        uint64_t* empty = values ? &bars->v_empty[st] : &bars->k_empty[st];
        if (!mbar_wait(smem_u32(empty), ((j >> 1) & 1) ^ 1)) {
          report(p.status, kTimeoutEmptyBarrier, b, j);
          *abort_flag = 1;
          return false;
        }
        const uint32_t fb = smem_u32(values ? &bars->v_full[st] : &bars->k_full[st]);
        const uint32_t dst = smem_u32(kv_s + st * stage_bytes) + (values ? nb_q * kBlkK : 0);
        const int row = ctx0 + keys.tile(j) * kTileK;
        if (values) {
          mbar_expect_tx(fb, p.nb_v * kBlkK);
          for (int c = 0; c < p.nb_v; ++c) tma_load_3d(dst + c * kBlkK, &map_v, fb, c * 64, head, row);
        } else {
          mbar_expect_tx(fb, nb_q * kBlkK);
          for (int c = 0; c < p.nb_n; ++c) tma_load_3d(dst + c * kBlkK, &map_k, fb, c * 64, head, row);
          for (int c = 0; c < p.nb_r; ++c) tma_load_3d(dst + (p.nb_n + c) * kBlkK, &map_kr, fb, c * 64, 0, row);
        }
        return true;
      };
      bool fed = load(0, false);
      for (int j = 0; fed && j < n && !*abort_flag; ++j) {
        if (j + 1 < n) fed = load(j + 1, false);
        if (fed) fed = load(j, true);
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issuer
    if (lane == 0) {
      constexpr uint32_t idesc_s = make_idesc(kTileQ, kTileK, 1, 1);
      const uint32_t idesc_pv = make_idesc(kTileQ, 64 * p.nb_v, 1, 1) | (1u << 16);      // B (values) is MN-major
      const int steps_n = (p.dim + 15) / 16, steps_r = (p.rot + 15) / 16;
      bool ok = mbar_wait(smem_u32(&bars->q_full), 0);
      if (!ok) report(p.status, kTimeoutFullBarrier, b, -1);
      tc_fence_after_sync();
      auto issue_pv = [&](int i) -> bool {
        if (!mbar_wait(smem_u32(&bars->v_full[i & 1]), (i >> 1) & 1)) {
          report(p.status, kTimeoutFullBarrier, b, 5000 + i);
          return false;
        }
        const uint32_t v_addr = smem_u32(kv_s + (i & 1) * stage_bytes) + nb_q * kBlkK;
        for (int t = 0; t < kTiles; ++t) {
          if (!qt[t].takes(i)) continue;
          const int li = qt[t].local(i);
          if (!mbar_wait(smem_u32(&bars->p_ready[t][li & 1]), (li >> 1) & 1)) {
            report(p.status, kTimeoutTmemFull, b, 1000 + i);
            return false;
          }
          tc_fence_after_sync();
          const uint32_t p_tm = tmem + t * kTmemTile + (li & 1) * kTileK, o_tm = tmem + t * kTmemTile + kTmemO;
#pragma unroll
          for (int term = 0; term < 2; ++term)
#pragma unroll
            for (int kk = 0; kk < kTileK / 16; ++kk)
              umma_bf16_ts(o_tm, p_tm + term * (kTileK / 2) + kk * 8,
                           make_smem_desc_sw128_mn(v_addr + kk * 16 * 128, kBlkK), idesc_pv,
                           (li > 0 || term > 0 || kk > 0) ? 1u : 0u);
          umma_commit(smem_u32(&bars->pv_done[t][li & 1]));
        }
        umma_commit(smem_u32(&bars->v_empty[i & 1]));
        return true;
      };
      for (int j = 0; ok && j < n && !*abort_flag; ++j) {
        const int st = j & 1;
        if (!mbar_wait(smem_u32(&bars->k_full[st]), (j >> 1) & 1)) {
          report(p.status, kTimeoutFullBarrier, b, j);
          ok = false;
          break;
        }
        const uint32_t k_addr = smem_u32(kv_s + st * stage_bytes);
        for (int t = 0; ok && t < kTiles; ++t) {
          if (!qt[t].takes(j)) continue;
          const int lj = qt[t].local(j), sb = lj & 1;
          // this S buffer holds P of the tile before last until its product is done
          if (lj >= 2 && !mbar_wait(smem_u32(&bars->pv_done[t][sb]), ((lj - 2) >> 1) & 1)) {
            report(p.status, kTimeoutTmemEmpty, b, j);
            ok = false;
            break;
          }
          tc_fence_after_sync();
          const uint32_t q_addr = smem_u32(q_s + t * nb_q * kBlkQ), s_tm = tmem + t * kTmemTile + sb * kTileK;
          for (int s = 0; s < steps_n + steps_r; ++s) {
            const int blk = s < steps_n ? s >> 2 : p.nb_n + ((s - steps_n) >> 2);
            const int sub = s < steps_n ? s & 3 : (s - steps_n) & 3;
            umma_bf16(s_tm, make_smem_desc_sw128(q_addr + blk * kBlkQ) + 2 * sub,
                      make_smem_desc_sw128(k_addr + blk * kBlkK) + 2 * sub, idesc_s, s > 0 ? 1u : 0u);
          }
          umma_commit(smem_u32(&bars->s_full[t][sb]));
        }
        if (!ok) break;
        umma_commit(smem_u32(&bars->k_empty[st]));
        if (j >= 1) ok = issue_pv(j - 1);
      }
      if (ok && !*abort_flag) ok = issue_pv(n - 1);
      if (!ok) *abort_flag = 1;
    }
  } else {
    // ------------------------------------------------------------------ softmax (one thread per query row)
    const int t = (warp - 2) >> 2, qd = warp & 3;
    const int row = qd * 32 + lane;
    const uint32_t tm = tmem + t * kTmemTile + (static_cast<uint32_t>(qd * 32) << 16);
    const int r_seq = q0 + t * kTileQ + row;                        // row within the sequence's new tokens
    const int kmax = r_seq >= q_len ? seq - 1 : prefix + r_seq;     // last visible key
    const int kmin = p.win.first(kmax);                             // first visible key
    const float scale_log2 = p.scale * kLog2E;
    const int nt = qt[t].count();
    float m_used = -INFINITY, l = 0.f;
    bool ok = nt > 0;
    for (int j = 0, lj = 0; ok && j < qt[t].n; ++j) {
      if (!qt[t].takes(j)) continue;
      const int st = lj & 1;
      // (votes keep the warp's control flow uniform: one lane per warp arrives on the barriers below)
      if (!__all_sync(0xffffffffu, mbar_wait(smem_u32(&bars->s_full[t][st]), (lj >> 1) & 1))) {
        report(p.status, kTimeoutTmemFull, b, j);
        *abort_flag = 1;
        ok = false;
        break;
      }
      tc_fence_after_sync();
      uint32_t v0[32], v1[32];
      const uint32_t s_addr = tm + st * kTileK;
      tmem_ld32(s_addr, v0);
      tmem_ld32(s_addr + 32, v1);
      tmem_ld_wait();
      // bit e: key e of this tile is visible
      const int k0 = keys.tile(j) * kTileK;
      auto below = [](int c) -> uint64_t { return c <= 0 ? 0ull : (c >= 64 ? ~0ull : (1ull << c) - 1); };
      const uint64_t seen = below(kmax - k0 + 1) & ~below(kmin - k0);
      const bool full = seen == ~0ull;
      const uint32_t see0 = static_cast<uint32_t>(seen), see1 = static_cast<uint32_t>(seen >> 32);
      float mx = -INFINITY;
      if (full) {
#pragma unroll
        for (int e = 0; e < 32; ++e) mx = fmaxf(mx, fmaxf(__uint_as_float(v0[e]), __uint_as_float(v1[e])));
      } else {
#pragma unroll
        for (int e = 0; e < 32; ++e) {
          if ((see0 >> e) & 1) mx = fmaxf(mx, __uint_as_float(v0[e]));
          if ((see1 >> e) & 1) mx = fmaxf(mx, __uint_as_float(v1[e]));
        }
      }
      mx *= scale_log2;
      const bool raise = lj > 0 && mx > m_used + kRescale;
      if (lj == 0) {
        m_used = mx;
      } else if (__any_sync(0xffffffffu, raise)) {
        // rare: bring O and the row sum to the new maximum, after the product in flight; tcgen05.ld / .st are
        // warp-collective, rows that do not need it take part with a factor of one
        if (!__all_sync(0xffffffffu, mbar_wait(smem_u32(&bars->pv_done[t][(lj - 1) & 1]), ((lj - 1) >> 1) & 1))) {
          report(p.status, kTimeoutTmemFull, b, 2000 + j);
          *abort_flag = 1;
          ok = false;
          break;
        }
        tc_fence_after_sync();
        const float f = raise ? exp2f(m_used - mx) : 1.f;
        l *= f;
#pragma unroll 1
        for (int c0 = 0; c0 < 64 * p.nb_v; c0 += 32) {
          uint32_t o[32];
          tmem_ld32(tm + kTmemO + c0, o);
          tmem_ld_wait();
#pragma unroll
          for (int e = 0; e < 32; ++e) o[e] = __float_as_uint(__uint_as_float(o[e]) * f);
          tmem_st32(tm + kTmemO + c0, o);
        }
        tmem_st_wait();
        if (raise) m_used = mx;
      }
      float sum = 0.f;
      const float ref = m_used == -INFINITY ? 0.f : m_used;         // (nothing seen so far)
      uint32_t hi[32], lo[32];
#pragma unroll
      for (int c = 0; c < 32; ++c) {
        const uint32_t a = c < 16 ? v0[2 * c] : v1[2 * c - 32], bb = c < 16 ? v0[2 * c + 1] : v1[2 * c - 31];
        float x = ex2_approx(fmaf(__uint_as_float(a), scale_log2, -ref));
        float y = ex2_approx(fmaf(__uint_as_float(bb), scale_log2, -ref));
        if (!full) {
          const uint32_t see = c < 16 ? see0 >> (2 * c) : see1 >> (2 * c - 32);
          if (!(see & 1)) x = 0.f;
          if (!(see & 2)) y = 0.f;
        }
        sum += x + y;
        hi[c] = pack_bf16(x, y);
        lo[c] = pack_bf16(x - __uint_as_float(hi[c] << 16), y - __uint_as_float(hi[c] & 0xffff0000u));
      }
      l += sum;
      tmem_st32(s_addr, hi);
      tmem_st32(s_addr + 32, lo);
      tmem_st_wait();
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(&bars->p_ready[t][st]));
      ++lj;
    }
    if (ok) {
      if (!__all_sync(0xffffffffu, mbar_wait(smem_u32(&bars->pv_done[t][(nt - 1) & 1]), ((nt - 1) >> 1) & 1))) {
        report(p.status, kTimeoutTmemFull, b, 3000);
        *abort_flag = 1;
      } else {
        tc_fence_after_sync();
        if (p.terms.sink != nullptr) l += exp2f(p.terms.sink_log2(head) - m_used);
        const float inv = l > 0.f ? 1.f / l : 0.f;
        __nv_bfloat16* orow = p.out + (p.q_start[b] + r_seq) * p.out_token_stride +
                              static_cast<long long>(head) * p.out_head_stride;
#pragma unroll 1
        for (int c0 = 0; c0 < p.vdim; c0 += 32) {
          uint32_t o[32];
          tmem_ld32(tm + kTmemO + c0, o);
          tmem_ld_wait();
          if (r_seq < q_len) {
#pragma unroll
            for (int e = 0; e < 32; e += 8)
              if (c0 + e < p.vdim)
                *reinterpret_cast<uint4*>(orow + c0 + e) =
                    make_uint4(pack_bf16(__uint_as_float(o[e]) * inv, __uint_as_float(o[e + 1]) * inv),
                               pack_bf16(__uint_as_float(o[e + 2]) * inv, __uint_as_float(o[e + 3]) * inv),
                               pack_bf16(__uint_as_float(o[e + 4]) * inv, __uint_as_float(o[e + 5]) * inv),
                               pack_bf16(__uint_as_float(o[e + 6]) * inv, __uint_as_float(o[e + 7]) * inv));
          }
        }
      }
    }
  }

  tc_fence_before_sync();
  __syncthreads();
  if (*abort_flag) {
    // give copies and products that are still in flight time to land before shared and tensor memory are released
    const uint64_t t0 = global_timer_ns();
    while (global_timer_ns() - t0 < 200000ull) __nanosleep(1000);
    __syncthreads();
  }
  if (warp == 1) {
    tc_fence_after_sync();
    tmem_dealloc(tmem, kTmemCols);
  }
}

int extend_smem(int dim, int rot, int vdim) {
  const int nb_q = (dim + 63) / 64 + (rot + 63) / 64, nb_v = (vdim + 63) / 64;
  const int need = kTiles * nb_q * kBlkQ + 2 * (nb_q + nb_v) * kBlkK + 256 + 1024;
  return need > kMinSmem ? need : kMinSmem;
}

}  // namespace
}  // namespace sglb

extern "C" {

// Whether the prefill kernel takes these head sizes.
int sglb_latent_extend_supported(int dim, int rot, int vdim) {
  return dim > 0 && rot > 0 && vdim > 0 && dim % 8 == 0 && rot % 8 == 0 && vdim % 8 == 0 && vdim <= 128 &&
         sglb::extend_smem(dim, rot, vdim) <= 227 * 1024;
}

// q: head h of token t at t * q_token_stride + h * (dim + rot), [unrotated | rotated] (total_q tokens);
// kv [ctx_total, heads, dim + vdim]; k_rot [ctx_total, rot]; out by strides.  B sequences with q_start / q_len (rows of q),
// prefix (tokens before them), ctx_start (first context row) and skip (tokens in front that have no context row, multiples of
// 64; null: none).  num_tiles = sum_b ceil(q_len / 256).  `window` (0: none): tokens a query sees, its own included; `sink`
// [heads] or null.
int sglb_latent_extend(const void* q, long long q_token_stride, int total_q, const void* kv, const void* k_rot,
                       int ctx_total, void* out, long long out_token_stride, int out_head_stride, const int* q_start,
                       const int* q_len, const int* prefix, const int* ctx_start, const int* skip, int B, int num_tiles,
                       int heads, int dim, int rot, int vdim, float scale, int window, const float* sink,
                       cudaStream_t stream) {
  using namespace sglb;
  if (B <= 0 || num_tiles <= 0 || total_q <= 0 || heads <= 0) return 0;
  if (!sglb_latent_extend_supported(dim, rot, vdim) || q_token_stride % 8 != 0 || out_token_stride % 8 != 0 ||
      out_head_stride % 8 != 0 || reinterpret_cast<uintptr_t>(out) % 16 != 0 || heads > 65535)
    return -kBadArgument;
  const __nv_bfloat16* qp = static_cast<const __nv_bfloat16*>(q);
  const __nv_bfloat16* kp = static_cast<const __nv_bfloat16*>(kv);
  const uint64_t qh = static_cast<uint64_t>(dim + rot) * 2, qt = static_cast<uint64_t>(q_token_stride) * 2;
  const uint64_t kh = static_cast<uint64_t>(dim + vdim) * 2, kt = kh * heads;
  CUtensorMap mqn, mqr, mk, mkr, mv;
  if (!encode_tmap_3d(&mqn, qp, dim, heads, total_q, qh, qt, kTileQ) ||
      !encode_tmap_3d(&mqr, qp + dim, rot, heads, total_q, qh, qt, kTileQ) ||
      !encode_tmap_3d(&mk, kp, dim, heads, ctx_total, kh, kt, kTileK) ||
      !encode_tmap_3d(&mkr, k_rot, rot, 1, ctx_total, static_cast<uint64_t>(rot) * 2, static_cast<uint64_t>(rot) * 2, kTileK) ||
      !encode_tmap_3d(&mv, kp + dim, vdim, heads, ctx_total, kh, kt, kTileK))
    return -100;
  Params p{};
  p.out = static_cast<__nv_bfloat16*>(out);
  p.out_token_stride = out_token_stride;
  p.out_head_stride = out_head_stride;
  p.q_start = q_start;
  p.q_len = q_len;
  p.prefix = prefix;
  p.ctx_start = ctx_start;
  p.skip = skip;
  p.status = device_status();
  p.B = B; p.dim = dim; p.rot = rot; p.vdim = vdim;
  p.nb_n = (dim + 63) / 64;
  p.nb_r = (rot + 63) / 64;
  p.nb_v = (vdim + 63) / 64;
  p.scale = scale;
  p.win = Window{window, 0};
  p.terms = ScoreTerms{0.f, nullptr, sink};
  const int smem = extend_smem(dim, rot, vdim);
  static int cfg = 0;
  if (cfg < smem) {
    const cudaError_t e = cudaFuncSetAttribute(latent_extend_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return static_cast<int>(e);
    cfg = smem;
  }
  latent_extend_kernel<<<dim3(num_tiles, heads), kThreads, smem, stream>>>(mqn, mqr, mk, mkr, mv, p);
  return static_cast<int>(cudaGetLastError());
}

}  // extern "C"
