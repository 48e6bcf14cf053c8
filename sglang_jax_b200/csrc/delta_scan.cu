// Gated delta rule over ragged batches, prefill and decode alike, the recurrence entirely in fp32:
//
//   delta_prep    short causal convolution + SiLU of the q / k / v channels of a fused projection (window = this step's
//                 rows, then the request's stored window, then zeros), unit q (times dim^-1/2) and k vectors, write
//                 strength beta = sigmoid(b) and decay g = exp(-exp(A_log) softplus(a + dt_bias))
//   delta_dots    scalar products of the k and q vectors inside blocks of four tokens (prefill)
//   delta_scan    S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q   in blocks of four tokens; columns of S
//                 are independent, so a CTA owns a few columns of one (sequence, head) and keeps them in registers from
//                 the first token to the last.  The state is read once and written once per step, whatever the number
//                 of tokens, and depends on how a prompt is cut by rounding only.  The convolution windows and the
//                 optional checkpoint (state after `track` tokens, for prefix sharing) are written here too.
//   delta_gate    rmsnorm(o) * w * silu(gate) per head, in the projections' type
//
// Both state tensors belong to `RecurrentStatePool`: windows [slots, channels, taps - 1], states [slots, H, D, V].
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

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

struct DeltaParams {
  const void* proj;              // [T, ld]: q | k | v channels at column 0, gate / b / a at the offsets below
  long long ld;
  int g_off, b_off, a_off;
  const void* conv_w;            // [channels, taps], channels = q | k | v
  const float* a_log;            // [H]
  const float* dt_bias;          // [H]
  void* conv_state;              // [slots, channels, taps - 1]
  float* state;                  // [slots, H, D, V]
  const long long* slots;        // [B]
  const int* cu;                 // [B + 1] first row of every sequence; null: one row each
  const int* prefix;             // [B] tokens before this step (0: start from zero state); null: continue
  const int* track_len;          // [B] tokens after which the state is also stored in track_slot (0: never); may be null
  const int* track_slot;         // [B]
  float* qk;                     // [T, Hk, 2, D] unit q * D^-1/2 | unit k
  float* v;                      // [T, H, V]
  float* gb;                     // [T, H, 2] decay, beta
  float* dots;                   // [T, Hk, 8], see delta_dots_kernel
  float* o;                      // [T, H, V]
  int B, T, H, Hk, D, V, taps;
};

// One warp per (run of RUN consecutive rows, head): the convolution window slides through registers.  A lane owns the
// channels lane, lane + 32, ... (NPL of them); TAPS >= taps, the kernel and the window are padded in front with zeros.
template <typename T, int NPL, int TAPS>
struct Conv {
  float w[NPL][TAPS], x[NPL][TAPS - 1];                // x[.][TAPS - 2] is the previous row

  __device__ __forceinline__ void load_kernel(const T* __restrict__ kernel, int c0, int width, int taps, int lane) {
#pragma unroll
    for (int i = 0; i < NPL; ++i)
#pragma unroll
      for (int j = 0; j < TAPS; ++j) {
        const int tap = j - (TAPS - taps), c = lane + 32 * i;
        w[i][j] = (tap >= 0 && c < width) ? to_f(kernel[static_cast<long long>(c0 + c) * taps + tap]) : 0.f;
      }
  }
  // window in front of row `start + local` of a sequence whose rows begin at `start`
  __device__ __forceinline__ void load_window(const T* __restrict__ proj, long long ld, const T* __restrict__ stored,
                                              bool fresh, int start, int local, int c0, int width, int taps, int lane) {
    const int win = taps - 1;
#pragma unroll
    for (int i = 0; i < NPL; ++i)
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j) {
        const int c = lane + 32 * i, back = TAPS - 1 - j, r = local - back;
        float v = 0.f;
        if (c < width && back <= win) {
          if (r >= 0) v = to_f(proj[(start + r) * ld + c0 + c]);
          else if (!fresh) v = to_f(stored[static_cast<long long>(c0 + c) * win + win + r]);
        }
        x[i][j] = v;
      }
  }
  // SiLU of the convolution at the next row, whose inputs are `in`
  __device__ __forceinline__ void step(const float (&in)[NPL], float (&out)[NPL]) {
#pragma unroll
    for (int i = 0; i < NPL; ++i) {
      float acc = w[i][TAPS - 1] * in[i];
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j) acc += w[i][j] * x[i][j];
#pragma unroll
      for (int j = 0; j < TAPS - 2; ++j) x[i][j] = x[i][j + 1];
      x[i][TAPS - 2] = in[i];
      out[i] = acc / (1.f + expf(-acc));
    }
  }
};

template <typename T, int NPL, int TAPS, int RUN>
__global__ void __launch_bounds__(128) delta_prep_kernel(const DeltaParams p) {
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int units = p.Hk + p.H;
  const long long wid = (blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x) >> 5;
  const long long runs = (p.T + RUN - 1) / RUN;
  if (wid >= runs * units) return;
  const int run = static_cast<int>(wid / units), unit = static_cast<int>(wid - static_cast<long long>(run) * units);
  const int t0 = run * RUN, t1 = min(t0 + RUN, p.T);
  int b0 = t0;
  if (p.cu != nullptr) {
    int lo = 0, hi = p.B - 1;
    while (lo < hi) {                                  // last sequence that starts at or before t0
      const int mid = (lo + hi + 1) >> 1;
      if (p.cu[mid] <= t0) lo = mid;
      else hi = mid - 1;
    }
    b0 = lo;
  }
  const int channels = 2 * p.Hk * p.D + p.H * p.V, taps = p.taps, win = taps - 1;
  const T* __restrict__ proj = static_cast<const T*>(p.proj);
  const T* __restrict__ kernel = static_cast<const T*>(p.conv_w);
  const T* __restrict__ windows = static_cast<const T*>(p.conv_state);
  // calls fn(t) for every row, after reload(b, start, local) wherever a sequence begins (or the run does)
  auto walk = [&](auto&& reload, auto&& fn) {
    int b = b0, end = t0;
    for (int t = t0; t < t1; ++t) {
      if (t == end || t == t0) {
        int start = t;
        if (p.cu != nullptr) {
          while (b + 1 < p.B && p.cu[b + 1] <= t) ++b;
          start = p.cu[b];
          end = b + 1 < p.B ? p.cu[b + 1] : p.T;
        } else {
          b = t;
          end = t + 1;
        }
        reload(windows + static_cast<long long>(p.slots[b]) * channels * win, p.prefix != nullptr && p.prefix[b] == 0,
               start, t - start);
      }
      fn(t);
    }
  };
  auto rows = [&](int t, int c0, int width, float (&in)[NPL]) {
    const T* src = proj + t * p.ld + c0;
#pragma unroll
    for (int i = 0; i < NPL; ++i) in[i] = lane + 32 * i < width ? to_f(src[lane + 32 * i]) : 0.f;
  };
  if (unit < p.Hk) {
    const int q0 = unit * p.D, k0 = p.Hk * p.D + unit * p.D;
    Conv<T, NPL, TAPS> cq, ck;
    cq.load_kernel(kernel, q0, p.D, taps, lane);
    ck.load_kernel(kernel, k0, p.D, taps, lane);
    const float scale = 1.f / sqrtf(static_cast<float>(p.D));
    walk(
        [&](const T* stored, bool fresh, int start, int local) {
          cq.load_window(proj, p.ld, stored, fresh, start, local, q0, p.D, taps, lane);
          ck.load_window(proj, p.ld, stored, fresh, start, local, k0, p.D, taps, lane);
        },
        [&](int t) {
          float in[NPL], q[NPL], k[NPL];
          rows(t, q0, p.D, in);
          cq.step(in, q);
          rows(t, k0, p.D, in);
          ck.step(in, k);
          float qq = 0.f, kk = 0.f;
#pragma unroll
          for (int i = 0; i < NPL; ++i) {
            qq += q[i] * q[i];
            kk += k[i] * k[i];
          }
#pragma unroll
          for (int o = 16; o > 0; o >>= 1) {
            qq += __shfl_xor_sync(0xffffffffu, qq, o);
            kk += __shfl_xor_sync(0xffffffffu, kk, o);
          }
          const float qs = scale / sqrtf(qq + 1e-6f), ks = 1.f / sqrtf(kk + 1e-6f);
          float* dst = p.qk + (static_cast<long long>(t) * p.Hk + unit) * 2 * p.D;
#pragma unroll
          for (int i = 0; i < NPL; ++i) {
            const int d = lane + 32 * i;
            if (d < p.D) {
              dst[d] = q[i] * qs;
              dst[p.D + d] = k[i] * ks;
            }
          }
        });
  } else {
    const int h = unit - p.Hk;
    for (int vb = 0; vb < p.V; vb += 32 * NPL) {
      const int v0 = 2 * p.Hk * p.D + h * p.V + vb, width = min(32 * NPL, p.V - vb);
      Conv<T, NPL, TAPS> cv;
      cv.load_kernel(kernel, v0, width, taps, lane);
      walk(
          [&](const T* stored, bool fresh, int start, int local) {
            cv.load_window(proj, p.ld, stored, fresh, start, local, v0, width, taps, lane);
          },
          [&](int t) {
            float in[NPL], v[NPL];
            rows(t, v0, width, in);
            cv.step(in, v);
            float* dst = p.v + (static_cast<long long>(t) * p.H + h) * p.V + vb;
#pragma unroll
            for (int i = 0; i < NPL; ++i)
              if (lane + 32 * i < width) dst[lane + 32 * i] = v[i];
          });
    }
    for (int t = t0 + lane; t < t1; t += 32) {
      const T* row = proj + static_cast<long long>(t) * p.ld;
      const float z = to_f(row[p.a_off + h]) + p.dt_bias[h];
      const float sp = fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)));
      float* gb = p.gb + (static_cast<long long>(t) * p.H + h) * 2;
      gb[0] = expf(-expf(p.a_log[h]) * sp);
      gb[1] = 1.f / (1.f + expf(-to_f(row[p.b_off + h])));
    }
  }
}

// Scalar products inside a block of kBlock tokens (blocks are counted from the first row of a sequence):
// dots[t][hk] = { k_j . k_t for the block's tokens j < t (kBlock - 1 places), k_j . q_t for j <= t (kBlock places) }.
constexpr int kBlock = 4;

__global__ void delta_dots_kernel(const DeltaParams p) {
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const long long wid = (blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x) >> 5;
  if (wid >= static_cast<long long>(p.T) * p.Hk) return;
  const int t = static_cast<int>(wid / p.Hk), hk = static_cast<int>(wid - static_cast<long long>(t) * p.Hk);
  int local = 0;
  if (p.cu != nullptr) {
    int lo = 0, hi = p.B - 1;
    while (lo < hi) {
      const int mid = (lo + hi + 1) >> 1;
      if (p.cu[mid] <= t) lo = mid;
      else hi = mid - 1;
    }
    local = t - p.cu[lo];
  }
  const int at = local % kBlock;                       // place of t in its block
  const long long stride = static_cast<long long>(p.Hk) * 2 * p.D;
  const float* own = p.qk + wid * 2 * p.D;
  float kk[kBlock], kq[kBlock];
#pragma unroll
  for (int j = 0; j < kBlock; ++j) kk[j] = kq[j] = 0.f;
  for (int d = lane; d < p.D; d += 32) {
    const float q = own[d], k = own[p.D + d];
#pragma unroll
    for (int j = 0; j < kBlock; ++j) {
      if (j <= at) {
        const float kj = j == at ? k : own[(j - at) * stride + p.D + d];
        kk[j] += kj * k;
        kq[j] += kj * q;
      }
    }
  }
#pragma unroll
  for (int j = 0; j < kBlock; ++j) {
    kk[j] = warp_sum(kk[j]);
    kq[j] = warp_sum(kq[j]);
  }
  if (lane == 0) {
    float4* dst = reinterpret_cast<float4*>(p.dots + wid * 2 * kBlock);
    dst[0] = make_float4(kk[0], kk[1], kk[2], 0.f);
    dst[1] = make_float4(kq[0], kq[1], kq[2], kq[3]);
  }
}

// ---------------------------------------------------------------------------------------------
constexpr int kScanThreads = 128;
constexpr int kChunk = 16;        // tokens staged in shared memory at a time (two buffers)
constexpr int kLanes = 8;         // lanes that share a column of the state

__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async4(void* dst, const void* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// RPL rows and CPL adjacent columns of the state per lane: D <= 8 * RPL, a CTA owns 16 * CPL columns.  CHUNK tokens are
// staged at a time; they are worked off in blocks of BLK: with S the state in front of a block, G_t the product of the
// block's decays up to and including t, and g_jt = G_t / G_j (again a product of decays),
//
//   u_t = beta_t (v_t - G_t S^T k_t - sum_{j<t} g_jt (k_j . k_t) u_j)
//   o_t = G_t S^T q_t + sum_{j<=t} g_jt (k_j . q_t) u_j          S <- G_n S + sum_j g_jn k_j u_j^T
//
// which is the recurrence with the block's read-outs taken from S at once: their reductions overlap.
template <int RPL, int CPL, int CHUNK>
struct ScanShape {
  static constexpr int kBlk = CHUNK < kBlock ? CHUNK : kBlock;
  static constexpr int kBufs = CHUNK == 1 ? 1 : 2;
  static constexpr int kDp = kLanes * RPL;
  static constexpr int kCols = (kScanThreads / kLanes) * CPL;
  static constexpr int kScal = 4 + 2 * kBlock;         // decay, beta, -, - | dots
  static constexpr int kStageFloats = CHUNK * (2 * kDp + kCols + kScal);
  static constexpr int kSmem = kBufs * kStageFloats * 4;
};

template <typename T, int RPL, int CPL, int CHUNK>
__global__ void __launch_bounds__(kScanThreads)
delta_scan_kernel(const DeltaParams p) {
  using Sh = ScanShape<RPL, CPL, CHUNK>;
  constexpr int BLK = Sh::kBlk;
  extern __shared__ float4 sm4[];
  float* sm = reinterpret_cast<float*>(sm4);
  pdl_wait();
  const int tid = threadIdx.x, lane = tid & 31, rl = lane & (kLanes - 1);
  const int b = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * Sh::kCols;
  const int hk = h / (p.H / p.Hk);
  const int start = p.cu != nullptr ? p.cu[b] : b;
  const int n = p.cu != nullptr ? p.cu[b + 1] - start : 1;
  if (n <= 0) return;
  const bool fresh = p.prefix != nullptr && p.prefix[b] == 0;
  const long long slot = p.slots[b];
  const int track = p.track_len != nullptr ? p.track_len[b] : 0;
  const int D = p.D, V = p.V;
  const int col = ((tid >> 5) * (32 / kLanes) + (lane / kLanes)) * CPL;      // first of this lane's columns in the CTA
  const long long plane = static_cast<long long>(D) * V;
  float* st = p.state + (slot * p.H + h) * plane;
  const int gc = c0 + col;                             // the same in the head
  const bool vec = CPL > 1 && V % CPL == 0;            // whole column groups: wide accesses

  // rows of this lane: groups of four, row = 4 * (i * kLanes + rl) + e
  auto row_of = [&](int i) { return 4 * ((i >> 2) * kLanes + rl) + (i & 3); };
  float S[RPL][CPL];
  auto store_state = [&](float* dst, const float (&M)[RPL][CPL]) {
#pragma unroll
    for (int i = 0; i < RPL; ++i) {
      const int r = row_of(i);
      float* d = dst + static_cast<long long>(r) * V + gc;
      if (r >= D || gc >= V) continue;
      if constexpr (CPL == 4) {
        if (vec) { *reinterpret_cast<float4*>(d) = make_float4(M[i][0], M[i][1], M[i][2], M[i][3]); continue; }
      }
      if constexpr (CPL == 2) {
        if (vec) { *reinterpret_cast<float2*>(d) = make_float2(M[i][0], M[i][1]); continue; }
      }
#pragma unroll
      for (int c = 0; c < CPL; ++c)
        if (gc + c < V) d[c] = M[i][c];
    }
  };
#pragma unroll
  for (int i = 0; i < RPL; ++i) {
    const int r = row_of(i);
    const float* d = st + static_cast<long long>(r) * V + gc;
#pragma unroll
    for (int c = 0; c < CPL; ++c) S[i][c] = 0.f;
    if (fresh || r >= D || gc >= V) continue;
    if constexpr (CPL == 4) {
      if (vec) {
        const float4 v = *reinterpret_cast<const float4*>(d);
        S[i][0] = v.x; S[i][1] = v.y; S[i][2] = v.z; S[i][3] = v.w;
        continue;
      }
    }
    if constexpr (CPL == 2) {
      if (vec) {
        const float2 v = *reinterpret_cast<const float2*>(d);
        S[i][0] = v.x; S[i][1] = v.y;
        continue;
      }
    }
#pragma unroll
    for (int c = 0; c < CPL; ++c)
      if (gc + c < V) S[i][c] = d[c];
  }
  // padding rows and columns, and the places of missing tokens, stay zero
  for (int i = tid; i < Sh::kBufs * Sh::kStageFloats; i += kScanThreads) sm[i] = 0.f;
  __syncthreads();

  auto stage = [&](int buf, int t0) {
    float* base = sm + buf * Sh::kStageFloats;
    const int m = min(CHUNK, n - t0);
    float* vs = base + CHUNK * 2 * Sh::kDp;
    float* ss = vs + CHUNK * Sh::kCols;
    const long long tok = static_cast<long long>(p.Hk) * 2 * D;
    const float* qk = p.qk + (start + t0) * tok + static_cast<long long>(hk) * 2 * D;
    // a warp per (token, q | k) vector
    for (int x = tid >> 5; x < 2 * m; x += kScanThreads / 32) {
      const float* src = qk + (x >> 1) * tok + (x & 1) * D;
      float* dst = base + x * Sh::kDp;
      if (D % 4 == 0)
        for (int e = lane * 4; e < D; e += 128) cp_async16(dst + e, src + e);
      else
        for (int e = lane; e < D; e += 32) cp_async4(dst + e, src + e);
    }
    for (int i = tid; i < m * Sh::kCols; i += kScanThreads) {
      const int tk = i / Sh::kCols, e = i % Sh::kCols;
      if (c0 + e < V) cp_async4(vs + i, p.v + (static_cast<long long>(start + t0 + tk) * p.H + h) * V + c0 + e);
    }
    if (tid < m) {
      const long long th = start + t0 + tid;
      cp_async4(ss + tid * Sh::kScal, p.gb + (th * p.H + h) * 2);
      cp_async4(ss + tid * Sh::kScal + 1, p.gb + (th * p.H + h) * 2 + 1);
      if (BLK > 1) {
        cp_async16(ss + tid * Sh::kScal + 4, p.dots + (th * p.Hk + hk) * 2 * kBlock);
        cp_async16(ss + tid * Sh::kScal + 8, p.dots + (th * p.Hk + hk) * 2 * kBlock + 4);
      }
    }
    cp_commit();
  };

  stage(0, 0);
  for (int t0 = 0, buf = 0; t0 < n; t0 += CHUNK, buf ^= (Sh::kBufs - 1)) {
    if (Sh::kBufs == 2 && t0 + CHUNK < n) {
      stage(buf ^ 1, t0 + CHUNK);
      cp_wait<1>();
    } else {
      cp_wait<0>();
    }
    __syncthreads();
    const float* base = sm + buf * Sh::kStageFloats;
    const float* vs = base + CHUNK * 2 * Sh::kDp;
    const float* ss = vs + CHUNK * Sh::kCols;
    const int m = min(CHUNK, n - t0);
#pragma unroll 1
    for (int t = 0; t < m; t += BLK) {
      const int nb = min(BLK, m - t);                  // tokens of this block
      float kd[BLK][CPL], qd[BLK][CPL];
      float self = 0.f;                                // k . q of a single token
#pragma unroll
      for (int j = 0; j < BLK; ++j) {
#pragma unroll
        for (int c = 0; c < CPL; ++c) kd[j][c] = qd[j][c] = 0.f;
        const float4* qv = reinterpret_cast<const float4*>(base + (t + j) * 2 * Sh::kDp) + rl;
        const float4* kv = reinterpret_cast<const float4*>(base + (t + j) * 2 * Sh::kDp + Sh::kDp) + rl;
#pragma unroll
        for (int i = 0; i < RPL; i += 4) {
          const float4 k4 = kv[(i >> 2) * kLanes], q4 = qv[(i >> 2) * kLanes];
#pragma unroll
          for (int c = 0; c < CPL; ++c) {
            kd[j][c] += S[i][c] * k4.x + S[i + 1][c] * k4.y + S[i + 2][c] * k4.z + S[i + 3][c] * k4.w;
            qd[j][c] += S[i][c] * q4.x + S[i + 1][c] * q4.y + S[i + 2][c] * q4.z + S[i + 3][c] * q4.w;
          }
          if (BLK == 1) self += k4.x * q4.x + k4.y * q4.y + k4.z * q4.z + k4.w * q4.w;
        }
      }
#pragma unroll
      for (int o = kLanes / 2; o > 0; o >>= 1) {
#pragma unroll
        for (int j = 0; j < BLK; ++j)
#pragma unroll
          for (int c = 0; c < CPL; ++c) {
            kd[j][c] += __shfl_xor_sync(0xffffffffu, kd[j][c], o);
            qd[j][c] += __shfl_xor_sync(0xffffffffu, qd[j][c], o);
          }
        if (BLK == 1) self += __shfl_xor_sync(0xffffffffu, self, o);
      }
      float u[BLK][CPL], g[BLK];
#pragma unroll
      for (int j = 0; j < BLK; ++j) {
        const float* sc = ss + (t + j) * Sh::kScal;
        g[j] = j < nb ? sc[0] : 1.f;
        const float beta = j < nb ? sc[1] : 0.f;
        // decay[i] = product of g over tokens i + 1 .. j, decay of the state itself in front of them
        float from[BLK], G = g[j];
        from[j] = 1.f;
#pragma unroll
        for (int i = j - 1; i >= 0; --i) {
          from[i] = G;
          G *= g[i];
        }
        float out[CPL];
#pragma unroll
        for (int c = 0; c < CPL; ++c) {
          float a = G * kd[j][c];
          out[c] = G * qd[j][c];
#pragma unroll
          for (int i = 0; i < j; ++i) {
            a += from[i] * sc[4 + i] * u[i][c];
            out[c] += from[i] * sc[4 + kBlock + i] * u[i][c];
          }
          u[j][c] = beta * (vs[(t + j) * Sh::kCols + col + c] - a);
          out[c] += (BLK == 1 ? self : sc[4 + kBlock + j]) * u[j][c];
        }
        if (rl == 0 && j < nb) {
          float* d = p.o + (static_cast<long long>(start + t0 + t + j) * p.H + h) * V + gc;
#pragma unroll
          for (int c = 0; c < CPL; ++c)
            if (gc + c < V) d[c] = out[c];
        }
      }
      // the state after the block's first `upto` tokens
      auto advance = [&](int upto, float (&M)[RPL][CPL]) {
        float w[BLK], G = 1.f;
#pragma unroll
        for (int j = BLK - 1; j >= 0; --j) {
          w[j] = j < upto ? G : 0.f;
          if (j < upto) G *= g[j];
        }
#pragma unroll
        for (int i = 0; i < RPL; ++i)
#pragma unroll
          for (int c = 0; c < CPL; ++c) M[i][c] = G * S[i][c];
#pragma unroll
        for (int j = 0; j < BLK; ++j) {
          const float4* kv = reinterpret_cast<const float4*>(base + (t + j) * 2 * Sh::kDp + Sh::kDp) + rl;
          float wu[CPL];
#pragma unroll
          for (int c = 0; c < CPL; ++c) wu[c] = w[j] * u[j][c];
#pragma unroll
          for (int i = 0; i < RPL; i += 4) {
            const float4 k4 = kv[(i >> 2) * kLanes];
#pragma unroll
            for (int c = 0; c < CPL; ++c) {
              M[i][c] += k4.x * wu[c];
              M[i + 1][c] += k4.y * wu[c];
              M[i + 2][c] += k4.z * wu[c];
              M[i + 3][c] += k4.w * wu[c];
            }
          }
        }
      };
      if (track > t0 + t && track <= t0 + t + nb) {
        float M[RPL][CPL];
        advance(track - t0 - t, M);
        store_state(p.state + (static_cast<long long>(p.track_slot[b]) * p.H + h) * plane, M);
      }
      advance(nb, S);
    }
    __syncthreads();                                   // this buffer is refilled in the next round
  }
  store_state(st, S);

  // convolution windows of this head's channels (the q / k channels by the first value head that uses them)
  if (blockIdx.z == 0) {
    const int win = p.taps - 1, channels = 2 * p.Hk * D + p.H * V;
    const T* proj = static_cast<const T*>(p.proj) + start * p.ld;
    T* cs = static_cast<T*>(p.conv_state);
    T* own = cs + slot * channels * win;
    auto window = [&](int c) {
      T* w = own + static_cast<long long>(c) * win;
      auto input = [&](int i) {                        // input number i of this step (negative: before it)
        return i >= 0 ? proj[i * p.ld + c] : (fresh ? from_f<T>(0.f) : w[win + i]);
      };
      if (track > 0 && track <= n) {
        T* sw = cs + (static_cast<long long>(p.track_slot[b]) * channels + c) * win;
        for (int j = 0; j < win; ++j) sw[j] = input(track - win + j);
      }
      for (int j = 0; j < win; ++j) w[j] = input(n - win + j);      // reads w[j + n] before w[j + n] is overwritten
    };
    for (int i = tid; i < V; i += kScanThreads) window(2 * p.Hk * D + h * V + i);
    if (h % (p.H / p.Hk) == 0) {
      for (int i = tid; i < D; i += kScanThreads) {
        window(hk * D + i);
        window(p.Hk * D + hk * D + i);
      }
    }
  }
}

// One warp per (token, head); a lane holds NV groups of four adjacent columns (V <= 128 * NV, V % 4 == 0), or takes single
// columns (NV = 0, any V).
template <typename T, int NV>
__global__ void delta_gate_kernel(const float* __restrict__ o, const T* __restrict__ gate, long long ld,
                                  const float* __restrict__ w, T* __restrict__ out, long long T_, int H, int V, float eps) {
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const long long wid = (blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x) >> 5;
  if (wid >= T_ * H) return;
  const long long t = wid / H;
  const int h = static_cast<int>(wid - t * H);
  const float* src = o + wid * V;
  const T* g = gate + t * ld + static_cast<long long>(h) * V;
  T* dst = out + wid * V;
  auto gated = [](float x, float gv) { return x * (gv / (1.f + expf(-gv))); };
  float ss = 0.f;
  if constexpr (NV > 0) {
    float4 v[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (lane + 32 * i) * 4;
      v[i] = c < V ? *reinterpret_cast<const float4*>(src + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    }
    const float inv = 1.f / sqrtf(warp_sum(ss) / V + eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (lane + 32 * i) * 4;
      if (c >= V) continue;
      const float4 wv = *reinterpret_cast<const float4*>(w + c);
      if constexpr (sizeof(T) == 2) {
        const uint2 raw = *reinterpret_cast<const uint2*>(g + c);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
        *reinterpret_cast<uint2*>(dst + c) =
            make_uint2(pack_bf16(gated(v[i].x * inv * wv.x, a.x), gated(v[i].y * inv * wv.y, a.y)),
                       pack_bf16(gated(v[i].z * inv * wv.z, b.x), gated(v[i].w * inv * wv.w, b.y)));
      } else {
        const float4 a = *reinterpret_cast<const float4*>(g + c);
        *reinterpret_cast<float4*>(dst + c) =
            make_float4(gated(v[i].x * inv * wv.x, a.x), gated(v[i].y * inv * wv.y, a.y),
                        gated(v[i].z * inv * wv.z, a.z), gated(v[i].w * inv * wv.w, a.w));
      }
    }
  } else {
    for (int i = lane; i < V; i += 32) ss += src[i] * src[i];
    const float inv = 1.f / sqrtf(warp_sum(ss) / V + eps);
    for (int i = lane; i < V; i += 32) dst[i] = from_f<T>(gated(src[i] * inv * w[i], to_f(g[i])));
  }
}

template <typename T>
int run_gate(const float* o, const void* gate, long long ld, const float* w, void* out, long long n, int H, int V,
             float eps, cudaStream_t s) {
  const dim3 grid(static_cast<unsigned>((n * H + 3) / 4));
  const T* g = static_cast<const T*>(gate);
  T* d = static_cast<T*>(out);
  const bool vec = V % 4 == 0 && ld % 4 == 0 && reinterpret_cast<uintptr_t>(gate) % (4 * sizeof(T)) == 0;
  if (vec && V <= 128) launch_pdl(delta_gate_kernel<T, 1>, grid, dim3(128), 0, s, o, g, ld, w, d, n, H, V, eps);
  else if (vec && V <= 256) launch_pdl(delta_gate_kernel<T, 2>, grid, dim3(128), 0, s, o, g, ld, w, d, n, H, V, eps);
  else launch_pdl(delta_gate_kernel<T, 0>, grid, dim3(128), 0, s, o, g, ld, w, d, n, H, V, eps);
  return static_cast<int>(cudaGetLastError());
}

template <typename T, int NPL, int TAPS>
int launch_prep(const DeltaParams& p, cudaStream_t s) {
  const int units = p.Hk + p.H;
  auto blocks = [&](int run) {
    return dim3(static_cast<unsigned>(((static_cast<long long>(p.T) + run - 1) / run * units + 3) / 4));
  };
  // long runs reuse the window and the kernel; short steps want the warps
  if (p.cu != nullptr && static_cast<long long>(p.T) * units >= 16 * 148 * 32)
    launch_pdl(delta_prep_kernel<T, NPL, TAPS, 16>, blocks(16), dim3(128), 0, s, p);
  else
    launch_pdl(delta_prep_kernel<T, NPL, TAPS, 1>, blocks(1), dim3(128), 0, s, p);
  return static_cast<int>(cudaGetLastError());
}

template <typename T, int RPL, int CPL, int CHUNK>
int launch_scan(const DeltaParams& p, cudaStream_t s) {
  using Sh = ScanShape<RPL, CPL, CHUNK>;
  static bool cfg = false;
  if (!cfg) {
    const cudaError_t e = cudaFuncSetAttribute(delta_scan_kernel<T, RPL, CPL, CHUNK>,
                                               cudaFuncAttributeMaxDynamicSharedMemorySize, Sh::kSmem);
    if (e != cudaSuccess) return static_cast<int>(e);
    cfg = true;
  }
  launch_pdl(delta_scan_kernel<T, RPL, CPL, CHUNK>, dim3(p.B, p.H, (p.V + Sh::kCols - 1) / Sh::kCols),
             dim3(kScanThreads), Sh::kSmem, s, p);
  return static_cast<int>(cudaGetLastError());
}

template <typename T, int RPL>
int launch_rows(const DeltaParams& p, cudaStream_t s) {
  const long long groups = static_cast<long long>(p.B) * p.H * ((p.V + 15) / 16);      // 16-column slices of all states
  if (p.cu == nullptr) {                               // one token each: the state streams through once
    if (RPL <= 16 && groups >= 148 * 32) return launch_scan<T, RPL, (RPL <= 16 ? 4 : 1), 1>(p, s);
    if (RPL <= 16 && groups >= 148 * 8) return launch_scan<T, RPL, (RPL <= 16 ? 2 : 1), 1>(p, s);
    return launch_scan<T, RPL, 1, 1>(p, s);
  }
  // two columns per lane once that still leaves the machine full: fewer shared-memory reads per state element
  if (RPL <= 16 && groups >= 148 * 8) return launch_scan<T, RPL, (RPL <= 16 ? 2 : 1), 16>(p, s);
  return launch_scan<T, RPL, 1, 16>(p, s);
}

template <typename T>
int run_delta(const DeltaParams& p, cudaStream_t s) {
  const int wide = p.D > p.V ? p.D : p.V;
  int e;
  if (p.taps <= 4)
    e = wide <= 64 ? launch_prep<T, 2, 4>(p, s) : wide <= 128 ? launch_prep<T, 4, 4>(p, s) : launch_prep<T, 8, 4>(p, s);
  else
    e = wide <= 128 ? launch_prep<T, 4, 16>(p, s) : launch_prep<T, 8, 16>(p, s);
  if (e != 0) return e;
  if (p.cu != nullptr) {
    const long long warps = static_cast<long long>(p.T) * p.Hk;
    launch_pdl(delta_dots_kernel, dim3(static_cast<unsigned>((warps + 3) / 4)), dim3(128), 0, s, p);
    e = static_cast<int>(cudaGetLastError());
    if (e != 0) return e;
  }
  const int rows = (p.D + kLanes - 1) / kLanes;
  if (rows <= 4) return launch_rows<T, 4>(p, s);
  if (rows <= 8) return launch_rows<T, 8>(p, s);
  if (rows <= 16) return launch_rows<T, 16>(p, s);
  return launch_rows<T, 32>(p, s);
}

}  // namespace
}  // namespace sglb

extern "C" {

// Shapes in DeltaParams; T = bf16 or fp32 (`is_f32`) is the type of `proj`, `conv_w` and `conv_state`.
int sglb_delta_scan(const void* proj, long long ld, int g_off, int b_off, int a_off, const void* conv_w,
                    const float* a_log, const float* dt_bias, void* conv_state, float* state, const long long* slots,
                    const int* cu, const int* prefix, const int* track_len, const int* track_slot, float* qk, float* v,
                    float* gb, float* dots, float* o, int B, int T, int H, int Hk, int D, int V, int taps, int is_f32,
                    cudaStream_t s) {
  using namespace sglb;
  if (B <= 0 || T <= 0) return 0;
  if (D < 1 || D > 32 * kLanes || V < 1 || Hk < 1 || H % Hk != 0 || taps < 1 || taps > 16 || H > 65535) return -kBadArgument;
  DeltaParams p{proj, ld, g_off, b_off, a_off, conv_w, a_log, dt_bias, conv_state, state, slots, cu, prefix, track_len,
                track_slot, qk, v, gb, dots, o, B, T, H, Hk, D, V, taps};
  return is_f32 ? run_delta<float>(p, s) : run_delta<__nv_bfloat16>(p, s);
}

// out [T, H * V] = rmsnorm(o [T, H, V], over V) * w [V] * silu(gate), gate at row stride `ld`.
int sglb_delta_gate(const float* o, const void* gate, long long ld, const float* w, void* out, long long T, int H, int V,
                    float eps, int is_f32, cudaStream_t s) {
  using namespace sglb;
  if (T <= 0) return 0;
  return is_f32 ? run_gate<float>(o, gate, ld, w, out, T, H, V, eps, s)
                : run_gate<__nv_bfloat16>(o, gate, ld, w, out, T, H, V, eps, s);
}

}  // extern "C"
