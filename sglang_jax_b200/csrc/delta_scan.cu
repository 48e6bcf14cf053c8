// Gated delta rule over ragged batches, prefill and decode alike, the recurrence entirely in fp32:
//
//   delta_prep    short causal convolution + SiLU of the q / k / v channels of a fused projection (window = this step's
//                 rows, then the request's stored window, then zeros), unit q (times dim^-1/2) and k vectors, write
//                 strength beta = sigmoid(b) and decay g = exp(-exp(A_log) softplus(a + dt_bias)); one warp per
//                 (token, head)
//   delta_scan    S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q   token after token; columns of S are
//                 independent, so a CTA owns a few columns of one (sequence, head) and keeps them in registers from
//                 the first token to the last.  The state is read once and written once per step, whatever the number
//                 of tokens, and its value does not depend on how a prompt is cut.  The convolution windows and the
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
  float* kq;                     // [T, Hk] k . q
  float* o;                      // [T, H, V]
  int B, T, H, Hk, D, V, taps;
};

constexpr int kMaxPerLane = 16;   // head widths up to 512 in delta_prep

template <typename T>
__global__ void delta_prep_kernel(const DeltaParams p) {
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int units = p.Hk + p.H;
  const long long wid = (blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x) >> 5;
  if (wid >= static_cast<long long>(p.T) * units) return;
  const int t = static_cast<int>(wid / units), unit = static_cast<int>(wid - static_cast<long long>(t) * units);
  int b = t, start = t;
  if (p.cu != nullptr) {
    int lo = 0, hi = p.B - 1;
    while (lo < hi) {                                  // last sequence that starts at or before t
      const int mid = (lo + hi + 1) >> 1;
      if (p.cu[mid] <= t) lo = mid;
      else hi = mid - 1;
    }
    b = lo;
    start = p.cu[lo];
  }
  const bool fresh = p.prefix != nullptr && p.prefix[b] == 0;
  const int channels = 2 * p.Hk * p.D + p.H * p.V, taps = p.taps, win = taps - 1;
  const T* proj = static_cast<const T*>(p.proj);
  const T* w = static_cast<const T*>(p.conv_w);
  const T* st = static_cast<const T*>(p.conv_state) + static_cast<long long>(p.slots[b]) * channels * win;
  auto conv = [&](int c) {
    float acc = 0.f;
    for (int j = 0; j < taps; ++j) {
      const int i = t - start - (win - j);             // index of this tap's input among the step's rows
      float x = 0.f;
      if (i >= 0) x = to_f(proj[(start + i) * p.ld + c]);
      else if (!fresh) x = to_f(st[static_cast<long long>(c) * win + win + i]);
      acc += to_f(w[static_cast<long long>(c) * taps + j]) * x;
    }
    return acc / (1.f + expf(-acc));
  };
  if (unit < p.Hk) {
    float q[kMaxPerLane], k[kMaxPerLane];
    float qq = 0.f, kk = 0.f;
    const int q0 = unit * p.D, k0 = p.Hk * p.D + unit * p.D;
#pragma unroll
    for (int i = 0; i < kMaxPerLane; ++i) {
      const int d = lane + 32 * i;
      if (d < p.D) {
        q[i] = conv(q0 + d);
        k[i] = conv(k0 + d);
        qq += q[i] * q[i];
        kk += k[i] * k[i];
      }
    }
    const float qs = 1.f / sqrtf(warp_sum(qq) + 1e-6f) / sqrtf(static_cast<float>(p.D));
    const float ks = 1.f / sqrtf(warp_sum(kk) + 1e-6f);
    float* dst = p.qk + (static_cast<long long>(t) * p.Hk + unit) * 2 * p.D;
    float dot = 0.f;
#pragma unroll
    for (int i = 0; i < kMaxPerLane; ++i) {
      const int d = lane + 32 * i;
      if (d < p.D) {
        const float qv = q[i] * qs, kv = k[i] * ks;
        dst[d] = qv;
        dst[p.D + d] = kv;
        dot += qv * kv;
      }
    }
    dot = warp_sum(dot);
    if (lane == 0) p.kq[static_cast<long long>(t) * p.Hk + unit] = dot;
  } else {
    const int h = unit - p.Hk;
    const int v0 = 2 * p.Hk * p.D + h * p.V;
    float* dst = p.v + (static_cast<long long>(t) * p.H + h) * p.V;
    for (int d = lane; d < p.V; d += 32) dst[d] = conv(v0 + d);
    if (lane == 0) {
      const T* row = proj + static_cast<long long>(t) * p.ld;
      const float bv = to_f(row[p.b_off + h]);
      const float z = to_f(row[p.a_off + h]) + p.dt_bias[h];
      const float sp = fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)));
      float* gb = p.gb + (static_cast<long long>(t) * p.H + h) * 2;
      gb[0] = expf(-expf(p.a_log[h]) * sp);
      gb[1] = 1.f / (1.f + expf(-bv));
    }
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

// RPL rows and CPL columns of the state per lane: D <= 8 * RPL, a CTA owns 16 * CPL columns.
template <int RPL, int CPL>
struct ScanShape {
  static constexpr int kDp = kLanes * RPL;
  static constexpr int kCols = (kScanThreads / kLanes) * CPL;
  static constexpr int kStageFloats = kChunk * (2 * kDp + kCols + 4);
  static constexpr int kSmem = 2 * kStageFloats * 4;
};

template <typename T, int RPL, int CPL>
__global__ void __launch_bounds__(kScanThreads)
delta_scan_kernel(const DeltaParams p) {
  using Sh = ScanShape<RPL, CPL>;
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

  // rows of this lane: groups of four, row = 4 * (i * kLanes + rl) + e
  float S[RPL][CPL];
#pragma unroll
  for (int i = 0; i < RPL; ++i) {
    const int r = 4 * ((i >> 2) * kLanes + rl) + (i & 3);
#pragma unroll
    for (int c = 0; c < CPL; ++c)
      S[i][c] = (!fresh && r < D && c0 + col + c < V) ? st[static_cast<long long>(r) * V + c0 + col + c] : 0.f;
  }
  for (int i = tid; i < 2 * Sh::kStageFloats; i += kScanThreads) sm[i] = 0.f;      // padding rows and columns stay zero
  __syncthreads();

  auto stage = [&](int buf, int t0) {
    float* base = sm + buf * Sh::kStageFloats;
    const int m = min(kChunk, n - t0);
    float* vs = base + kChunk * 2 * Sh::kDp;
    float* ss = vs + kChunk * Sh::kCols;
    const float* qk = p.qk + (static_cast<long long>(start + t0) * p.Hk + hk) * 2 * D;
    const long long tok = static_cast<long long>(p.Hk) * 2 * D;
    if (D % 4 == 0) {
      const int per = D / 4;
      for (int i = tid; i < m * 2 * per; i += kScanThreads) {
        const int tk = i / (2 * per), j = i - tk * 2 * per, which = j >= per, e = j - which * per;
        cp_async16(base + tk * 2 * Sh::kDp + which * Sh::kDp + e * 4, qk + tk * tok + which * D + e * 4);
      }
    } else {
      for (int i = tid; i < m * 2 * D; i += kScanThreads) {
        const int tk = i / (2 * D), j = i - tk * 2 * D, which = j >= D, e = j - which * D;
        cp_async4(base + tk * 2 * Sh::kDp + which * Sh::kDp + e, qk + tk * tok + which * D + e);
      }
    }
    const int cols = min(Sh::kCols, V - c0);
    for (int i = tid; i < m * cols; i += kScanThreads) {
      const int tk = i / cols, e = i - tk * cols;
      cp_async4(vs + tk * Sh::kCols + e, p.v + (static_cast<long long>(start + t0 + tk) * p.H + h) * V + c0 + e);
    }
    for (int tk = tid; tk < m; tk += kScanThreads) {
      const long long th = static_cast<long long>(start + t0 + tk);
      cp_async4(ss + tk * 4, p.gb + (th * p.H + h) * 2);
      cp_async4(ss + tk * 4 + 1, p.gb + (th * p.H + h) * 2 + 1);
      cp_async4(ss + tk * 4 + 2, p.kq + th * p.Hk + hk);
    }
    cp_commit();
  };

  stage(0, 0);
  for (int t0 = 0, buf = 0; t0 < n; t0 += kChunk, buf ^= 1) {
    if (t0 + kChunk < n) {
      stage(buf ^ 1, t0 + kChunk);
      cp_wait<1>();
    } else {
      cp_wait<0>();
    }
    __syncthreads();
    const float* base = sm + buf * Sh::kStageFloats;
    const float* vs = base + kChunk * 2 * Sh::kDp;
    const float* ss = vs + kChunk * Sh::kCols;
    const int m = min(kChunk, n - t0);
    for (int tk = 0; tk < m; ++tk) {
      const float4* qv = reinterpret_cast<const float4*>(base + tk * 2 * Sh::kDp) + rl;
      const float4* kv = reinterpret_cast<const float4*>(base + tk * 2 * Sh::kDp + Sh::kDp) + rl;
      const float4 sc = *reinterpret_cast<const float4*>(ss + tk * 4);           // decay, beta, k . q
      float kd[CPL], qd[CPL];
#pragma unroll
      for (int c = 0; c < CPL; ++c) kd[c] = qd[c] = 0.f;
      float kr[RPL];
#pragma unroll
      for (int i = 0; i < RPL; i += 4) {
        const float4 k4 = kv[(i >> 2) * kLanes], q4 = qv[(i >> 2) * kLanes];
        kr[i] = k4.x; kr[i + 1] = k4.y; kr[i + 2] = k4.z; kr[i + 3] = k4.w;
#pragma unroll
        for (int c = 0; c < CPL; ++c) {
          kd[c] += S[i][c] * k4.x + S[i + 1][c] * k4.y + S[i + 2][c] * k4.z + S[i + 3][c] * k4.w;
          qd[c] += S[i][c] * q4.x + S[i + 1][c] * q4.y + S[i + 2][c] * q4.z + S[i + 3][c] * q4.w;
        }
      }
#pragma unroll
      for (int o = kLanes / 2; o > 0; o >>= 1) {
#pragma unroll
        for (int c = 0; c < CPL; ++c) {
          kd[c] += __shfl_xor_sync(0xffffffffu, kd[c], o);
          qd[c] += __shfl_xor_sync(0xffffffffu, qd[c], o);
        }
      }
#pragma unroll
      for (int c = 0; c < CPL; ++c) {
        const float u = sc.y * (vs[tk * Sh::kCols + col + c] - sc.x * kd[c]);
        // o = S'^T q with S' = g S + k u^T, that is g (S^T q) + u (k . q)
        if (rl == 0 && c0 + col + c < V)
          p.o[(static_cast<long long>(start + t0 + tk) * p.H + h) * V + c0 + col + c] = sc.x * qd[c] + u * sc.z;
#pragma unroll
        for (int i = 0; i < RPL; ++i) S[i][c] = sc.x * S[i][c] + kr[i] * u;
      }
      if (t0 + tk + 1 == track) {
        float* snap = p.state + (static_cast<long long>(p.track_slot[b]) * p.H + h) * plane;
#pragma unroll
        for (int i = 0; i < RPL; ++i) {
          const int r = 4 * ((i >> 2) * kLanes + rl) + (i & 3);
#pragma unroll
          for (int c = 0; c < CPL; ++c)
            if (r < D && c0 + col + c < V) snap[static_cast<long long>(r) * V + c0 + col + c] = S[i][c];
        }
      }
    }
    __syncthreads();                                   // this buffer is refilled in the next round
  }
#pragma unroll
  for (int i = 0; i < RPL; ++i) {
    const int r = 4 * ((i >> 2) * kLanes + rl) + (i & 3);
#pragma unroll
    for (int c = 0; c < CPL; ++c)
      if (r < D && c0 + col + c < V) st[static_cast<long long>(r) * V + c0 + col + c] = S[i][c];
  }

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

template <typename T>
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
  float ss = 0.f;
  for (int i = lane; i < V; i += 32) ss += src[i] * src[i];
  const float inv = 1.f / sqrtf(warp_sum(ss) / V + eps);
  for (int i = lane; i < V; i += 32) {
    const float gv = to_f(g[i]);
    dst[i] = from_f<T>(src[i] * inv * w[i] * (gv / (1.f + expf(-gv))));
  }
}

template <typename T, int RPL, int CPL>
int launch_scan(const DeltaParams& p, cudaStream_t s) {
  using Sh = ScanShape<RPL, CPL>;
  static bool cfg = false;
  if (!cfg) {
    const cudaError_t e = cudaFuncSetAttribute(delta_scan_kernel<T, RPL, CPL>,
                                               cudaFuncAttributeMaxDynamicSharedMemorySize, Sh::kSmem);
    if (e != cudaSuccess) return static_cast<int>(e);
    cfg = true;
  }
  launch_pdl(delta_scan_kernel<T, RPL, CPL>, dim3(p.B, p.H, (p.V + Sh::kCols - 1) / Sh::kCols), dim3(kScanThreads),
             Sh::kSmem, s, p);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
int run_delta(const DeltaParams& p, cudaStream_t s) {
  const long long warps = static_cast<long long>(p.T) * (p.Hk + p.H);
  launch_pdl(delta_prep_kernel<T>, dim3(static_cast<unsigned>((warps + 3) / 4)), dim3(128), 0, s, p);
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) return static_cast<int>(e);
  // two columns per lane once that still leaves the machine full: fewer shared-memory reads per state element
  const bool wide = static_cast<long long>(p.B) * p.H * ((p.V + 15) / 16) >= 148 * 8;
  const int rows = (p.D + kLanes - 1) / kLanes;
  if (rows <= 4) return wide ? launch_scan<T, 4, 2>(p, s) : launch_scan<T, 4, 1>(p, s);
  if (rows <= 8) return wide ? launch_scan<T, 8, 2>(p, s) : launch_scan<T, 8, 1>(p, s);
  if (rows <= 16) return wide ? launch_scan<T, 16, 2>(p, s) : launch_scan<T, 16, 1>(p, s);
  return launch_scan<T, 32, 1>(p, s);
}

}  // namespace
}  // namespace sglb

extern "C" {

// Shapes in DeltaParams; T = bf16 or fp32 (`is_f32`) is the type of `proj`, `conv_w` and `conv_state`.
int sglb_delta_scan(const void* proj, long long ld, int g_off, int b_off, int a_off, const void* conv_w,
                    const float* a_log, const float* dt_bias, void* conv_state, float* state, const long long* slots,
                    const int* cu, const int* prefix, const int* track_len, const int* track_slot, float* qk, float* v,
                    float* gb, float* kq, float* o, int B, int T, int H, int Hk, int D, int V, int taps, int is_f32,
                    cudaStream_t s) {
  using namespace sglb;
  if (B <= 0 || T <= 0) return 0;
  if (D < 1 || D > 32 * kLanes || V < 1 || Hk < 1 || H % Hk != 0 || taps < 1 || H > 65535) return -kBadArgument;
  DeltaParams p{proj, ld, g_off, b_off, a_off, conv_w, a_log, dt_bias, conv_state, state, slots, cu, prefix, track_len,
                track_slot, qk, v, gb, kq, o, B, T, H, Hk, D, V, taps};
  return is_f32 ? run_delta<float>(p, s) : run_delta<__nv_bfloat16>(p, s);
}

// out [T, H * V] = rmsnorm(o [T, H, V], over V) * w [V] * silu(gate), gate at row stride `ld`.
int sglb_delta_gate(const float* o, const void* gate, long long ld, const float* w, void* out, long long T, int H, int V,
                    float eps, int is_f32, cudaStream_t s) {
  using namespace sglb;
  if (T <= 0) return 0;
  const long long blocks = (T * H + 3) / 4;
  if (is_f32)
    launch_pdl(delta_gate_kernel<float>, dim3(static_cast<unsigned>(blocks)), dim3(128), 0, s, o,
               static_cast<const float*>(gate), ld, w, static_cast<float*>(out), T, H, V, eps);
  else
    launch_pdl(delta_gate_kernel<__nv_bfloat16>, dim3(static_cast<unsigned>(blocks)), dim3(128), 0, s, o,
               static_cast<const __nv_bfloat16*>(gate), ld, w, static_cast<__nv_bfloat16*>(out), T, H, V, eps);
  return static_cast<int>(cudaGetLastError());
}

}  // extern "C"
