// Linear recurrences with a [key channel x value channel] state per head, as sequential scans over a varlen batch
// (prefill portions and decode tokens alike), the state in registers and in fp32 throughout:
//
//   kChannelDelta   S <- diag(a_t) S;  u = beta_t (v_t - S^T k_t);  S <- S + k_t u^T;  o_t = S^T q_t
//                   a_t = exp(-exp(A_log_h) softplus(x_t + dt_bias)) per key channel, beta_t = sigmoid(b_t);
//                   q, k scaled to unit length per head (and q by `scale`)
//   kFixedDecay     S <- decay_h S + k_t v_t^T;  o_t = S^T q_t, with SiLU applied to q, k, v on the way in
//   kGatedWrite     S <- diag(f_t) S + (1 - f_t) v_t^T;  o_t = S^T q_t:  f_t = l + (1 - l) sigmoid(x_t + bias) per key
//                   channel with a lower bound l, SiLU applied to q
//
// Everything that enters the recurrence (gates, decays, unit norms) is computed here in fp32 from the raw projections.
// One block = 128 threads = 128 / TPR state rows (value channels) x TPR threads that share a row's key channels.
// Tokens are staged through shared memory a chunk at a time; the next chunk's raw values wait in registers.
#include "../api.h"
#include "../common/launch.cuh"
#include "../common/utils.cuh"

namespace b200 {
namespace {

constexpr int kThreads = 128;

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

enum RecurrenceKind : int { kChannelDelta = 0, kFixedDecay = 1, kGatedWrite = 2 };

// CH: tokens per staged chunk.  CH = 1 is the decode instance: few registers, so that enough state rows are in flight to
// stream the states at memory rate.
template <typename T, int DK, int TPR, int KIND, int CH>
__global__ void __launch_bounds__(kThreads, CH == 1 && DK <= 128 ? (KIND == kFixedDecay ? 6 : 4) : 1) linear_recurrence_kernel(const RecurrenceArgs p) {
  constexpr int RB = kThreads / TPR;                 // state rows of a block
  constexpr int QW = DK / TPR;                       // key channels of a thread
  constexpr int QK_PER = (CH * DK + kThreads - 1) / kThreads;
  constexpr int V_PER = (CH * RB + kThreads - 1) / kThreads;
  static_assert(QW % 4 == 0, "tile");
  constexpr bool kDelta = KIND == kChannelDelta, kGated = KIND == kGatedWrite;
  constexpr bool kHasA = kDelta || kGated;            // a per-channel projection beside q, k, v
  __shared__ __align__(16) float sk[CH][DK];
  __shared__ __align__(16) float sq[CH][DK];
  __shared__ __align__(16) float sg[kHasA ? CH : 1][kHasA ? DK : 4];
  __shared__ float sv[CH][RB];
  __shared__ float sb[CH], srk[CH], srq[CH];
  griddep_launch();
  griddep_wait();
  const int tid = threadIdx.x, rl = tid / TPR, qd = tid % TPR, warp = tid >> 5, lane = tid & 31;
  const int h = blockIdx.y, r = blockIdx.z, hk = h / (p.H / p.Hk);
  const int row0 = blockIdx.x * RB, row = row0 + rl;
  const int s = p.cu[r], L = p.cu[r + 1] - s, slot = p.slots[r];
  if (L <= 0 || slot < 0) return;
  const T* q = reinterpret_cast<const T*>(p.q) + hk * p.Dk;
  const T* k = reinterpret_cast<const T*>(p.k) + hk * p.Dk;
  const T* v = reinterpret_cast<const T*>(p.v) + h * p.Dv;
  const T* a = reinterpret_cast<const T*>(p.a) + (kHasA ? h * p.Dk : 0);
  const T* b = reinterpret_cast<const T*>(p.b) + (kDelta ? h : 0);
  const bool row_ok = row < p.Dv;
  // registers S[4i .. 4i+3] of lane qd hold key channels 4 (TPR i + qd) .. + 3: the TPR lanes of a row read
  // consecutive float4 of the staged vectors and of the state row
  float* sp = p.states + (((int64_t)slot * p.H + h) * p.Dv + row) * p.Dks + qd * 4;
  float S[QW];
#pragma unroll
  for (int j = 0; j < QW; j += 4) {
    float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
    if (p.has_init[r] && row_ok && j * TPR + qd * 4 < p.Dks) x = *reinterpret_cast<const float4*>(sp + j * TPR);
    S[j] = x.x; S[j + 1] = x.y; S[j + 2] = x.z; S[j + 3] = x.w;
  }
  const float rate = kDelta ? -expf(p.A_log[h]) : 0.f;
  const float decay = KIND == kFixedDecay ? p.decay[h] : 0.f;
  float rq_[QK_PER], rk_[QK_PER], ra_[kHasA ? QK_PER : 1], rv_[V_PER], rb = 0.f;
  auto fetch = [&](int c0) {
#pragma unroll
    for (int i = 0; i < QK_PER; ++i) {
      const int e = i * kThreads + tid, t = e / DK, d = e % DK;
      const bool ok = t < CH && c0 + t < L && d < p.Dk;
      const int64_t tok = s + c0 + t;
      if constexpr (!kGated) rk_[i] = ok ? to_f(k[tok * p.qkv_stride + d]) : 0.f;
      rq_[i] = ok ? to_f(q[tok * p.qkv_stride + d]) : 0.f;
      if constexpr (kHasA) ra_[i] = ok ? to_f(a[tok * p.a_stride + d]) : 0.f;
    }
#pragma unroll
    for (int i = 0; i < V_PER; ++i) {
      const int e = i * kThreads + tid, t = e / RB, d = e % RB;
      rv_[i] = (t < CH && c0 + t < L && row0 + d < p.Dv) ? to_f(v[(int64_t)(s + c0 + t) * p.qkv_stride + row0 + d]) : 0.f;
    }
    if (kDelta && tid < CH && c0 + tid < L) rb = to_f(b[(int64_t)(s + c0 + tid) * p.b_stride]);
  };
  fetch(0);
  for (int c0 = 0; c0 < L; c0 += CH) {
    const int n = min(CH, L - c0);
    __syncthreads();  // the previous chunk has been consumed
#pragma unroll
    for (int i = 0; i < QK_PER; ++i) {
      const int e = i * kThreads + tid, t = e / DK, d = e % DK;
      if (t < n) {
        if constexpr (kDelta) {
          sk[t][d] = rk_[i];
          sq[t][d] = rq_[i];
          sg[t][d] = d < p.Dk ? expf(rate * softplus_f(ra_[i] + p.dt_bias[h * p.Dk + d])) : 0.f;
        } else if constexpr (kGated) {
          float f = 0.f, w = 0.f;     // kept and written share; padding channels stay zero
          if (d < p.Dk) {
            const float z = ra_[i] + p.dt_bias[h * p.Dk + d], low = p.lower[h * p.Dk + d];
            const float e = expf(-fabsf(z)), big = 1.f / (1.f + e), small = e * big;   // sigmoid of |z| and of -|z|
            f = low + (1.f - low) * (z >= 0.f ? big : small);
            w = (1.f - low) * (z >= 0.f ? small : big);
          }
          sg[t][d] = f;
          sk[t][d] = w;
          sq[t][d] = silu_f(rq_[i]);
        } else {
          sk[t][d] = silu_f(rk_[i]);
          sq[t][d] = silu_f(rq_[i]);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < V_PER; ++i) {
      const int e = i * kThreads + tid, t = e / RB, d = e % RB;
      if (t < n) sv[t][d] = KIND == kFixedDecay ? silu_f(rv_[i]) : rv_[i];
    }
    if (kDelta && tid < n) sb[tid] = sigmoid_f(rb);
    __syncthreads();
    if constexpr (kDelta) {
      for (int t = warp; t < n; t += kThreads / 32) {
        float k2 = 0.f, q2 = 0.f;
        for (int d = lane; d < DK; d += 32) { k2 += sk[t][d] * sk[t][d]; q2 += sq[t][d] * sq[t][d]; }
        k2 = warp_sum(k2);
        q2 = warp_sum(q2);
        if (lane == 0) {
          srk[t] = 1.f / sqrtf(k2 + p.unit_eps);
          srq[t] = p.scale / sqrtf(q2 + p.unit_eps);
        }
      }
    }
    if (c0 + CH < L) fetch(c0 + CH);  // the next chunk's loads fly while this one is processed
    if constexpr (kDelta) __syncthreads();
    for (int t = 0; t < n; ++t) {
      const float* kk = &sk[t][qd * 4];
      const float* qq = &sq[t][qd * 4];
      const float vt = sv[t][rl];
      float o = 0.f, o2 = 0.f;
      if constexpr (kDelta) {
        const float* gg = &sg[t][qd * 4];
        const float rk = srk[t], bt = sb[t];
        float pred = 0.f, pred2 = 0.f;
#pragma unroll
        for (int j = 0; j < QW; j += 4) {
          const float4 k4 = *reinterpret_cast<const float4*>(kk + j * TPR);
          const float4 g4 = *reinterpret_cast<const float4*>(gg + j * TPR);
          S[j] *= g4.x; S[j + 1] *= g4.y; S[j + 2] *= g4.z; S[j + 3] *= g4.w;
          pred += S[j] * k4.x + S[j + 1] * k4.y;
          pred2 += S[j + 2] * k4.z + S[j + 3] * k4.w;
        }
        pred += pred2;
#pragma unroll
        for (int m = 1; m < TPR; m <<= 1) pred += __shfl_xor_sync(0xffffffff, pred, m);
        const float u = (vt - pred * rk) * bt * rk;
#pragma unroll
        for (int j = 0; j < QW; j += 4) {
          const float4 k4 = *reinterpret_cast<const float4*>(kk + j * TPR);
          const float4 q4 = *reinterpret_cast<const float4*>(qq + j * TPR);
          S[j] += u * k4.x; S[j + 1] += u * k4.y; S[j + 2] += u * k4.z; S[j + 3] += u * k4.w;
          o += S[j] * q4.x + S[j + 1] * q4.y;
          o2 += S[j + 2] * q4.z + S[j + 3] * q4.w;
        }
      } else if constexpr (kGated) {
        const float* gg = &sg[t][qd * 4];
#pragma unroll
        for (int j = 0; j < QW; j += 4) {
          const float4 k4 = *reinterpret_cast<const float4*>(kk + j * TPR);
          const float4 q4 = *reinterpret_cast<const float4*>(qq + j * TPR);
          const float4 g4 = *reinterpret_cast<const float4*>(gg + j * TPR);
          S[j] = S[j] * g4.x + vt * k4.x; S[j + 1] = S[j + 1] * g4.y + vt * k4.y;
          S[j + 2] = S[j + 2] * g4.z + vt * k4.z; S[j + 3] = S[j + 3] * g4.w + vt * k4.w;
          o += S[j] * q4.x + S[j + 1] * q4.y;
          o2 += S[j + 2] * q4.z + S[j + 3] * q4.w;
        }
      } else {
#pragma unroll
        for (int j = 0; j < QW; j += 4) {
          const float4 k4 = *reinterpret_cast<const float4*>(kk + j * TPR);
          const float4 q4 = *reinterpret_cast<const float4*>(qq + j * TPR);
          S[j] = S[j] * decay + vt * k4.x; S[j + 1] = S[j + 1] * decay + vt * k4.y;
          S[j + 2] = S[j + 2] * decay + vt * k4.z; S[j + 3] = S[j + 3] * decay + vt * k4.w;
          o += S[j] * q4.x + S[j + 1] * q4.y;
          o2 += S[j + 2] * q4.z + S[j + 3] * q4.w;
        }
      }
      o += o2;
#pragma unroll
      for (int m = 1; m < TPR; m <<= 1) o += __shfl_xor_sync(0xffffffff, o, m);
      if (qd == 0 && row_ok) p.out[(int64_t)(s + c0 + t) * p.out_stride + h * p.Dv + row] = kDelta ? o * srq[t] : o;
    }
  }
#pragma unroll
  for (int j = 0; j < QW; j += 4)
    if (row_ok && j * TPR + qd * 4 < p.Dks)
      *reinterpret_cast<float4*>(sp + j * TPR) = make_float4(S[j], S[j + 1], S[j + 2], S[j + 3]);
}

template <typename T, int DK, int TPR, int CH>
void launch_ch(const RecurrenceArgs& a, dim3 grid, cudaStream_t st) {
  if (a.kind == kChannelDelta)
    launch_pdl(linear_recurrence_kernel<T, DK, TPR, kChannelDelta, CH>, grid, dim3(kThreads), 0, st, a);
  else if (a.kind == kGatedWrite)
    launch_pdl(linear_recurrence_kernel<T, DK, TPR, kGatedWrite, CH>, grid, dim3(kThreads), 0, st, a);
  else
    launch_pdl(linear_recurrence_kernel<T, DK, TPR, kFixedDecay, CH>, grid, dim3(kThreads), 0, st, a);
}

template <typename T, int DK, int TPR>
int launch(const RecurrenceArgs& a, cudaStream_t st) {
  constexpr int RB = kThreads / TPR;
  dim3 grid((a.Dv + RB - 1) / RB, a.H, a.R);
  if (a.decode) launch_ch<T, DK, TPR, 1>(a, grid, st);
  else launch_ch<T, DK, TPR, DK <= 128 ? 16 : (DK <= 256 ? 8 : 4)>(a, grid, st);
  return (int)cudaGetLastError();
}

template <typename T>
int dispatch(const RecurrenceArgs& a, cudaStream_t st) {
  if (a.Dk <= 16) return launch<T, 16, 4>(a, st);
  if (a.Dk <= 32) return launch<T, 32, 4>(a, st);
  if (a.Dk <= 64) return launch<T, 64, 4>(a, st);
  if (a.Dk <= 96) return launch<T, 96, 4>(a, st);
  if (a.Dk <= 128) return launch<T, 128, 4>(a, st);
  if (a.Dk <= 256) return launch<T, 256, 8>(a, st);
  if (a.Dk <= 512) return launch<T, 512, 16>(a, st);
  return 3;
}

}  // namespace
}  // namespace b200

extern "C" int b200_linear_recurrence(const RecurrenceArgs* a, int dtype, cudaStream_t st) {
  if (a->R == 0) return 0;
  if (a->H % a->Hk || a->Dks % 4 || a->Dks < a->Dk || a->R > 65535 || a->H > 65535) return 3;
  switch (dtype) {
    case b200::kF32: return b200::dispatch<float>(*a, st);
    case b200::kBF16: return b200::dispatch<__nv_bfloat16>(*a, st);
    case b200::kF16: return b200::dispatch<__half>(*a, st);
  }
  return 1;
}
