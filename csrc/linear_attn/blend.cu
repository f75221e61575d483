// Element-wise gated recurrence whose gates read only the current token (minGRU):
//   S_t = (1 - z) S_(t-1) + z c,   z = sigmoid(zr + bz),   c = u + 1/2 (u >= 0) or sigmoid(u) (u < 0),   u = ur + bu
//   out_t = S_t * silu(g)
// over raw projections zr, ur, g; the state [slots][W] is fp32 and carried per request.
// A token is the map S -> a S + b with a = 1 - z = sigmoid(-(zr + bz)), b = z c, and maps compose: a' a, a' b + b'.  One CTA takes
// 32 channels of one request, a lane each; its 16 warps take consecutive runs of tokens of a block and compose their run, one warp
// applies the runs' maps to the state in turn, and every warp walks its run from the state in front of it, while the next block's projections are on their way.  Products only: no
// logarithms, no quotients of gates, so gates near zero and one are safe.  Single tokens: a thread per channel.
// Launched with programmatic dependent launch: no __restrict__ on what a predecessor writes.  Compiled without fast-math.
#include "../api.h"
#include "../common/launch.cuh"
#include "../common/utils.cuh"

namespace b200 {
namespace {

constexpr int kWarps = 16, kRun = 8, kBlock = kWarps * kRun;   // tokens per warp and per block of tokens

// A token's map S -> a S + b and its output gate silu(g).  sigmoid(x) and sigmoid(-x) come from exp(-|x|) without cancellation.
// 16-bit models use the hardware exponential and one hardware reciprocal for the three denominators, which lie between one and two
// (a few units in the last place of fp32).
template <typename T>
__device__ __forceinline__ void token(float zr, float ur, float g, float bz, float bu, float& a, float& b, float& gate) {
  const float z = zr + bz, u = ur + bu;
  float ez, eu, eg, rz, ru, rg;
  if constexpr (sizeof(T) == 4) {
    ez = expf(-fabsf(z)); eu = expf(-fabsf(u)); eg = expf(-fabsf(g));
    rz = 1.f / (1.f + ez); ru = 1.f / (1.f + eu); rg = 1.f / (1.f + eg);
  } else {
    ez = __expf(-fabsf(z)); eu = __expf(-fabsf(u)); eg = __expf(-fabsf(g));
    const float dz = 1.f + ez, du = 1.f + eu, dg = 1.f + eg, zu = dz * du, r = __fdividef(1.f, zu * dg), t = r * dg;
    rz = t * du; ru = t * dz; rg = r * zu;
  }
  a = z >= 0.f ? ez * rz : rz;
  b = (z >= 0.f ? rz : ez * rz) * (u >= 0.f ? u + 0.5f : eu * ru);
  gate = g * (g >= 0.f ? rg : eg * rg);
}

template <typename T>
__global__ void __launch_bounds__(kWarps * 32, 2) blend_scan_kernel(BlendArgs p) {
  __shared__ float sa[2][kWarps][32], sb[2][kWarps][32], ss[2][kWarps][32];
  griddep_launch();
  griddep_wait();
  const int req = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int64_t q0 = p.qsl[req], q1 = p.qsl[req + 1];
  int64_t slot = p.slots[req];
  if (slot >= p.num_slots) slot = -1;
  if (q0 >= q1 || slot < 0) return;
  // lanes behind the last channel compute the last one again and store nothing
  const bool on = blockIdx.x * 32 + lane < p.width;
  const int c = min(blockIdx.x * 32 + lane, p.width - 1);
  const float bz = p.z_bias[c], bu = p.x_bias[c];
  float S = p.has_init[req] ? p.state[slot * p.width + c] : 0.f;     // warp 0: state in front of the block
  const int64_t first = q0 + warp * kRun;
  const T* z = reinterpret_cast<const T*>(p.z) + first * p.stride + c;
  const T* x = reinterpret_cast<const T*>(p.x) + first * p.stride + c;
  const T* g = reinterpret_cast<const T*>(p.g) + first * p.stride + c;
  T* out = reinterpret_cast<T*>(p.out) + first * p.out_stride + c;
  const uint32_t row = (uint32_t)p.stride, out_row = (uint32_t)p.out_stride;
  const int64_t block_step = (int64_t)kBlock * p.stride, out_step = (int64_t)kBlock * p.out_stride;
  T zr[kRun], ur[kRun], gr[kRun];
  auto fetch = [&](int n) {             // n rows of this warp's run, then the pointers move on to the next block
    if (n >= kRun) {
#pragma unroll
      for (int i = 0; i < kRun; ++i) { zr[i] = z[i * row]; ur[i] = x[i * row]; gr[i] = g[i * row]; }
    } else {
#pragma unroll
      for (int i = 0; i < kRun; ++i)
        if (i < n) { zr[i] = z[i * row]; ur[i] = x[i * row]; gr[i] = g[i * row]; }
    }
    z += block_step;
    x += block_step;
    g += block_step;
  };
  int left = (int)(q1 - first);         // rows from this warp's run on
  fetch(left);
  int buf = 0;
  for (int64_t base = q0; base < q1; base += kBlock, left -= kBlock, buf ^= 1) {
    float a[kRun], b[kRun], gate[kRun], A = 1.f, B = 0.f;
#pragma unroll
    for (int i = 0; i < kRun; ++i) {
      token<T>(to_f(zr[i]), to_f(ur[i]), to_f(gr[i]), bz, bu, a[i], b[i], gate[i]);
      if (i >= left) { a[i] = 1.f; b[i] = 0.f; }     // behind the request's end: nothing happens
      B = fmaf(a[i], B, b[i]);
      A *= a[i];
    }
    if (base + kBlock < q1) fetch(left - kBlock);
    sa[buf][warp][lane] = A;
    sb[buf][warp][lane] = B;
    __syncthreads();
    if (warp == 0) {      // states in front of every warp's run; buffers alternate, so two barriers per block suffice
#pragma unroll
      for (int w = 0; w < kWarps; ++w) {
        ss[buf][w][lane] = S;
        S = fmaf(sa[buf][w][lane], S, sb[buf][w][lane]);
      }
    }
    __syncthreads();
    float mine = ss[buf][warp][lane];
#pragma unroll
    for (int i = 0; i < kRun; ++i) {
      mine = fmaf(a[i], mine, b[i]);
      if (on && i < left) out[i * out_row] = from_f<T>(mine * gate[i]);
    }
    out += out_step;
  }
  if (warp == 0 && on) p.state[slot * p.width + c] = S;
}

// A thread per channel walks the request's tokens: requests of one token (or a few).
template <typename T>
__global__ void __launch_bounds__(128) blend_step_kernel(BlendArgs p) {
  griddep_launch();
  griddep_wait();
  const int req = blockIdx.y, c = blockIdx.x * 128 + threadIdx.x;
  const int64_t q0 = p.qsl[req], q1 = p.qsl[req + 1];
  int64_t slot = p.slots[req];
  if (slot >= p.num_slots) slot = -1;
  if (q0 >= q1 || c >= p.width) return;
  float S = slot >= 0 && p.has_init[req] ? p.state[slot * p.width + c] : 0.f;
  const float bz = p.z_bias[c], bu = p.x_bias[c];
  for (int64_t t = q0; t < q1; ++t) {
    float a, b, gate;
    const int64_t o = t * p.stride + c;
    token<T>(to_f(reinterpret_cast<const T*>(p.z)[o]), to_f(reinterpret_cast<const T*>(p.x)[o]),
             to_f(reinterpret_cast<const T*>(p.g)[o]), bz, bu, a, b, gate);
    S = fmaf(a, S, b);
    reinterpret_cast<T*>(p.out)[t * p.out_stride + c] = from_f<T>(S * gate);
  }
  if (slot >= 0) p.state[slot * p.width + c] = S;
}

}  // namespace
}  // namespace b200

extern "C" int b200_gated_blend(const BlendArgs* args, int dtype, cudaStream_t st) {
  using namespace b200;
  const BlendArgs& a = *args;
  if (a.R == 0 || a.width == 0) return 0;
  if (a.R > 65535 || a.stride >= (1 << 28) || a.out_stride >= (1 << 28)) return 3;
  B200_DISPATCH_DTYPE(dtype, {
    if (a.steps)
      launch_pdl(blend_step_kernel<T>, dim3((a.width + 127) / 128, a.R), dim3(128), 0, st, a);
    else
      launch_pdl(blend_scan_kernel<T>, dim3((a.width + 31) / 32, a.R), dim3(kWarps * 32), 0, st, a);
  });
  return (int)cudaGetLastError();
}
