// Element-wise gated recurrence whose gates read only the current token (minGRU):
//   S_t = (1 - z) S_(t-1) + z c,   z = sigmoid(zr + bz),   c = u + 1/2 (u >= 0) or sigmoid(u) (u < 0),   u = ur + bu
//   out_t = S_t * silu(g)
// over raw projections zr, ur, g; the state [slots][W] is fp32 and carried per request.
// A token is the map S -> a S + b with a = 1 - z = sigmoid(-(zr + bz)), b = z c, and maps compose: a' a, a' b + b'.  One CTA takes
// 32 columns (two channels each) of one request; its 16 warps take consecutive runs of tokens of a block, compose their run,
// meet over shared memory and apply the map of everything in front.  Products only: no logarithms, no quotients, so gates near
// zero and one are safe.  Single tokens: a thread per channel.
// Launched with programmatic dependent launch: no __restrict__ on what a predecessor writes.  Compiled without fast-math.
#include "../api.h"
#include "../common/launch.cuh"
#include "../common/utils.cuh"

namespace b200 {
namespace {

constexpr int kWarps = 16, kRun = 8, kBlock = kWarps * kRun;   // tokens per warp and per block of tokens

template <typename T> struct alignas(2 * sizeof(T)) Pair { T v[2]; };
template <typename T> __device__ __forceinline__ float2 load2(const T* p) {
  const Pair<T> r = *reinterpret_cast<const Pair<T>*>(p);
  return make_float2(to_f(r.v[0]), to_f(r.v[1]));
}
template <typename T> __device__ __forceinline__ void store2(T* p, float a, float b) {
  Pair<T> r;
  r.v[0] = from_f<T>(a);
  r.v[1] = from_f<T>(b);
  *reinterpret_cast<Pair<T>*>(p) = r;
}
// sigmoid(-x) and sigmoid(x), both without cancellation
__device__ __forceinline__ void sigmoids(float x, float& neg, float& pos) {
  const float e = expf(-fabsf(x)), r = 1.f / (1.f + e);
  pos = x >= 0.f ? r : e * r;
  neg = x >= 0.f ? e * r : r;
}
__device__ __forceinline__ void token_map(float zr, float ur, float bz, float bu, float& a, float& b) {
  float z, n;
  sigmoids(zr + bz, a, z);
  const float u = ur + bu;
  float c = u + 0.5f;
  if (u < 0.f) sigmoids(u, n, c);
  b = z * c;
}
__device__ __forceinline__ float silu(float g) {
  float n, p;
  sigmoids(g, n, p);
  return g * p;
}

template <typename T>
__global__ void __launch_bounds__(kWarps * 32) blend_scan_kernel(BlendArgs p) {
  __shared__ float2 sa[kWarps][32], sb[kWarps][32];
  griddep_launch();
  griddep_wait();
  const int req = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int64_t q0 = p.qsl[req], q1 = p.qsl[req + 1];
  int64_t slot = p.slots[req];
  if (slot >= p.num_slots) slot = -1;
  if (q0 >= q1 || slot < 0) return;
  const int c = (blockIdx.x * 32 + lane) * 2;
  const bool on = c < p.width, both = c + 1 < p.width;    // the projections' columns are padded to an even number
  float2 bz = make_float2(0.f, 0.f), bu = bz, S = bz;
  if (on) {
    bz.x = p.z_bias[c]; bu.x = p.x_bias[c];
    if (both) { bz.y = p.z_bias[c + 1]; bu.y = p.x_bias[c + 1]; }
    if (p.has_init[req]) {
      S.x = p.state[slot * p.width + c];
      if (both) S.y = p.state[slot * p.width + c + 1];
    }
  }
  const T* z = reinterpret_cast<const T*>(p.z) + c;
  const T* x = reinterpret_cast<const T*>(p.x) + c;
  const T* g = reinterpret_cast<const T*>(p.g) + c;
  T* out = reinterpret_cast<T*>(p.out) + c;
  for (int64_t base = q0; base < q1; base += kBlock) {
    const int64_t t0 = base + warp * kRun;
    const int n = on ? (int)max((int64_t)0, min((int64_t)kRun, q1 - t0)) : 0;
    float2 a[kRun], b[kRun];
    float2 zr[kRun], ur[kRun];
#pragma unroll
    for (int i = 0; i < kRun; ++i)
      if (i < n) { zr[i] = load2(z + (t0 + i) * p.stride); ur[i] = load2(x + (t0 + i) * p.stride); }
    float2 A = make_float2(1.f, 1.f), B = make_float2(0.f, 0.f);
#pragma unroll
    for (int i = 0; i < kRun; ++i) {
      if (i >= n) break;
      token_map(zr[i].x, ur[i].x, bz.x, bu.x, a[i].x, b[i].x);
      token_map(zr[i].y, ur[i].y, bz.y, bu.y, a[i].y, b[i].y);
      B.x = fmaf(a[i].x, B.x, b[i].x); B.y = fmaf(a[i].y, B.y, b[i].y);
      A.x *= a[i].x; A.y *= a[i].y;
    }
    sa[warp][lane] = A;
    sb[warp][lane] = B;
    __syncthreads();
    // state in front of this warp's run, and behind the block
    float2 mine = S;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) {
      if (w == warp) mine = S;
      const float2 wa = sa[w][lane], wb = sb[w][lane];
      S.x = fmaf(wa.x, S.x, wb.x); S.y = fmaf(wa.y, S.y, wb.y);
    }
    __syncthreads();      // the maps are overwritten by the next block
#pragma unroll
    for (int i = 0; i < kRun; ++i)
      if (i < n) zr[i] = load2(g + (t0 + i) * p.stride);
#pragma unroll
    for (int i = 0; i < kRun; ++i) {
      if (i >= n) break;
      mine.x = fmaf(a[i].x, mine.x, b[i].x); mine.y = fmaf(a[i].y, mine.y, b[i].y);
      store2(out + (t0 + i) * p.out_stride, mine.x * silu(zr[i].x), both ? mine.y * silu(zr[i].y) : 0.f);
    }
  }
  if (warp == 0 && on) {
    p.state[slot * p.width + c] = S.x;
    if (both) p.state[slot * p.width + c + 1] = S.y;
  }
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
    float a, b;
    token_map(to_f(reinterpret_cast<const T*>(p.z)[t * p.stride + c]), to_f(reinterpret_cast<const T*>(p.x)[t * p.stride + c]), bz,
              bu, a, b);
    S = fmaf(a, S, b);
    reinterpret_cast<T*>(p.out)[t * p.out_stride + c] =
        from_f<T>(S * silu(to_f(reinterpret_cast<const T*>(p.g)[t * p.stride + c])));
  }
  if (slot >= 0) p.state[slot * p.width + c] = S;
}

}  // namespace
}  // namespace b200

extern "C" int b200_gated_blend(const BlendArgs* args, int dtype, cudaStream_t st) {
  using namespace b200;
  const BlendArgs& a = *args;
  if (a.R == 0 || a.width == 0) return 0;
  if (a.R > 65535) return 3;
  const uintptr_t al = (uintptr_t)a.z | (uintptr_t)a.x | (uintptr_t)a.g | (uintptr_t)a.out;
  if (!a.steps && (al % 8 || a.stride % 2 || a.out_stride % 2 || a.out_stride < (a.width + 1) / 2 * 2)) return 3;
  B200_DISPATCH_DTYPE(dtype, {
    if (a.steps)
      launch_pdl(blend_step_kernel<T>, dim3((a.width + 127) / 128, a.R), dim3(128), 0, st, a);
    else
      launch_pdl(blend_scan_kernel<T>, dim3((a.width + 63) / 64, a.R), dim3(kWarps * 32), 0, st, a);
  });
  return (int)cudaGetLastError();
}
