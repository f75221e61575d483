// Kernels of decoders whose residual stream is kept in fp32 and normalised on the sublayers' outputs:
//   embed_layernorm        token row + sinusoidal position vector -> LayerNorm -> stream (fp32) + 16-bit copy
//   layernorm_residual     stream += LayerNorm(s1 y1 [+ s2 y2]) (or the final norm of the stream) + 16-bit copy
//   gated_group_rmsnorm    RMS norm over groups of a mixer's output, times weight and (with a gate) sigmoid(gate)
//   qk_unit_norm_cache     split a fused projection, scale q / k to unit RMS per head, K / V into the paged cache
// These kernels are launched with programmatic dependent launch, so they may be resident while the producer of their
// inputs still runs: the pointers carry no __restrict__, which would let the compiler read them through the
// non-coherent path.
// All statistics in fp32 (this file is compiled without fast-math).  `ld` is the row length of stream and copy: the
// width rounded up so that rows stay 16-byte aligned; the padding columns are kept at zero.
#include "../api.h"
#include "../common/launch.cuh"
#include "../common/utils.cuh"

namespace b200 {
namespace {

constexpr int kLnThreads = 256;

template <typename T> struct alignas(4 * sizeof(T)) Vec4 { T v[4]; };
template <typename T> __device__ __forceinline__ void load4(float (&d)[4], const T* p) {
  const Vec4<T> r = *reinterpret_cast<const Vec4<T>*>(p);
#pragma unroll
  for (int j = 0; j < 4; ++j) d[j] = to_f(r.v[j]);
}
template <typename T> __device__ __forceinline__ void store4(T* p, const float (&s)[4]) {
  Vec4<T> r;
#pragma unroll
  for (int j = 0; j < 4; ++j) r.v[j] = from_f<T>(s[j]);
  *reinterpret_cast<Vec4<T>*>(p) = r;
}

// Normalise NV x 4 values per thread (columns 4 (i kLnThreads + tid) ..), zero beyond H.
template <int NV>
__device__ __forceinline__ void layer_norm_regs(float (&y)[NV][4], int H, float eps, const float* w, float* red) {
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) s += y[i][j];  // columns beyond H hold zeros
  const float mean = block_sum(s, red) / H;
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int c = (i * kLnThreads + threadIdx.x) * 4 + j;
      const float d = c < H ? y[i][j] - mean : 0.f;
      y[i][j] = d;
      ss += d * d;
    }
  const float inv = 1.f / sqrtf(block_sum(ss, red) / H + eps);
#pragma unroll
  for (int i = 0; i < NV; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int c = (i * kLnThreads + threadIdx.x) * 4 + j;
      y[i][j] = c < H ? y[i][j] * inv * w[c] : 0.f;
    }
}

// freq[i]: turns (angle / 2 pi) per position of column pair i as a 64-bit fixed-point fraction.  The product with the
// position wraps modulo one turn by itself, so the angle keeps fp32 accuracy at any position.
template <typename T, int NV>
__global__ void __launch_bounds__(kLnThreads) embed_layernorm_kernel(float* x, T* h,
                                                                    const int64_t* ids,
                                                                    const int64_t* positions,
                                                                    const T* table,
                                                                    const int64_t* freq,
                                                                    const float* w, int H, int ld,
                                                                    int64_t rows, float eps) {
  __shared__ float red[32];
  griddep_launch();
  griddep_wait();
  const int64_t t = blockIdx.x, id = ids[t];
  const bool ok = id >= 0 && id < rows;
  const uint64_t pos = (uint64_t)positions[t];
  float y[NV][4];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * kLnThreads + threadIdx.x) * 4;
    y[i][0] = y[i][1] = y[i][2] = y[i][3] = 0.f;
    if (c >= ld) continue;
    if (ok) load4(y[i], table + id * ld + c);
#pragma unroll
    for (int j = 0; j < 4; j += 2) {
      if (c + j >= H) continue;
      const int64_t turns = (int64_t)(pos * (uint64_t)freq[(c + j) >> 1]);  // [-1/2, 1/2) of a turn in units of 2^-64
      float sn, cs;
      sincospif((float)turns * 0x1p-63f, &sn, &cs);
      y[i][j] += sn;
      if (c + j + 1 < H) y[i][j + 1] += cs;
    }
  }
  layer_norm_regs<NV>(y, H, eps, w, red);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * kLnThreads + threadIdx.x) * 4;
    if (c >= ld) continue;
    store4(x + t * ld + c, y[i]);
    if ((void*)h != (void*)x) store4(h + t * ld + c, y[i]);
  }
}

template <typename T, int NV>
__global__ void __launch_bounds__(kLnThreads) layernorm_residual_kernel(float* x, T* h,
                                                                       const T* y1, int64_t y1_stride, float s1,
                                                                       const T* y2, int64_t y2_stride, float s2,
                                                                       const float* w, int H, int ld, float eps,
                                                                       int add) {
  __shared__ float red[32];
  griddep_launch();
  griddep_wait();
  const int64_t t = blockIdx.x;
  float* xr = x + t * ld;
  float y[NV][4], res[NV][4];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * kLnThreads + threadIdx.x) * 4;
    y[i][0] = y[i][1] = y[i][2] = y[i][3] = 0.f;
    if (c >= ld) continue;
    if (add) {
      load4(res[i], xr + c);
      load4(y[i], y1 + t * y1_stride + c);
      if (y2 != nullptr) {
        float z[4];
        load4(z, y2 + t * y2_stride + c);
#pragma unroll
        for (int j = 0; j < 4; ++j) y[i][j] = s1 * y[i][j] + s2 * z[j];
      } else {
#pragma unroll
        for (int j = 0; j < 4; ++j) y[i][j] *= s1;
      }
    } else {
      load4(y[i], xr + c);
    }
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (c + j >= H) y[i][j] = 0.f;
  }
  layer_norm_regs<NV>(y, H, eps, w, red);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * kLnThreads + threadIdx.x) * 4;
    if (c >= ld) continue;
    if (add) {
#pragma unroll
      for (int j = 0; j < 4; ++j) y[i][j] += res[i][j];
      store4(xr + c, y[i]);
    }
    if ((void*)h != (void*)x) store4(h + t * ld + c, y[i]);
  }
}

// out = o / sqrt(mean(o^2) + eps) * w [* sigmoid(gate)] over groups of D columns; RT threads per group.
template <typename T, int RT, bool VEC>
__global__ void __launch_bounds__(256) gated_group_rmsnorm_kernel(T* out, int64_t out_stride,
                                                                  const float* o, int64_t o_stride,
                                                                  const T* gate, int64_t gate_stride,
                                                                  const float* w, int64_t rows, int groups,
                                                                  int D, float eps) {
  constexpr int V = VEC ? 4 : 1;
  __shared__ float red[32];
  griddep_launch();
  griddep_wait();
  const int64_t row = (int64_t)blockIdx.x * (256 / RT) + threadIdx.x / RT;
  if (RT == 32 && row >= rows) return;
  const int lane = threadIdx.x % RT;
  const int64_t t = row / groups;
  const int g = (int)(row % groups);
  const float* orow = o + t * o_stride + (int64_t)g * D;
  const T* grow = gate == nullptr ? nullptr : gate + t * gate_stride + (int64_t)g * D;
  T* dst = out + t * out_stride + (int64_t)g * D;
  float ss = 0.f;
  for (int i = lane * V; i < D; i += RT * V) {
    if constexpr (VEC) {
      float a[4];
      load4(a, orow + i);
      ss += a[0] * a[0] + a[1] * a[1] + a[2] * a[2] + a[3] * a[3];
    } else {
      ss += orow[i] * orow[i];
    }
  }
  ss = RT == 32 ? warp_sum(ss) : block_sum(ss, red);
  const float inv = 1.f / sqrtf(ss / D + eps);
  for (int i = lane * V; i < D; i += RT * V) {
    if constexpr (VEC) {
      float a[4], b[4], ww[4];
      load4(a, orow + i);
      if (grow != nullptr) load4(b, grow + i);
      load4(ww, w + i);
#pragma unroll
      for (int j = 0; j < 4; ++j) a[j] = a[j] * inv * ww[j] * (grow != nullptr ? 1.f / (1.f + expf(-b[j])) : 1.f);
      store4(dst + i, a);
    } else {
      dst[i] = from_f<T>(orow[i] * inv * w[i] * (grow != nullptr ? 1.f / (1.f + expf(-to_f(grow[i]))) : 1.f));
    }
  }
}

// One warp per (token, head) of q, k and v.  Head sizes D (q, k) and Dv (v) are zero-padded to Dc in q_out and in the
// cache [block][2][Hkv][slot][Dc].
template <typename T>
__global__ void __launch_bounds__(256) qk_unit_norm_cache_kernel(T* q_out, const T* q,
                                                                 const T* k, const T* v,
                                                                 int64_t stride, T* cache,
                                                                 const int64_t* slots, int Hq, int Hkv, int D,
                                                                 int Dv, int Dc, int block_size, int64_t num_blocks,
                                                                 float eps, int vec) {
  griddep_launch();
  griddep_wait();
  const int64_t t = blockIdx.x;
  const int head = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (head >= Hq + 2 * Hkv) return;
  const bool is_q = head < Hq, is_v = head >= Hq + Hkv;
  const int n = is_v ? Dv : D;
  const T* src;
  T* dst;
  if (is_q) {
    src = q + t * stride + (int64_t)head * D;
    dst = q_out + (t * Hq + head) * (int64_t)Dc;
  } else {
    const int64_t slot = slots[t];
    if (slot < 0 || slot >= num_blocks * block_size) return;
    const int kvh = is_v ? head - Hq - Hkv : head - Hq;
    src = (is_v ? v : k) + t * stride + (int64_t)kvh * n;
    dst = cache + ((((slot / block_size) * 2 + (is_v ? 1 : 0)) * Hkv + kvh) * block_size + slot % block_size) * (int64_t)Dc;
  }
  float inv = 1.f;
  if (!is_v) {
    float ss = 0.f;
    if (vec) {
      for (int i = lane * 4; i < n; i += 128) {
        float a[4];
        load4(a, src + i);
        ss += a[0] * a[0] + a[1] * a[1] + a[2] * a[2] + a[3] * a[3];
      }
    } else {
      for (int i = lane; i < n; i += 32) { const float f = to_f(src[i]); ss += f * f; }
    }
    inv = 1.f / sqrtf(warp_sum(ss) / n + eps);
  }
  if (vec) {
    for (int i = lane * 4; i < Dc; i += 128) {
      float a[4] = {0.f, 0.f, 0.f, 0.f};
      if (i < n) load4(a, src + i);
#pragma unroll
      for (int j = 0; j < 4; ++j) a[j] *= inv;
      store4(dst + i, a);
    }
  } else {
    for (int i = lane; i < Dc; i += 32) dst[i] = from_f<T>(i < n ? to_f(src[i]) * inv : 0.f);
  }
}

#define B200_LN_NV(NVEC, ...)                                                     \
  {                                                                               \
    const int need_ = (ld / 4 + kLnThreads - 1) / kLnThreads;                     \
    if (need_ <= 1) { constexpr int NVEC = 1; __VA_ARGS__; }                      \
    else if (need_ <= 2) { constexpr int NVEC = 2; __VA_ARGS__; }                 \
    else if (need_ <= 4) { constexpr int NVEC = 4; __VA_ARGS__; }                 \
    else if (need_ <= 8) { constexpr int NVEC = 8; __VA_ARGS__; }                 \
    else if (need_ <= 16) { constexpr int NVEC = 16; __VA_ARGS__; }               \
    else return 3;                                                                \
  }

}  // namespace
}  // namespace b200

using namespace b200;

extern "C" int b200_embed_layernorm(float* x, void* h, const int64_t* ids, const int64_t* positions, const void* table,
                                    const int64_t* freq, const float* w, int64_t T_, int H, int ld, int64_t rows, float eps,
                                    int dtype, cudaStream_t st) {
  if (T_ == 0) return 0;
  if (ld % 4 || H > ld) return 3;
  B200_DISPATCH_DTYPE(dtype, B200_LN_NV(NV, launch_pdl(embed_layernorm_kernel<T, NV>, dim3(T_), dim3(kLnThreads), 0, st, x,
                                                      (T*)h, ids, positions, (const T*)table, freq, w, H, ld, rows, eps)));
  return (int)cudaGetLastError();
}

extern "C" int b200_layernorm_residual(float* x, void* h, const void* y1, int64_t y1_stride, float s1, const void* y2,
                                       int64_t y2_stride, float s2, const float* w, int64_t T_, int H, int ld, float eps,
                                       int add, int dtype, cudaStream_t st) {
  if (T_ == 0) return 0;
  if (ld % 4 || H > ld || (add && y1_stride % 4) || (y2 && y2_stride % 4)) return 3;
  B200_DISPATCH_DTYPE(dtype, B200_LN_NV(NV, launch_pdl(layernorm_residual_kernel<T, NV>, dim3(T_), dim3(kLnThreads), 0, st,
                                                      x, (T*)h, (const T*)y1, y1_stride, s1, (const T*)y2, y2_stride, s2, w,
                                                      H, ld, eps, add)));
  return (int)cudaGetLastError();
}

extern "C" int b200_gated_group_rmsnorm(void* out, int64_t out_stride, const float* o, int64_t o_stride, const void* gate,
                                        int64_t gate_stride, const float* w, int64_t T_, int groups, int D, float eps,
                                        int dtype, cudaStream_t st) {
  const int64_t rows = T_ * groups;
  if (rows == 0) return 0;
  const bool vec = D % 4 == 0 && out_stride % 4 == 0 && o_stride % 4 == 0 && gate_stride % 4 == 0 &&
                   (uintptr_t)gate % 16 == 0 && (uintptr_t)out % 16 == 0 && (uintptr_t)o % 16 == 0;
#define B200_GGN(RT, VEC)                                                                                              \
  launch_pdl(gated_group_rmsnorm_kernel<T, RT, VEC>, dim3((rows + 256 / RT - 1) / (256 / RT)), dim3(256), 0, st, (T*)out, \
             out_stride, o, o_stride, (const T*)gate, gate_stride, w, rows, groups, D, eps)
  B200_DISPATCH_DTYPE(dtype, {
    if (D <= 512) {
      if (vec) B200_GGN(32, true); else B200_GGN(32, false);
    } else {
      if (vec) B200_GGN(256, true); else B200_GGN(256, false);
    }
  });
#undef B200_GGN
  return (int)cudaGetLastError();
}

extern "C" int b200_qk_unit_norm_cache(void* q_out, const void* q, const void* k, const void* v, int64_t stride,
                                       void* kv_cache, const int64_t* slots, int64_t T_, int Hq, int Hkv, int D, int Dv,
                                       int Dc, int block_size, int64_t num_blocks, float eps, int dtype, cudaStream_t st) {
  if (T_ == 0) return 0;
  if (D > Dc || Dv > Dc) return 3;
  const uintptr_t al = (uintptr_t)q | (uintptr_t)k | (uintptr_t)v;
  const int vec = D % 4 == 0 && Dv % 4 == 0 && Dc % 4 == 0 && stride % 4 == 0 && al % 16 == 0;
  dim3 grid((unsigned)T_, (Hq + 2 * Hkv + 7) / 8);
  B200_DISPATCH_DTYPE(dtype, launch_pdl(qk_unit_norm_cache_kernel<T>, grid, dim3(256), 0, st, (T*)q_out, (const T*)q,
                                       (const T*)k, (const T*)v, stride, (T*)kv_cache, slots, Hq, Hkv, D, Dv, Dc, block_size,
                                       num_blocks, eps, vec));
  return (int)cudaGetLastError();
}
