// Kernels of decoders that normalise before and after every sublayer around an fp32 residual stream:
//   embed_rmsnorm        token row -> stream (fp32), its RMS norm in the model's dtype
//   sandwich_rmsnorm     stream += rms(y) * w_post;  h = rms(stream) * w_pre        (one sublayer's end, the next one's start;
//                        y may be given as `k` rows per token in expert order, which are summed on the way in)
//   poly_norm            a N(z) + b N(z^2) + c N(z^3) + e over a feed-forward row, N = division by the root mean square
//   attn_prep_cache      split a fused projection: q and k heads normed and rotated (or as they are), q times a temperature that
//                        grows with the position, v as it is or of unit root mean square and mixed with another layer's
//                        values; K / V into the paged cache
// Weights come ready to multiply (a weight stored around zero arrives as 1 + w, a residual factor folded in).
// These kernels are launched with programmatic dependent launch: pointers carry no __restrict__, which would let the
// compiler read them through the non-coherent path before the producers have finished.  Statistics are fp32 (this file is
// compiled without fast-math).  `ld` is the row length of stream and copy: the width rounded up, padding columns zero.
#include "../api.h"
#include "../common/launch.cuh"
#include "../common/utils.cuh"

namespace b200 {
namespace {

constexpr int kThr = 256;

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

// 1 / root mean square of a row spread over the block (columns beyond H hold zeros)
template <int NV>
__device__ __forceinline__ float inv_rms(const float (&y)[NV][4], int H, float eps, float* red) {
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) s += y[i][j] * y[i][j];
  return 1.f / sqrtf(block_sum(s, red) / H + eps);
}

template <typename T, int NV>
__device__ __forceinline__ void store_normed(T* h, const float (&x)[NV][4], const float* w, float inv, int H, int ld) {
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * kThr + threadIdx.x) * 4;
    if (c >= ld) continue;
    float o[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) o[j] = c + j < H ? x[i][j] * inv * w[c + j] : 0.f;
    store4(h + c, o);
  }
}

template <typename T, int NV>
__global__ void __launch_bounds__(kThr) embed_rmsnorm_kernel(float* x, T* h, const int64_t* ids, const T* table,
                                                             const float* w, int H, int ld, int64_t rows, float eps) {
  __shared__ float red[32];
  griddep_launch();
  griddep_wait();
  const int64_t t = blockIdx.x, id = ids[t];
  const bool ok = id >= 0 && id < rows;
  float y[NV][4];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * kThr + threadIdx.x) * 4;
    y[i][0] = y[i][1] = y[i][2] = y[i][3] = 0.f;
    if (c >= ld) continue;
    if (ok) load4(y[i], table + id * ld + c);
    store4(x + t * ld + c, y[i]);
  }
  store_normed<T, NV>(h + t * ld, y, w, inv_rms<NV>(y, H, eps, red), H, ld);
}

template <typename T, int NV>
__global__ void __launch_bounds__(kThr) sandwich_rmsnorm_kernel(float* x, T* h, const T* y_, int64_t y_stride, const int* pos,
                                                                int k, const float* w_post, const float* w_pre, int H,
                                                                int ld, float eps) {
  __shared__ float red[32];
  griddep_launch();
  griddep_wait();
  const int64_t t = blockIdx.x;
  float y[NV][4], s[NV][4];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * kThr + threadIdx.x) * 4;
    y[i][0] = y[i][1] = y[i][2] = y[i][3] = s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
    if (c >= ld) continue;
    load4(s[i], x + t * ld + c);
    if (pos == nullptr) {
      load4(y[i], y_ + t * y_stride + c);
    } else {
      for (int q = 0; q < k; ++q) {
        const int r = pos[t * k + q];
        if (r < 0) continue;
        float z[4];
        load4(z, y_ + (int64_t)r * y_stride + c);
#pragma unroll
        for (int j = 0; j < 4; ++j) y[i][j] += z[j];
      }
    }
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (c + j >= H) y[i][j] = 0.f;
  }
  const float inv = inv_rms<NV>(y, H, eps, red);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * kThr + threadIdx.x) * 4;
    if (c >= ld) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (c + j < H) s[i][j] += y[i][j] * inv * w_post[c + j];
    store4(x + t * ld + c, s[i]);
  }
  store_normed<T, NV>(h + t * ld, s, w_pre, inv_rms<NV>(s, H, eps, red), H, ld);
}

// Three sums of a row at once, broadcast to the block.
template <int THR>
__device__ __forceinline__ void block_sum3(float& a, float& b, float& c, float (*red)[3]) {
  a = warp_sum(a);
  b = warp_sum(b);
  c = warp_sum(c);
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31;
  if (l == 0) { red[w][0] = a; red[w][1] = b; red[w][2] = c; }
  __syncthreads();
  const bool on = l < THR / 32;
  a = warp_sum(on ? red[l][0] : 0.f);
  b = warp_sum(on ? red[l][1] : 0.f);
  c = warp_sum(on ? red[l][2] : 0.f);
}

// NV 16-byte vectors per thread stay in registers as they were read; NV = 0: rows of any length, read twice.  Columns F .. ld
// of the output are zero.
template <typename T, int THR, int NV>
__global__ void __launch_bounds__(THR) poly_norm_kernel(T* out, int64_t ldo, const T* z, int64_t ldz, const float* coeff,
                                                        int F, int ld, float eps) {
  constexpr int V = Vec16<T>::N, NR = NV > 0 ? NV : 1;
  __shared__ float red[THR / 32][3];
  griddep_launch();
  griddep_wait();
  const int64_t t = blockIdx.x;
  const T* zr = z + t * ldz;
  Vec16<T> v[NR];
  float s1 = 0.f, s2 = 0.f, s3 = 0.f;
  auto add = [&](const Vec16<T>& a, int c) {
#pragma unroll
    for (int j = 0; j < V; ++j) {
      const float x = to_f(a.v[j]), q = c + j < F ? x * x : 0.f, q2 = q * q;
      s1 += q;
      s2 += q2;
      s3 = fmaf(q2, q, s3);
    }
  };
  if constexpr (NV > 0) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * THR + threadIdx.x) * V;
      if (c < ld) v[i] = ld_vec(zr + c);
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * THR + threadIdx.x) * V;
      if (c < ld) add(v[i], c);
    }
  } else {
    for (int c = threadIdx.x * V; c < ld; c += THR * V) add(ld_vec(zr + c), c);
  }
  block_sum3<THR>(s1, s2, s3, red);
  const float k1 = coeff[0] / sqrtf(s1 / F + eps), k2 = coeff[1] / sqrtf(s2 / F + eps), k3 = coeff[2] / sqrtf(s3 / F + eps),
              k0 = coeff[3];
  auto put = [&](Vec16<T> a, int c) {
#pragma unroll
    for (int j = 0; j < V; ++j) {
      const float x = to_f(a.v[j]);
      a.v[j] = from_f<T>(c + j < F ? fmaf(x, fmaf(x, fmaf(x, k3, k2), k1), k0) : 0.f);
    }
    st_vec(out + t * ldo + c, a);
  };
  if constexpr (NV > 0) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * THR + threadIdx.x) * V;
      if (c < ld) put(v[i], c);
    }
  } else {
    for (int c = threadIdx.x * V; c < ld; c += THR * V) put(ld_vec(zr + c), c);
  }
}

// One warp per (token, head) of q, k and v; head sizes D (q, k) and Dv (v) are zero-padded to Dc in q_out and in the cache
// [block][2][Hkv][slot][Dc].  See AttnPrepArgs for what happens to a head on the way.
template <typename T>
__global__ void __launch_bounds__(256) attn_prep_cache_kernel(AttnPrepArgs a, int vec) {
  griddep_launch();
  griddep_wait();
  const int64_t t = blockIdx.x;
  const int Hq = a.Hq, Hkv = a.Hkv, Dc = a.Dc;
  const int head = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (head >= Hq + 2 * Hkv) return;
  const bool is_q = head < Hq, is_v = head >= Hq + Hkv;
  const int n = is_v ? a.Dv : a.D;
  const int kvh = is_v ? head - Hq - Hkv : head - Hq;
  const T* src;
  T* dst = nullptr;
  float f = 1.f;
  if (is_q) {
    src = reinterpret_cast<const T*>(a.q) + t * a.stride + (int64_t)head * n;
    dst = reinterpret_cast<T*>(a.q_out) + (t * Hq + head) * (int64_t)Dc;
    if (a.temp_every > 0) f = 1.f + a.temp_coef * logf((float)((a.positions[t] + 1) / a.temp_every + 1));
  } else {
    src = reinterpret_cast<const T*>(is_v ? a.v : a.k) + t * a.stride + (int64_t)kvh * n;
    const int64_t slot = a.slots[t];
    if (slot >= 0 && slot < a.num_blocks * a.block_size) {      // fewer than 2^31 slots: 32-bit division
      const uint32_t block = (uint32_t)slot / (uint32_t)a.block_size, cell = (uint32_t)slot % (uint32_t)a.block_size;
      dst = reinterpret_cast<T*>(a.cache) +
            (((int64_t)block * 2 + (is_v ? 1 : 0)) * Hkv + kvh) * ((int64_t)a.block_size * Dc) + (int64_t)cell * Dc;
    }
  }
  const float* w = is_v ? nullptr : is_q ? a.q_norm : a.k_norm;
  // heads that fit one quad per lane stay in registers; their rotation partners come from another lane
  const bool held = vec && Dc <= 128;
  float own[4] = {0.f, 0.f, 0.f, 0.f};
  if (held && lane * 4 < n) load4(own, src + lane * 4);
  if (is_v ? a.v_norm != 0 : w != nullptr) {
    float ss = 0.f;
    if (held) {
      ss = own[0] * own[0] + own[1] * own[1] + own[2] * own[2] + own[3] * own[3];
    } else if (vec) {
      for (int i = lane * 4; i < n; i += 128) {
        float x[4];
        load4(x, src + i);
        ss += x[0] * x[0] + x[1] * x[1] + x[2] * x[2] + x[3] * x[3];
      }
    } else {
      for (int i = lane; i < n; i += 32) { const float x = to_f(src[i]); ss += x * x; }
    }
    f *= 1.f / sqrtf(warp_sum(ss) / n + a.eps);
  }
  const int pairs = is_v || a.table == nullptr ? 0 : a.pairs;   // column i < pairs turns with column i + pairs
  const float* turn = a.table == nullptr ? nullptr : a.table + t * a.pairs * 2;
  const int64_t vo = (t * Hkv + kvh) * (int64_t)a.Dv;
  const T* mix = is_v && a.v_in != nullptr ? reinterpret_cast<const T*>(a.v_in) + vo : nullptr;
  T* keep = is_v && a.v_out != nullptr ? reinterpret_cast<T*>(a.v_out) + vo : nullptr;
  if (held) {
    const int i = lane * 4, shift = pairs / 4;
    const bool lower = i < pairs;
    float x[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) x[j] = own[j] * (w == nullptr || i >= n ? f : f * w[i + j]);
    if (pairs > 0) {        // the same for the whole warp
#pragma unroll
      for (int j = 0; j < 4; ++j) own[j] = __shfl_sync(0xffffffffu, x[j], (lower ? lane + shift : lane - shift) & 31);
      if (i < 2 * pairs) {
        const float* cs = turn + 2 * (lower ? i : i - pairs);
        float c[4], s[4];
        load4(c, cs);
        load4(s, cs + 4);
        const float sg = lower ? -1.f : 1.f;
        x[0] = x[0] * c[0] + sg * own[0] * c[1];
        x[1] = x[1] * c[2] + sg * own[1] * c[3];
        x[2] = x[2] * s[0] + sg * own[2] * s[1];
        x[3] = x[3] * s[2] + sg * own[3] * s[3];
      }
    }
    if (i >= Dc) return;
    if (i < n) {
      if (keep != nullptr) store4(keep + i, x);
      if (mix != nullptr) {
        float b[4];
        load4(b, mix + i);
#pragma unroll
        for (int j = 0; j < 4; ++j) x[j] = (1.f - a.share) * x[j] + a.share * b[j];
      }
    }
    if (dst != nullptr) store4(dst + i, x);
  } else if (vec) {
    auto scaled = [&](float (&x)[4], int i) {
      load4(x, src + i);
#pragma unroll
      for (int j = 0; j < 4; ++j) x[j] *= w == nullptr ? f : f * w[i + j];
    };
    for (int i = lane * 4; i < Dc; i += 128) {
      float x[4] = {0.f, 0.f, 0.f, 0.f};
      if (i < n) {
        scaled(x, i);
        if (i < 2 * pairs) {
          const bool lower = i < pairs;
          float o[4];
          scaled(o, lower ? i + pairs : i - pairs);
          const float* cs = turn + 2 * (lower ? i : i - pairs);
#pragma unroll
          for (int j = 0; j < 4; ++j) x[j] = x[j] * cs[2 * j] + (lower ? -o[j] : o[j]) * cs[2 * j + 1];
        }
        if (keep != nullptr) store4(keep + i, x);
        if (mix != nullptr) {
          float b[4];
          load4(b, mix + i);
#pragma unroll
          for (int j = 0; j < 4; ++j) x[j] = (1.f - a.share) * x[j] + a.share * b[j];
        }
      }
      if (dst != nullptr) store4(dst + i, x);
    }
  } else {
    auto scaled = [&](int i) { return to_f(src[i]) * (w == nullptr ? f : f * w[i]); };
    for (int i = lane; i < Dc; i += 32) {
      float x = 0.f;
      if (i < n) {
        x = scaled(i);
        if (i < 2 * pairs) {
          const bool lower = i < pairs;
          const float o = scaled(lower ? i + pairs : i - pairs);
          const float* cs = turn + 2 * (lower ? i : i - pairs);
          x = x * cs[0] + (lower ? -o : o) * cs[1];
        }
        if (keep != nullptr) keep[i] = from_f<T>(x);
        if (mix != nullptr) x = (1.f - a.share) * x + a.share * to_f(mix[i]);
      }
      if (dst != nullptr) dst[i] = from_f<T>(x);
    }
  }
}

#define B200_SW_NV(NVEC, ...)                                                     \
  {                                                                               \
    const int need_ = (ld / 4 + kThr - 1) / kThr;                                 \
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

extern "C" int b200_embed_rmsnorm(float* x, void* h, const int64_t* ids, const void* table, const float* w, int64_t T_, int H,
                                  int ld, int64_t rows, float eps, int dtype, cudaStream_t st) {
  if (T_ == 0) return 0;
  if (ld % 4 || H > ld) return 3;
  B200_DISPATCH_DTYPE(dtype, B200_SW_NV(NV, launch_pdl(embed_rmsnorm_kernel<T, NV>, dim3(T_), dim3(kThr), 0, st, x, (T*)h, ids,
                                                      (const T*)table, w, H, ld, rows, eps)));
  return (int)cudaGetLastError();
}

extern "C" int b200_sandwich_rmsnorm(float* x, void* h, const void* y, int64_t y_stride, const int* pos, int k,
                                     const float* w_post, const float* w_pre, int64_t T_, int H, int ld, float eps, int dtype,
                                     cudaStream_t st) {
  if (T_ == 0) return 0;
  if (ld % 4 || H > ld || y_stride % 4) return 3;
  B200_DISPATCH_DTYPE(dtype, B200_SW_NV(NV, launch_pdl(sandwich_rmsnorm_kernel<T, NV>, dim3(T_), dim3(kThr), 0, st, x, (T*)h,
                                                      (const T*)y, y_stride, pos, k, w_post, w_pre, H, ld, eps)));
  return (int)cudaGetLastError();
}

extern "C" int b200_poly_norm(void* out, int64_t ldo, const void* z, int64_t ldz, const float* coeff, int64_t T_, int F, int ld,
                              float eps, int dtype, cudaStream_t st) {
  if (T_ == 0) return 0;
  if (F > ld || ((uintptr_t)out | (uintptr_t)z) % 16) return 3;
#define B200_PN(THR, NVEC)                                                                                          \
  launch_pdl(poly_norm_kernel<T, THR, NVEC>, dim3(T_), dim3(THR), 0, st, (T*)out, ldo, (const T*)z, ldz, coeff, F, ld, eps)
  B200_DISPATCH_DTYPE(dtype, {
    constexpr int V = Vec16<T>::N;
    if (ld % V || ldo % V || ldz % V) return 3;
    const int need = ld / V;
    if (need <= 256) B200_PN(256, 1);
    else if (need <= 512) B200_PN(256, 2);
    else if (need <= 1024) B200_PN(512, 2);
    else if (need <= 1536) B200_PN(512, 3);
    else if (need <= 2048) B200_PN(512, 4);
    else if (need <= 4096) B200_PN(1024, 4);
    else B200_PN(512, 0);
  });
#undef B200_PN
  return (int)cudaGetLastError();
}

extern "C" int b200_attn_prep_cache(const AttnPrepArgs* args, int64_t T_, int dtype, cudaStream_t st) {
  const AttnPrepArgs& a = *args;
  if (T_ == 0) return 0;
  if (a.D > a.Dc || a.Dv > a.Dc || (a.table != nullptr && 2 * a.pairs > a.D)) return 3;
  if (a.num_blocks * a.block_size >= ((int64_t)1 << 31)) return 3;
  const uintptr_t al = (uintptr_t)a.q | (uintptr_t)a.k | (uintptr_t)a.v | (uintptr_t)a.v_out | (uintptr_t)a.v_in;
  const int vec = a.D % 4 == 0 && a.Dv % 4 == 0 && a.Dc % 4 == 0 && a.stride % 4 == 0 && al % 16 == 0 &&
                  (a.table == nullptr || a.pairs % 4 == 0);
  dim3 grid((unsigned)T_, (a.Hq + 2 * a.Hkv + 7) / 8);
  B200_DISPATCH_DTYPE(dtype, launch_pdl(attn_prep_cache_kernel<T>, grid, dim3(256), 0, st, a, vec));
  return (int)cudaGetLastError();
}
