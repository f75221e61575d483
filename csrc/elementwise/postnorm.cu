// Kernels of decoders whose sublayers read a short causal convolution of an fp32 residual stream and are normalised on their
// output:
//   postnorm      x += LayerNorm(y) * w (or x = scaled token row), y being a row, or the weighted sum of a token's expert rows;
//                 then, for requests of a few tokens, the next sublayer's input x + conv(x), or the model's last norm
//   input_conv    x + conv(x) alone, for prompt portions
// conv(x)_t = sum_j c_j x_(t - n + 1 + j) per channel, zeros in front of a request's first token.  The last n - 1 rows of the
// stream are a request's state (fp32): every thread reads and replaces its own columns of it, and one CTA owns them.
// Launched with programmatic dependent launch: no __restrict__ on pointers whose contents a resident predecessor may still be
// writing.  Compiled without fast-math; all arithmetic in fp32.  `ld` is the row length: the width rounded up, padding columns
// zero.
#include "../api.h"
#include "../common/launch.cuh"
#include "../common/utils.cuh"

namespace b200 {
namespace {

template <typename T> struct alignas(4 * sizeof(T)) Quad { T v[4]; };
template <typename T> __device__ __forceinline__ void load4(float (&d)[4], const T* p) {
  const Quad<T> r = *reinterpret_cast<const Quad<T>*>(p);
#pragma unroll
  for (int j = 0; j < 4; ++j) d[j] = to_f(r.v[j]);
}
template <typename T> __device__ __forceinline__ void store4(T* p, const float (&s)[4]) {
  Quad<T> r;
#pragma unroll
  for (int j = 0; j < 4; ++j) r.v[j] = from_f<T>(s[j]);
  *reinterpret_cast<Quad<T>*>(p) = r;
}

// x + conv(x): `before` holds the rows in front, the oldest first; only the last n taps of TAPS exist.
template <int TAPS>
__device__ __forceinline__ void conv_add(float (&o)[4], const float (&x)[4], const float (&before)[TAPS - 1][4], const float* c,
                                         int n, int ld) {
  float w[4];
  load4(w, c + (int64_t)(n - 1) * ld);
#pragma unroll
  for (int e = 0; e < 4; ++e) o[e] = fmaf(w[e], x[e], x[e]);
#pragma unroll
  for (int j = 0; j < TAPS - 1; ++j) {
    const int k = j - (TAPS - n);         // tap of this row
    if (k < 0) continue;
    load4(w, c + (int64_t)k * ld);
#pragma unroll
    for (int e = 0; e < 4; ++e) o[e] = fmaf(w[e], before[j][e], o[e]);
  }
}

// TAPS = 0: a CTA per row.  Otherwise a CTA per request, which walks its (few) rows with the preceding ones in registers.
// NT threads hold a row as NV quads each.
template <typename T, int NT, int NV, int TAPS>
__global__ void __launch_bounds__(NT) postnorm_kernel(PostNormArgs a) {
  constexpr int kBefore = TAPS > 1 ? TAPS - 1 : 1;
  __shared__ float red[2][32];
  griddep_launch();
  griddep_wait();
  const int H = a.width, ld = a.ld, c0 = threadIdx.x * 4;
  const float inv_h = 1.f / H;
  int64_t t0 = blockIdx.x, t1 = t0 + 1, slot = -1;
  bool carried = false;
  if constexpr (TAPS > 0) {
    t0 = a.qsl[blockIdx.x];
    t1 = a.qsl[blockIdx.x + 1];
    slot = a.slots[blockIdx.x];
    if (slot >= a.num_slots || a.taps < 2) slot = -1;
    carried = slot >= 0 && a.has_init[blockIdx.x];
  }
  if (t0 >= t1) return;

  auto block_total = [&](float v, int buf) -> float {   // buffers alternate: one barrier per sum
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) red[buf][threadIdx.x >> 5] = v;
    __syncthreads();
    return warp_sum((threadIdx.x & 31) < NT / 32 ? red[buf][threadIdx.x & 31] : 0.f);
  };
  auto layer_norm = [&](float (&y)[NV][4], const float* w) {
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) s += (y[i][0] + y[i][1]) + (y[i][2] + y[i][3]);
    const float mean = block_total(s, 0) * inv_h;
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        y[i][j] = c0 + i * NT * 4 + j < H ? y[i][j] - mean : 0.f;
        ss += y[i][j] * y[i][j];
      }
    const float inv = 1.f / sqrtf(block_total(ss, 1) * inv_h + a.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int c = c0 + i * NT * 4 + j;
        y[i][j] = c < H ? y[i][j] * inv * w[c] : 0.f;
      }
  };

  [[maybe_unused]] float before[NV][kBefore][4];
  if constexpr (TAPS > 1) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = c0 + i * NT * 4;
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j) {
        const int k = j - (TAPS - a.taps);
#pragma unroll
        for (int e = 0; e < 4; ++e) before[i][j][e] = 0.f;
        if (carried && k >= 0 && c < ld) load4(before[i][j], a.state + (slot * (a.taps - 1) + k) * ld + c);
      }
    }
  }
  for (int64_t t = t0; t < t1; ++t) {
    float x[NV][4];
    if (a.table != nullptr) {
      const int64_t id = a.ids[t];
      const bool ok = id >= 0 && id < a.table_rows;
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = c0 + i * NT * 4;
        x[i][0] = x[i][1] = x[i][2] = x[i][3] = 0.f;
        if (c >= ld || !ok) continue;
        load4(x[i], reinterpret_cast<const T*>(a.table) + id * ld + c);
#pragma unroll
        for (int j = 0; j < 4; ++j) x[i][j] *= a.scale;
      }
    } else {
      float y[NV][4];
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = c0 + i * NT * 4;
        x[i][0] = x[i][1] = x[i][2] = x[i][3] = y[i][0] = y[i][1] = y[i][2] = y[i][3] = 0.f;
        if (c >= ld) continue;
        load4(x[i], a.x + t * ld + c);
        if (a.y != nullptr) load4(y[i], reinterpret_cast<const T*>(a.y) + t * a.y_stride + c);
      }
      for (int q = 0; q < a.k; ++q) {      // experts' rows; a choice without a row is the sublayer's input itself
        const int place = a.places[t * a.k + q];
        const float f = a.weights[t * a.k + q];
        const T* src = place >= 0 ? reinterpret_cast<const T*>(a.rows) + place * a.rows_stride
                                  : reinterpret_cast<const T*>(a.pass) + t * a.pass_stride;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
          const int c = c0 + i * NT * 4;
          if (c >= ld) continue;
          float z[4];
          load4(z, src + c);
#pragma unroll
          for (int j = 0; j < 4; ++j) y[i][j] = fmaf(f, z[j], y[i][j]);
        }
      }
#pragma unroll
      for (int i = 0; i < NV; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j)
          if (c0 + i * NT * 4 + j >= H) y[i][j] = 0.f;
      layer_norm(y, a.weight);
#pragma unroll
      for (int i = 0; i < NV; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) x[i][j] += y[i][j];
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = c0 + i * NT * 4;
      if (c < ld) store4(a.x + t * ld + c, x[i]);
    }
    T* h = reinterpret_cast<T*>(a.h) + t * ld;
    if constexpr (TAPS > 0) {
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = c0 + i * NT * 4;
        if (c >= ld) continue;
        float o[4];
        if constexpr (TAPS > 1) {
          conv_add<TAPS>(o, x[i], before[i], a.conv + c, a.taps, ld);
#pragma unroll
          for (int j = 0; j + 1 < TAPS - 1; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) before[i][j][e] = before[i][j + 1][e];
#pragma unroll
          for (int e = 0; e < 4; ++e) before[i][TAPS - 2][e] = x[i][e];
        }
        store4(h + c, o);
      }
    } else if (a.final_weight != nullptr) {
      layer_norm(x, a.final_weight);
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = c0 + i * NT * 4;
        if (c < ld) store4(h + c, x[i]);
      }
    }
  }
  if constexpr (TAPS > 1) {
    if (slot < 0) return;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = c0 + i * NT * 4;
      if (c >= ld) continue;
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j) {
        const int k = j - (TAPS - a.taps);
        if (k >= 0) store4(a.state + (slot * (a.taps - 1) + k) * ld + c, before[i][j]);
      }
    }
  }
}

// Thread = four columns, CTA = a run of rows of one request.  The first run's CTA owns the request's state.
constexpr int kConvThreads = 128, kConvRun = 32, kConvBatch = 4;
template <typename T, int TAPS>
__global__ void __launch_bounds__(kConvThreads) input_conv_kernel(PostNormArgs a) {
  griddep_launch();
  griddep_wait();
  const int c = (blockIdx.x * kConvThreads + threadIdx.x) * 4, ld = a.ld, n = a.taps, req = blockIdx.z;
  const int64_t q0 = a.qsl[req], q1 = a.qsl[req + 1], t0 = q0 + (int64_t)blockIdx.y * kConvRun, t1 = min(q1, t0 + kConvRun);
  if (t0 >= t1 || c >= ld) return;
  const float* x = a.x + c;
  float before[TAPS - 1][4];
  int64_t slot = a.slots[req];
  if (slot >= a.num_slots || n < 2 || t0 > q0) slot = -1;
  float* state = a.state + slot * (n - 1) * ld + c;       // used where slot >= 0
  const bool carried = slot >= 0 && a.has_init[req];
#pragma unroll
  for (int j = 0; j < TAPS - 1; ++j) {
    const int k = j - (TAPS - n);
#pragma unroll
    for (int e = 0; e < 4; ++e) before[j][e] = 0.f;
    if (k < 0) continue;
    // a run is at least TAPS - 1 rows long: only the first one reaches in front of the portion
    if (t0 > q0) load4(before[j], x + (t0 - (n - 1) + k) * ld);
    else if (carried) load4(before[j], state + (int64_t)k * ld);
  }
  if (slot >= 0) {      // the last n - 1 rows of old state and portion; row n - 1 - i from the end, old rows read before
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) {
      const int k = j - (TAPS - n);
      if (k < 0) continue;
      const int64_t t = q1 - (n - 1) + k;
      float v[4] = {0.f, 0.f, 0.f, 0.f};
      if (t >= q0) {
        load4(v, x + t * ld);
      } else {
        const int64_t back = q0 - t;          // rows in front of the portion: 1 = the newest old one
#pragma unroll
        for (int i = 0; i < TAPS - 1; ++i)
          if (TAPS - 1 - i == back) {
#pragma unroll
            for (int e = 0; e < 4; ++e) v[e] = before[i][e];
          }
      }
      store4(state + (int64_t)k * ld, v);
    }
  }
  T* h = reinterpret_cast<T*>(a.h) + c;
  for (int64_t t = t0; t < t1; t += kConvBatch) {
    float r[kConvBatch][4];
#pragma unroll
    for (int i = 0; i < kConvBatch; ++i)
      if (t + i < t1) load4(r[i], x + (t + i) * ld);
#pragma unroll
    for (int i = 0; i < kConvBatch; ++i) {
      if (t + i >= t1) break;
      float o[4];
      conv_add<TAPS>(o, r[i], before, a.conv + c, n, ld);
      store4(h + (t + i) * ld, o);
#pragma unroll
      for (int j = 0; j + 1 < TAPS - 1; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) before[j][e] = before[j + 1][e];
#pragma unroll
      for (int e = 0; e < 4; ++e) before[TAPS - 2][e] = r[i][e];
    }
  }
}

template <typename T, int TAPS>
int launch_postnorm(const PostNormArgs& a, cudaStream_t st) {
  const dim3 grid((unsigned)(TAPS > 0 ? a.num_reqs : a.T));
  const int quads = a.ld / 4;
#define B200_PN_LAUNCH(NT, NV) return (int)launch_pdl(postnorm_kernel<T, NT, NV, TAPS>, grid, dim3(NT), 0, st, a)
  if (quads <= 128) B200_PN_LAUNCH(128, 1);
  if (quads <= 256) B200_PN_LAUNCH(256, 1);
  if (quads <= 512) B200_PN_LAUNCH(512, 1);
  if (quads <= 1024) B200_PN_LAUNCH(512, 2);
  if (quads <= 2048) B200_PN_LAUNCH(1024, 2);
  if (quads <= 4096) B200_PN_LAUNCH(1024, 4);
#undef B200_PN_LAUNCH
  return 3;
}

template <typename T, int TAPS>
int launch_conv(const PostNormArgs& a, cudaStream_t st) {
  const dim3 grid((a.ld / 4 + kConvThreads - 1) / kConvThreads, (a.max_query_len + kConvRun - 1) / kConvRun, a.num_reqs);
  return (int)launch_pdl(input_conv_kernel<T, TAPS>, grid, dim3(kConvThreads), 0, st, a);
}

}  // namespace
}  // namespace b200

// The numbers of taps the kernels are built for serve every smaller one as well.
#define B200_TAPS(FN)                               \
  B200_DISPATCH_DTYPE(dtype, {                      \
    if (a.taps <= 3) return FN<T, 3>(a, st);        \
    if (a.taps <= 4) return FN<T, 4>(a, st);        \
    if (a.taps <= 8) return FN<T, 8>(a, st);        \
    if (a.taps <= 16) return FN<T, 16>(a, st);      \
    return 3;                                       \
  });

extern "C" int b200_postnorm(const PostNormArgs* args, int dtype, cudaStream_t st) {
  using namespace b200;
  const PostNormArgs& a = *args;
  if (a.T == 0) return 0;
  if (a.ld % 4 || a.width > a.ld || a.y_stride % 4 || a.rows_stride % 4 || a.pass_stride % 4) return 3;
  if (a.taps == 0) B200_DISPATCH_DTYPE(dtype, return (launch_postnorm<T, 0>(a, st)));
  B200_TAPS(launch_postnorm)
  return 3;
}

extern "C" int b200_input_conv(const PostNormArgs* args, int dtype, cudaStream_t st) {
  using namespace b200;
  const PostNormArgs& a = *args;
  if (a.T == 0) return 0;
  if (a.ld % 4 || a.taps < 1 || a.num_reqs > 65535 || (a.max_query_len + kConvRun - 1) / kConvRun > 65535) return 3;
  B200_TAPS(launch_conv)
  return 3;
}
