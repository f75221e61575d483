// Kernels of decoders with an fp32 residual stream that is normalised once per layer and feeds several sublayers:
//   bigram_rows          row of the bigram table per token, from the token and the one before it (kept per request)
//   stream_layernorm     a row of the stream - scaled token row + bigram row, or stream + sum of sigmoid(gate) * y - then
//                        its LayerNorm in the GEMMs' type, and the same mixed with the previous token's (token shift)
// The previous token's norm is recomputed where it belongs to another CTA, so rows have no order among CTAs; the stream is
// therefore written to a second buffer.  A request's first row reads the norm that an earlier step left in its state slot,
// and the CTA of that row also leaves the norm of the request's last row there (recomputed): one CTA owns a slot.
// Launched with programmatic dependent launch: no __restrict__ on pointers whose contents a resident predecessor may still
// be writing.  Compiled without fast-math; all arithmetic in fp32.  `ld` is the row length: the width rounded up so that
// rows stay 16-byte aligned; padding columns are zero.
#include "../api.h"
#include "../common/launch.cuh"
#include "../common/utils.cuh"

namespace b200 {
namespace {

constexpr int kThreads = 256;

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

// One CTA per request: the state is read before any row is written and replaced at the end.
__global__ void __launch_bounds__(kThreads) bigram_rows_kernel(int64_t* rows, const int64_t* ids, int64_t* state,
                                                               const int* qsl, const int* slots, const int* has_init,
                                                               int64_t num_slots, int64_t mul_prev, int64_t mul_cur,
                                                               int64_t buckets) {
  griddep_launch();
  griddep_wait();
  const int r = blockIdx.x, t0 = qsl[r], t1 = qsl[r + 1];
  const int64_t slot = slots[r];
  const bool held = slot >= 0 && slot < num_slots;
  int64_t before = -1;
  if (held && has_init[r]) before = state[slot];
  __syncthreads();
  for (int t = t0 + threadIdx.x; t < t1; t += kThreads) {
    const int64_t prev = t > t0 ? ids[t - 1] : before;
    rows[t] = prev < 0 ? buckets : (prev * mul_prev + ids[t] * mul_cur) % buckets;
  }
  if (threadIdx.x == 0 && held && t1 > t0) state[slot] = ids[t1 - 1];
}

// kEmbed: rows come from the tables; otherwise from the stream and up to two gated summands.
template <typename T, int NV, bool kEmbed>
__global__ void __launch_bounds__(kThreads) stream_layernorm_kernel(StreamNormArgs a) {
  __shared__ float red[32];
  griddep_launch();
  griddep_wait();
  const int H = a.width, ld = a.ld;
  T* hp = reinterpret_cast<T*>(a.h);
  T* sp = reinterpret_cast<T*>(a.shifted);

  auto row = [&](int64_t t, float (&y)[NV][4]) {
    [[maybe_unused]] int64_t id = 0, bg = 0;
    [[maybe_unused]] bool id_ok = false, bg_ok = false;
    if constexpr (kEmbed) {
      id = a.ids[t];
      id_ok = id >= 0 && id < a.table_rows;
      bg = a.bigram_rows != nullptr ? a.bigram_rows[t] : -1;
      bg_ok = bg >= 0 && bg < a.bigram_table_rows;
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * kThreads + threadIdx.x) * 4;
      y[i][0] = y[i][1] = y[i][2] = y[i][3] = 0.f;
      if (c >= ld) continue;
      float u[4], g[4];
      if constexpr (kEmbed) {
        if (id_ok) {
          load4(u, reinterpret_cast<const T*>(a.table) + id * ld + c);
#pragma unroll
          for (int j = 0; j < 4; ++j) y[i][j] = u[j] * a.scale;
        }
        if (bg_ok) {
          load4(u, reinterpret_cast<const T*>(a.bigram_table) + bg * ld + c);
#pragma unroll
          for (int j = 0; j < 4; ++j) y[i][j] += u[j];
        }
      } else {
        load4(y[i], a.x_in + t * ld + c);
        if (a.y1 != nullptr) {
          load4(u, reinterpret_cast<const T*>(a.y1) + t * a.y1_stride + c);
          load4(g, reinterpret_cast<const T*>(a.g1) + t * a.g1_stride + c);
#pragma unroll
          for (int j = 0; j < 4; ++j) u[j] = u[j] / (1.f + expf(-g[j]));
          if (a.y2 != nullptr) {
            float u2[4];
            load4(u2, reinterpret_cast<const T*>(a.y2) + t * a.y2_stride + c);
            load4(g, reinterpret_cast<const T*>(a.g2) + t * a.g2_stride + c);
#pragma unroll
            for (int j = 0; j < 4; ++j) u[j] += u2[j] / (1.f + expf(-g[j]));
          }
#pragma unroll
          for (int j = 0; j < 4; ++j) y[i][j] += u[j];
        }
      }
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (c + j >= H) y[i][j] = 0.f;
    }
  };
  auto norm = [&](float (&y)[NV][4]) {
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) s += y[i][j];
    const float mean = block_sum(s, red) / H;
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int c = (i * kThreads + threadIdx.x) * 4 + j;
        const float d = c < H ? y[i][j] - mean : 0.f;
        y[i][j] = d;
        ss += d * d;
      }
    const float inv = 1.f / sqrtf(block_sum(ss, red) / H + a.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int c = (i * kThreads + threadIdx.x) * 4 + j;
        y[i][j] = c < H ? y[i][j] * inv * a.weight[c] : 0.f;
      }
  };

  const int64_t lo = (int64_t)blockIdx.x * a.rows_per_cta, hi = min(a.T, lo + a.rows_per_cta);
  float y[NV][4], prev[NV][4];
  for (int64_t t = lo; t < hi; ++t) {
    int64_t slot = -1, last = t;
    bool first = false;
    if (sp != nullptr) {
      const int r = a.req_of_token[t];
      first = t == a.qsl[r];
      if (first) {
        last = a.qsl[r + 1] - 1;
        slot = a.slots[r];
        if (slot >= a.num_slots) slot = -1;
        const bool carried = slot >= 0 && a.has_init[r];
#pragma unroll
        for (int i = 0; i < NV; ++i) {
          const int c = (i * kThreads + threadIdx.x) * 4;
          prev[i][0] = prev[i][1] = prev[i][2] = prev[i][3] = 0.f;
          if (carried && c < ld) load4(prev[i], a.state + slot * ld + c);
        }
      } else if (t == lo) {
        row(t - 1, prev);
        norm(prev);
      }
    }
    row(t, y);
    if (a.x_out != nullptr) {
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = (i * kThreads + threadIdx.x) * 4;
        if (c < ld) store4(a.x_out + t * ld + c, y[i]);
      }
    }
    norm(y);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * kThreads + threadIdx.x) * 4;
      if (c >= ld) continue;
      store4(hp + t * ld + c, y[i]);
      if (sp == nullptr) continue;
      float m[4], o[4];
      load4(m, a.mix + c);
#pragma unroll
      for (int j = 0; j < 4; ++j) o[j] = y[i][j] + (prev[i][j] - y[i][j]) * m[j];
      store4(sp + t * ld + c, o);
    }
    if (sp == nullptr) continue;
    if (slot >= 0) {          // first row of a request: its last row's norm becomes the state
      if (last > t) {
        row(last, prev);
        norm(prev);
      }
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = (i * kThreads + threadIdx.x) * 4;
        if (c < ld) store4(a.state + slot * ld + c, last > t ? prev[i] : y[i]);
      }
    }
#pragma unroll
    for (int i = 0; i < NV; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) prev[i][j] = y[i][j];
  }
}

template <typename T, int NV>
void launch_stream(const StreamNormArgs& a, cudaStream_t st) {
  const dim3 grid((unsigned)((a.T + a.rows_per_cta - 1) / a.rows_per_cta));
  if (a.table != nullptr) launch_pdl(stream_layernorm_kernel<T, NV, true>, grid, dim3(kThreads), 0, st, a);
  else launch_pdl(stream_layernorm_kernel<T, NV, false>, grid, dim3(kThreads), 0, st, a);
}

}  // namespace
}  // namespace b200

extern "C" int b200_bigram_rows(int64_t* rows, const int64_t* ids, int64_t* state, const int* qsl, const int* slots,
                                const int* has_init, int B, int64_t num_slots, int64_t mul_prev, int64_t mul_cur,
                                int64_t buckets, cudaStream_t st) {
  using namespace b200;
  if (B == 0) return 0;
  if (buckets < 1) return 2;
  launch_pdl(bigram_rows_kernel, dim3(B), dim3(kThreads), 0, st, rows, ids, state, qsl, slots, has_init, num_slots, mul_prev,
             mul_cur, buckets);
  return (int)cudaGetLastError();
}

extern "C" int b200_stream_layernorm(const StreamNormArgs* args, int dtype, cudaStream_t st) {
  using namespace b200;
  StreamNormArgs a = *args;
  if (a.T == 0) return 0;
  if (a.ld % 4 || a.width > a.ld || a.y1_stride % 4 || a.y2_stride % 4 || a.g1_stride % 4 || a.g2_stride % 4) return 3;
  if (a.x_out != nullptr && a.x_out == a.x_in) return 2;   // rows are read again by the CTA of the next row
  // decode-sized batches: a CTA per row; long portions: runs of rows, so that few rows are computed twice
  a.rows_per_cta = a.T <= 1024 ? 1 : 8;
  const int need = (a.ld / 4 + kThreads - 1) / kThreads;
  B200_DISPATCH_DTYPE(dtype, {
    if (need <= 1) launch_stream<T, 1>(a, st);
    else if (need <= 2) launch_stream<T, 2>(a, st);
    else if (need <= 4) launch_stream<T, 4>(a, st);
    else if (need <= 8) launch_stream<T, 8>(a, st);
    else if (need <= 16) launch_stream<T, 16>(a, st);
    else return 3;
  });
  return (int)cudaGetLastError();
}
