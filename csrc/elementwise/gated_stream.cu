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

constexpr int kThreads = 256;      // of bigram_rows

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

template <int N> __device__ __forceinline__ void copy_async(void* smem, const void* gmem) {
  const uint32_t s = static_cast<uint32_t>(__cvta_generic_to_shared(smem));
  asm volatile("cp.async.ca.shared.global [%0], [%1], %2;" ::"r"(s), "l"(gmem), "n"(N) : "memory");
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

// sigmoid with the hardware exponential and reciprocal (a few units in the last place of fp32)
__device__ __forceinline__ float gate(float z) { return __fdividef(1.f, 1.f + __expf(-z)); }

// kEmbed: rows come from the tables; otherwise from the stream and up to two gated summands.  NT threads hold a row as NV
// quads each.  kAhead (runs of rows): the next row travels into shared memory while this one is normalised and written;
// every thread copies and reads its own quads only, so that needs no barrier.
template <typename T, int NT, int NV, bool kEmbed, bool kAhead>
__global__ void __launch_bounds__(NT, 1024 / NT) stream_layernorm_kernel(StreamNormArgs a) {
  extern __shared__ __align__(16) uint8_t ahead[];
  __shared__ __align__(16) float red[2][NT / 32];
  griddep_launch();
  griddep_wait();
  const int H = a.width, ld = a.ld;
  const float inv_h = 1.f / H;
  T* hp = reinterpret_cast<T*>(a.h);
  T* sp = reinterpret_cast<T*>(a.shifted);
  const int c0 = threadIdx.x * 4;

  auto block_total = [&](float v, int buf) -> float {   // buffers alternate: one barrier per sum
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) red[buf][threadIdx.x >> 5] = v;
    __syncthreads();
    if constexpr (NT > 256) return warp_sum((threadIdx.x & 31) < NT / 32 ? red[buf][threadIdx.x & 31] : 0.f);
    float r = 0.f;
#pragma unroll
    for (int w = 0; w < NT / 32; w += 4) {
      const float4 q = *reinterpret_cast<const float4*>(&red[buf][w]);
      r += (q.x + q.y) + (q.z + q.w);
    }
    return r;
  };
  auto clear_tail = [&](float (&q)[4], int c) {         // columns from the width on
    if (c + 4 > H) {
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (c + j >= H) q[j] = 0.f;
    }
  };
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
      const int c = c0 + i * NT * 4;
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
          for (int j = 0; j < 4; ++j) y[i][j] += u[j] * gate(g[j]);
        }
        if (a.y2 != nullptr) {
          load4(u, reinterpret_cast<const T*>(a.y2) + t * a.y2_stride + c);
          load4(g, reinterpret_cast<const T*>(a.g2) + t * a.g2_stride + c);
#pragma unroll
          for (int j = 0; j < 4; ++j) y[i][j] += u[j] * gate(g[j]);
        }
      }
      clear_tail(y[i], c);
    }
  };
  // shared memory of kAhead: NV quads of the stream per thread, then of y1, g1, y2, g2
  auto own_x = [&](int i) { return reinterpret_cast<float*>(ahead) + (i * NT + threadIdx.x) * 4; };
  auto own_t = [&](int k, int i) {
    return reinterpret_cast<T*>(ahead + NV * NT * 16) + ((k * NV + i) * NT + threadIdx.x) * 4;
  };
  auto fetch = [&](int64_t t) {
    if constexpr (kAhead) {
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = c0 + i * NT * 4;
        if (c >= ld) continue;
        copy_async<16>(own_x(i), a.x_in + t * ld + c);
        if (a.y1 != nullptr) {
          copy_async<4 * sizeof(T)>(own_t(0, i), reinterpret_cast<const T*>(a.y1) + t * a.y1_stride + c);
          copy_async<4 * sizeof(T)>(own_t(1, i), reinterpret_cast<const T*>(a.g1) + t * a.g1_stride + c);
        }
        if (a.y2 != nullptr) {
          copy_async<4 * sizeof(T)>(own_t(2, i), reinterpret_cast<const T*>(a.y2) + t * a.y2_stride + c);
          copy_async<4 * sizeof(T)>(own_t(3, i), reinterpret_cast<const T*>(a.g2) + t * a.g2_stride + c);
        }
      }
      asm volatile("cp.async.commit_group;" ::: "memory");
    }
  };
  auto fetched_row = [&](float (&y)[NV][4]) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = c0 + i * NT * 4;
      y[i][0] = y[i][1] = y[i][2] = y[i][3] = 0.f;
      if (c >= ld) continue;
      load4(y[i], own_x(i));
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        if ((k == 0 ? a.y1 : a.y2) == nullptr) continue;
        float u[4], g[4];
        load4(u, own_t(2 * k, i));
        load4(g, own_t(2 * k + 1, i));
#pragma unroll
        for (int j = 0; j < 4; ++j) y[i][j] += u[j] * gate(g[j]);
      }
      clear_tail(y[i], c);
    }
  };
  auto norm = [&](float (&y)[NV][4], int64_t next) {    // next >= 0: the row to fetch once this one has been read
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) s += (y[i][0] + y[i][1]) + (y[i][2] + y[i][3]);
    const float mean = block_total(s, 0) * inv_h;
    if (next >= 0) fetch(next);
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
#pragma unroll
      for (int j = 0; j < 4; ++j) y[i][j] -= mean;
      clear_tail(y[i], c0 + i * NT * 4);
      ss += (y[i][0] * y[i][0] + y[i][1] * y[i][1]) + (y[i][2] * y[i][2] + y[i][3] * y[i][3]);
    }
    const float inv = 1.f / sqrtf(block_total(ss, 1) * inv_h + a.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = c0 + i * NT * 4;
      if (c >= H) continue;
      float w[4];
      if (c + 4 <= H) {
        load4(w, a.weight + c);
      } else {
#pragma unroll
        for (int j = 0; j < 4; ++j) w[j] = c + j < H ? a.weight[c + j] : 0.f;
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) y[i][j] *= inv * w[j];
    }
  };

  const int64_t lo = (int64_t)blockIdx.x * a.rows_per_cta, hi = min(a.T, lo + a.rows_per_cta);
  float y[NV][4], prev[NV][4];
  if (lo < hi) fetch(lo);
  for (int64_t t = lo; t < hi; ++t) {
    int64_t slot = -1, last = t;
    if (sp != nullptr) {
      const int r = a.req_of_token[t];
      if (t == a.qsl[r]) {                       // first row of a request
        last = a.qsl[r + 1] - 1;
        slot = a.slots[r];
        if (slot >= a.num_slots) slot = -1;
        const bool carried = slot >= 0 && a.has_init[r];
#pragma unroll
        for (int i = 0; i < NV; ++i) {
          const int c = c0 + i * NT * 4;
          prev[i][0] = prev[i][1] = prev[i][2] = prev[i][3] = 0.f;
          if (carried && c < ld) load4(prev[i], a.state + slot * ld + c);
        }
      } else if (t == lo) {
        row(t - 1, prev);
        norm(prev, -1);
      }
    }
    if constexpr (kAhead) fetched_row(y);
    else row(t, y);
    if (a.x_out != nullptr) {
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = c0 + i * NT * 4;
        if (c < ld) store4(a.x_out + t * ld + c, y[i]);
      }
    }
    norm(y, kAhead && t + 1 < hi ? t + 1 : -1);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = c0 + i * NT * 4;
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
    if (slot >= 0) {          // its last row's norm becomes the request's state
      if (last > t) {
        row(last, prev);
        norm(prev, -1);
      }
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = c0 + i * NT * 4;
        if (c < ld) store4(a.state + slot * ld + c, last > t ? prev[i] : y[i]);
      }
    }
#pragma unroll
    for (int i = 0; i < NV; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) prev[i][j] = y[i][j];
  }
}

// Runs of rows: one wave of CTAs, each with an equal share.
template <typename T, int NT, int NV>
int launch_runs(StreamNormArgs a, cudaStream_t st) {
  const int per_sm = 1024 / NT;
  a.rows_per_cta = (int)max((int64_t)4, (a.T + 148 * per_sm - 1) / (148 * per_sm));
  const dim3 grid((unsigned)((a.T + a.rows_per_cta - 1) / a.rows_per_cta));
  if (a.table != nullptr) return (int)launch_pdl(stream_layernorm_kernel<T, NT, NV, true, false>, grid, dim3(NT), 0, st, a);
  const int smem = NT * NV * (16 + 16 * (int)sizeof(T));
  const auto kern = stream_layernorm_kernel<T, NT, NV, false, true>;
  const cudaError_t e = ensure_dynamic_smem((const void*)kern, smem);
  if (e != cudaSuccess) return (int)e;
  return (int)launch_pdl(kern, grid, dim3(NT), smem, st, a);
}
// A CTA per row.
template <typename T, int NT, int NV>
int launch_rows(StreamNormArgs a, cudaStream_t st) {
  a.rows_per_cta = 1;
  const dim3 grid((unsigned)a.T);
  if (a.table != nullptr) return (int)launch_pdl(stream_layernorm_kernel<T, NT, NV, true, false>, grid, dim3(NT), 0, st, a);
  return (int)launch_pdl(stream_layernorm_kernel<T, NT, NV, false, false>, grid, dim3(NT), 0, st, a);
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
  // few rows: a CTA of up to 1024 threads for each; long portions: small CTAs over runs of rows, so that few rows are
  // computed twice
  const int quads = a.ld / 4;
  if (a.T <= 1024 || quads > 1024) {
    B200_DISPATCH_DTYPE(dtype, {
      if (quads <= 256) return launch_rows<T, 256, 1>(a, st);
      if (quads <= 512) return launch_rows<T, 512, 1>(a, st);
      if (quads <= 1024) return launch_rows<T, 1024, 1>(a, st);
      if (quads <= 2048) return launch_rows<T, 1024, 2>(a, st);
      if (quads <= 4096) return launch_rows<T, 1024, 4>(a, st);
    });
    return 3;
  }
  B200_DISPATCH_DTYPE(dtype, {
    if (quads <= 256) return launch_runs<T, 256, 1>(a, st);
    if (quads <= 512) return launch_runs<T, 256, 2>(a, st);
    return launch_runs<T, 512, 2>(a, st);
  });
  return (int)cudaGetLastError();
}
