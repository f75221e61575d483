// Kernels around multi-head latent attention with any sizes (one latent row and one rotated key part per token, shared by
// all heads):
//   rotary_table     cos / sin of every position of the step, shared by all layers with the same rotation
//   latent_prep      one pass over a token's down-projections: RMS norm of the query latent (input of the next GEMM), RMS
//                    norm of the key / value latent and rotation of the shared key part, both into the paged cache
//   rotate_heads     the rotated part of every query head, in place (prompt portions)
//   absorb_query     q_head . W_uk (a token's query in the latent space) next to its rotated part (decoding)
//   expand_value     latent outputs . W_uv^T, times the head's output gate (decoding)
//   gather_window    the cached rows that the portions of a step can see, request by request, contiguous
// absorb_query and expand_value stream the weights of a head through the tensor cores for the 512 / 64 / 128 sizes of
// 16-bit models; the generic forms take any size and fp32.  Rotations pair column i with i + n / 2.
// No __restrict__ on pointers that a resident predecessor may still be writing (programmatic dependent launch); weights are
// fetched before the dependency wait.  Compiled without fast-math.
#include "../api.h"
#include "../common/launch.cuh"
#include "attn_common.cuh"

namespace b200 {
namespace {

__global__ void __launch_bounds__(256) rotary_table_kernel(float2* out, const int64_t* positions, const int64_t* turns,
                                                           int pairs, int64_t n) {
  griddep_launch();
  griddep_wait();
  const int64_t i = (int64_t)blockIdx.x * 256 + threadIdx.x;
  if (i >= n) return;
  // turns per position as a 64-bit fraction of a turn: the product wraps modulo one turn by itself
  const int64_t a = (int64_t)((uint64_t)positions[i / pairs] * (uint64_t)turns[i % pairs]);
  float s, c;
  sincospif((float)a * 0x1p-63f, &s, &c);
  out[i] = make_float2(c, s);
}

// value of column i of a vector x whose first 2 * pairs columns are rotated
template <typename F>
__device__ __forceinline__ float rotated(int i, int pairs, const float2* cs, F x) {
  if (i >= 2 * pairs) return x(i);
  const int j = i < pairs ? i : i - pairs;
  const float2 r = cs[j];
  return i < pairs ? x(i) * r.x - x(i + pairs) * r.y : x(i) * r.x + x(i - pairs) * r.y;
}

template <typename T> struct alignas(4 * sizeof(T)) Quad { T v[4]; };
template <typename T> __device__ __forceinline__ float4 get4(const T* p) {
  const Quad<T> r = *reinterpret_cast<const Quad<T>*>(p);
  return make_float4(to_f(r.v[0]), to_f(r.v[1]), to_f(r.v[2]), to_f(r.v[3]));
}
template <typename T> __device__ __forceinline__ void put4(T* p, float a, float b, float c, float d) {
  *reinterpret_cast<Quad<T>*>(p) = Quad<T>{{from_f<T>(a), from_f<T>(b), from_f<T>(c), from_f<T>(d)}};
}

template <typename T, int NT>
__global__ void __launch_bounds__(NT) latent_prep_kernel(LatentPrepArgs a) {
  extern __shared__ __align__(16) float sv[];          // [Q query latent | C + R key / value latent and shared key part]
  __shared__ float red[2][NT / 32];
  griddep_launch();
  griddep_wait();
  const int64_t t = blockIdx.x;
  const int tid = threadIdx.x, Q = a.q_rank, C = a.kv_rank, R = a.rot_dim;
  const T* q = reinterpret_cast<const T*>(a.q_down) + t * a.stride;
  const T* kv = reinterpret_cast<const T*>(a.kv_down) + t * a.stride;
  float sq = 0.f, sc = 0.f;
  if (a.vec) {
#pragma unroll 4
    for (int i = tid * 4; i < Q; i += 4 * NT) {
      const float4 f = get4(q + i);
      *reinterpret_cast<float4*>(sv + i) = f;
      sq += (f.x * f.x + f.y * f.y) + (f.z * f.z + f.w * f.w);
    }
#pragma unroll 2
    for (int i = tid * 4; i < C + R; i += 4 * NT) {
      const float4 f = get4(kv + i);
      *reinterpret_cast<float4*>(sv + Q + i) = f;
      if (i < C) sc += (f.x * f.x + f.y * f.y) + (f.z * f.z + f.w * f.w);
    }
  } else {
    for (int i = tid; i < Q; i += NT) { const float f = to_f(q[i]); sv[i] = f; sq += f * f; }
    for (int i = tid; i < C + R; i += NT) { const float f = to_f(kv[i]); sv[Q + i] = f; if (i < C) sc += f * f; }
  }
  sq = warp_sum(sq);
  sc = warp_sum(sc);
  if ((tid & 31) == 0) { red[0][tid >> 5] = sq; red[1][tid >> 5] = sc; }
  __syncthreads();
  sq = sc = 0.f;
#pragma unroll
  for (int w = 0; w < NT / 32; ++w) { sq += red[0][w]; sc += red[1][w]; }
  const float iq = 1.f / sqrtf(sq / Q + a.eps), ic = 1.f / sqrtf(sc / C + a.eps);
  T* qo = reinterpret_cast<T*>(a.q_out) + t * a.q_out_stride;
  const int64_t slot = a.slots[t];
  const bool store = slot >= 0 && slot < a.total_slots;
  T* co = reinterpret_cast<T*>(a.cache) + (store ? slot : 0) * a.row;
  const float2* cs = reinterpret_cast<const float2*>(a.table) + t * a.pairs;
  const float* sk = sv + Q + C;
  // cache row: latent, zeros up to rot_off, shared key part, zeros
  auto cached = [&](int i) -> float {
    if (i < C) return sv[Q + i] * ic * a.kv_norm[i];
    const int j = i - a.rot_off;
    return j >= 0 && j < R ? rotated(j, a.pairs, cs, [&](int k) { return sk[k]; }) : 0.f;
  };
  if (a.vec) {   // sizes are multiples of 4: a quad lies inside one part
    auto scaled = [&](const float* x, float inv, const float* w, T* dst) {
      const float4 u = *reinterpret_cast<const float4*>(x), v = *reinterpret_cast<const float4*>(w);
      put4(dst, u.x * inv * v.x, u.y * inv * v.y, u.z * inv * v.z, u.w * inv * v.w);
    };
    for (int i = tid * 4; i < a.q_out_stride; i += 4 * NT) {
      if (i < Q) scaled(sv + i, iq, a.q_norm + i, qo + i);
      else put4(qo + i, 0.f, 0.f, 0.f, 0.f);
    }
    if (store)
      for (int i = tid * 4; i < a.row; i += 4 * NT) {
        if (i < C) scaled(sv + Q + i, ic, a.kv_norm + i, co + i);
        else put4(co + i, cached(i), cached(i + 1), cached(i + 2), cached(i + 3));
      }
  } else {
    for (int i = tid; i < a.q_out_stride; i += NT) qo[i] = from_f<T>(i < Q ? sv[i] * iq * a.q_norm[i] : 0.f);
    if (store)
      for (int i = tid; i < a.row; i += NT) co[i] = from_f<T>(cached(i));
  }
}

// q [T, H, D]: columns off .. off + 2 * pairs of every head; V pairs per thread
template <typename T, int V>
__global__ void __launch_bounds__(256) rotate_heads_kernel(T* q, const float2* table, int64_t n, int H, int D, int off,
                                                           int pairs) {
  griddep_launch();
  griddep_wait();
  const int per = pairs / V;
  const int64_t i = (int64_t)blockIdx.x * 256 + threadIdx.x;
  if (i >= n) return;
  const int64_t th = i / per;
  const int p = (int)(i % per) * V;
  T* u = q + th * D + off + p;
  const float2* cs = table + (th / H) * pairs + p;
#pragma unroll
  for (int j = 0; j < V; j += 2) {
    if constexpr (V == 1) {
      const float a = to_f(u[0]), b = to_f(u[pairs]);
      u[0] = from_f<T>(a * cs[0].x - b * cs[0].y);
      u[pairs] = from_f<T>(b * cs[0].x + a * cs[0].y);
    } else {
      struct alignas(2 * sizeof(T)) Two { T a, b; };
      Two x = *reinterpret_cast<const Two*>(u + j), y = *reinterpret_cast<const Two*>(u + j + pairs);
      const float2 c0 = cs[j], c1 = cs[j + 1];
      const float xa = to_f(x.a), xb = to_f(x.b), ya = to_f(y.a), yb = to_f(y.b);
      x.a = from_f<T>(xa * c0.x - ya * c0.y); x.b = from_f<T>(xb * c1.x - yb * c1.y);
      y.a = from_f<T>(ya * c0.x + xa * c0.y); y.b = from_f<T>(yb * c1.x + xb * c1.y);
      *reinterpret_cast<Two*>(u + j) = x;
      *reinterpret_cast<Two*>(u + j + pairs) = y;
    }
  }
}

// ------------------------------------------------------------------------------------------------ 512 / 64 / 128 sizes
constexpr int kC = 512, kR = 64, kD = 128, kRow = kC + kR, kQ = kD + kR;
constexpr int kTile = 64;     // latent columns per CTA of absorb_query
constexpr int kVTile = 16;    // value columns per CTA of expand_value

__device__ __forceinline__ int lane_row() { return (threadIdx.x & 7) + ((threadIdx.x >> 3) & 1) * 8; }
__device__ __forceinline__ int lane_chunk() { return (threadIdx.x & 31) >> 4; }

// out[t, h, n] = sum_d q[t, h, d] W[h, d, n] for a tile of 64 columns and 16 MT tokens; the last column block rotates.
template <typename T, int MT>
__global__ void __launch_bounds__(128) absorb_query_kernel(T* out, const T* q, const T* w, int64_t w_head, const float2* table,
                                                           int H, int pairs, int64_t T_) {
  __shared__ __align__(16) T sW[kD * kTile];
  __shared__ __align__(16) T sQ[16 * MT * kD];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.y;
  const int64_t t0 = (int64_t)blockIdx.z * 16 * MT;
  const int nt = (int)min((int64_t)(16 * MT), T_ - t0);
  const bool rot = blockIdx.x == kC / kTile;
  griddep_launch();
  if (!rot) {
    const T* src = w + h * w_head + blockIdx.x * kTile;
#pragma unroll
    for (int c = tid; c < kD * (kTile / 8); c += 128)
      cp_async16(sW + swz<kTile>(c / (kTile / 8), c % (kTile / 8)), src + (int64_t)(c / (kTile / 8)) * kC + (c % (kTile / 8)) * 8,
                 true);
    cp_async_commit();
  }
  griddep_wait();
  if (rot) {
    for (int i = tid; i < nt * kR; i += 128) {
      const int64_t t = t0 + i / kR;
      const T* x = q + (t * H + h) * kQ + kD;
      out[(t * H + h) * kRow + kC + i % kR] = from_f<T>(rotated(i % kR, pairs, table + t * pairs, [&](int k) { return to_f(x[k]); }));
    }
    return;
  }
  for (int c = tid; c < 16 * MT * (kD / 8); c += 128) {
    const int r = c / (kD / 8), ch = c % (kD / 8);
    const bool ok = r < nt;
    cp_async16(sQ + swz<kD>(r, ch), q + ((t0 + (ok ? r : 0)) * H + h) * kQ + ch * 8, ok);
  }
  cp_async_commit();
  cp_async_wait<0>();
  __syncthreads();
  float acc[MT][2][4] = {};
#pragma unroll
  for (int k = 0; k < kD / 16; ++k) {
    uint32_t b[4];
    ldmatrix_x4_trans(b, sW + swz<kTile>(k * 16 + lane_row(), warp * 2 + lane_chunk()));
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      uint32_t a[4];
      ldmatrix_x4(a, sQ + swz<kD>(m * 16 + lane_row(), k * 2 + lane_chunk()));
      MmaTraits<T>::mma(acc[m][0], a, b[0], b[1]);
      MmaTraits<T>::mma(acc[m][1], a, b[2], b[3]);
    }
  }
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int r = m * 16 + (lane >> 2) + half * 8;
      if (r >= nt) continue;
      T* dst = out + ((t0 + r) * H + h) * kRow + blockIdx.x * kTile + warp * 16 + (lane & 3) * 2;
#pragma unroll
      for (int j = 0; j < 2; ++j)
        *reinterpret_cast<uint32_t*>(dst + j * 8) = MmaTraits<T>::pack(acc[m][j][half * 2], acc[m][j][half * 2 + 1]);
    }
}

// out[t, h, v] = sigmoid(gate[t, h]) * sum_c o[t, h, c] W[h, v, c] for 16 value columns and 16 MT tokens; the four warps
// take a quarter of the latent columns each.
template <typename T, int MT>
__global__ void __launch_bounds__(128) expand_value_kernel(T* out, const T* o, const T* w, int64_t w_head, const T* gate,
                                                           int64_t gate_stride, int H, int64_t T_) {
  extern __shared__ __align__(16) uint8_t smem_ev[];
  T* sW = reinterpret_cast<T*>(smem_ev);                 // [16][512]
  T* sO = sW + kVTile * kC;                              // [16 MT][512], then the warps' partial sums
  float* sS = reinterpret_cast<float*>(sO);              // [4][16 MT][16]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.y;
  const int64_t t0 = (int64_t)blockIdx.z * 16 * MT;
  const int nt = (int)min((int64_t)(16 * MT), T_ - t0);
  griddep_launch();
  const T* src = w + h * w_head + (int64_t)blockIdx.x * kVTile * kC;
#pragma unroll
  for (int c = tid; c < kVTile * (kC / 8); c += 128)
    cp_async16(sW + swz<kC>(c / (kC / 8), c % (kC / 8)), src + (int64_t)c * 8, true);
  cp_async_commit();
  griddep_wait();
  for (int c = tid; c < 16 * MT * (kC / 8); c += 128) {
    const int r = c / (kC / 8), ch = c % (kC / 8);
    const bool ok = r < nt;
    cp_async16(sO + swz<kC>(r, ch), o + ((t0 + (ok ? r : 0)) * H + h) * kC + ch * 8, ok);
  }
  cp_async_commit();
  cp_async_wait<0>();
  __syncthreads();
  float acc[MT][2][4] = {};
#pragma unroll
  for (int k = 0; k < kC / 64; ++k) {
    const int ks = warp * (kC / 64) + k;
    uint32_t b[4];
    ldmatrix_x4(b, sW + swz<kC>((lane & 7) + (lane >> 4) * 8, ks * 2 + ((lane >> 3) & 1)));
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      uint32_t a[4];
      ldmatrix_x4(a, sO + swz<kC>(m * 16 + lane_row(), ks * 2 + lane_chunk()));
      MmaTraits<T>::mma(acc[m][0], a, b[0], b[1]);
      MmaTraits<T>::mma(acc[m][1], a, b[2], b[3]);
    }
  }
  __syncthreads();
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e)
        sS[(warp * 16 * MT + m * 16 + (lane >> 2) + (e >> 1) * 8) * 16 + j * 8 + (lane & 3) * 2 + (e & 1)] = acc[m][j][e];
  __syncthreads();
  for (int i = tid; i < nt * 8; i += 128) {
    const int r = i / 8, c = (i % 8) * 2;
    float2 s = make_float2(0.f, 0.f);
#pragma unroll
    for (int g = 0; g < 4; ++g) {
      const float2 v = *reinterpret_cast<const float2*>(sS + (g * 16 * MT + r) * 16 + c);
      s.x += v.x; s.y += v.y;
    }
    if (gate != nullptr) {
      const float f = 1.f / (1.f + expf(-to_f(gate[(t0 + r) * gate_stride + h])));
      s.x *= f; s.y *= f;
    }
    *reinterpret_cast<uint32_t*>(out + ((t0 + r) * H + h) * kD + blockIdx.x * kVTile + c) = MmaTraits<T>::pack(s.x, s.y);
  }
}

template <typename T, int MT>
int launch_absorb(void* out, const void* q, const void* w, int64_t w_head, const float* table, int64_t T_, int H, int pairs,
                  cudaStream_t st) {
  const dim3 grid(kC / kTile + 1, H, (unsigned)((T_ + 16 * MT - 1) / (16 * MT)));
  return (int)launch_pdl(absorb_query_kernel<T, MT>, grid, dim3(128), 0, st, (T*)out, (const T*)q, (const T*)w, w_head,
                         (const float2*)table, H, pairs, T_);
}
template <typename T, int MT>
int launch_expand(void* out, const void* o, const void* w, int64_t w_head, const void* gate, int64_t gate_stride, int64_t T_,
                  int H, cudaStream_t st) {
  const size_t smem = (size_t)(kVTile + 16 * MT) * kC * sizeof(T);
  const cudaError_t e = ensure_dynamic_smem((const void*)expand_value_kernel<T, MT>, (int)smem);
  if (e != cudaSuccess) return (int)e;
  const dim3 grid(kD / kVTile, H, (unsigned)((T_ + 16 * MT - 1) / (16 * MT)));
  return (int)launch_pdl(expand_value_kernel<T, MT>, grid, dim3(128), smem, st, (T*)out, (const T*)o, (const T*)w, w_head,
                         (const T*)gate, gate_stride, H, T_);
}

// ------------------------------------------------------------------------------------------------ any size
// q [T, H, D + R], w [H][D][C] (rows C apart) -> out [T, H, row] = [q . W | zeros | rotated part at rot_off | zeros]
template <typename T>
__global__ void __launch_bounds__(128) absorb_query_generic_kernel(T* out, const T* q, const T* w, int64_t w_head,
                                                                   const float2* table, int H, int D, int R, int C, int rot_off,
                                                                   int row, int pairs) {
  extern __shared__ float sx[];
  griddep_launch();
  griddep_wait();
  const int64_t t = blockIdx.x;
  const int h = blockIdx.y;
  const T* x = q + (t * H + h) * (int64_t)(D + R);
  for (int i = threadIdx.x; i < D + R; i += 128) sx[i] = to_f(x[i]);
  __syncthreads();
  T* dst = out + (t * H + h) * (int64_t)row;
  for (int n = threadIdx.x; n < row; n += 128) {
    float s = 0.f;
    if (n < C) {
      const T* wc = w + h * w_head + n;
      for (int d = 0; d < D; ++d) s += sx[d] * to_f(wc[(int64_t)d * C]);
    } else if (n >= rot_off && n < rot_off + R) {
      s = rotated(n - rot_off, pairs, table + t * pairs, [&](int k) { return sx[D + k]; });
    }
    dst[n] = from_f<T>(s);
  }
}

// o [T, H, C], w [H][Dv][C] -> out [T, H, Dv] (rows of a token out_stride apart)
template <typename T>
__global__ void __launch_bounds__(128) expand_value_generic_kernel(T* out, int64_t out_stride, const T* o, const T* w,
                                                                   int64_t w_head, const T* gate, int64_t gate_stride, int H,
                                                                   int Dv, int C) {
  extern __shared__ float sx[];
  griddep_launch();
  griddep_wait();
  const int64_t t = blockIdx.x;
  const int h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const T* x = o + (t * H + h) * (int64_t)C;
  for (int i = threadIdx.x; i < C; i += 128) sx[i] = to_f(x[i]);
  __syncthreads();
  const float f = gate != nullptr ? 1.f / (1.f + expf(-to_f(gate[t * gate_stride + h]))) : 1.f;
  for (int v = warp; v < Dv; v += 4) {
    const T* wr = w + h * w_head + (int64_t)v * C;
    float s = 0.f;
    for (int c = lane; c < C; c += 32) s += sx[c] * to_f(wr[c]);
    s = warp_sum(s);
    if (lane == 0) out[t * out_stride + (int64_t)h * Dv + v] = from_f<T>(s * f);
  }
}

// Request r's last lens[r] cached rows into out[starts[r] ..]; one warp per row of `units` 16-byte units.
__global__ void __launch_bounds__(256) gather_window_kernel(uint4* out, const uint4* cache, const int* block_tables,
                                                            const int* seq_lens, const int* starts, const int* lens,
                                                            int64_t max_blocks, int block_size, int64_t num_blocks,
                                                            int units, int64_t total) {
  griddep_launch();
  griddep_wait();
  const int r = blockIdx.y, i = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (i >= lens[r]) return;
  const int pos = seq_lens[r] - lens[r] + i;
  const int64_t dst = (int64_t)starts[r] + i, bi = pos / block_size;
  if (pos < 0 || dst < 0 || dst >= total) return;
  int64_t blk = bi < max_blocks ? block_tables[r * max_blocks + bi] : -1;
  const bool ok = blk >= 0 && blk < num_blocks;
  const uint4* src = cache + ((ok ? blk : 0) * block_size + pos % block_size) * units;
  for (int u = lane; u < units; u += 32) out[dst * units + u] = ok ? src[u] : make_uint4(0, 0, 0, 0);
}

}  // namespace
}  // namespace b200

using namespace b200;

extern "C" int b200_rotary_table(float* out, const int64_t* positions, const int64_t* turns, int64_t T_, int pairs,
                                 cudaStream_t st) {
  const int64_t n = T_ * pairs;
  if (n == 0) return 0;
  launch_pdl(rotary_table_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, st, (float2*)out, positions, turns, pairs, n);
  return (int)cudaGetLastError();
}

extern "C" int b200_latent_prep(const LatentPrepArgs* args, int64_t T_, int dtype, cudaStream_t st) {
  LatentPrepArgs a = *args;
  if (T_ == 0) return 0;
  if (a.rot_off < a.kv_rank || a.rot_off + a.rot_dim > a.row || 2 * a.pairs > a.rot_dim || a.q_rank > a.q_out_stride) return 2;
  const size_t smem = (size_t)(a.q_rank + a.kv_rank + a.rot_dim) * sizeof(float);
  if (smem > 46 * 1024) return 3;
  a.vec = a.q_rank % 4 == 0 && a.kv_rank % 4 == 0 && a.rot_dim % 4 == 0 && a.stride % 4 == 0 && a.q_out_stride % 4 == 0 &&
          a.row % 4 == 0 && a.rot_off % 4 == 0 && ((uintptr_t)a.q_norm | (uintptr_t)a.kv_norm | (uintptr_t)a.q_down | (uintptr_t)a.kv_down | (uintptr_t)a.q_out | (uintptr_t)a.cache) % 16 == 0;
  // few tokens: more threads each, for a short chain; many tokens: more of them at once
  B200_DISPATCH_DTYPE(dtype, {
    if (T_ <= 256) launch_pdl(latent_prep_kernel<T, 512>, dim3((unsigned)T_), dim3(512), smem, st, a);
    else launch_pdl(latent_prep_kernel<T, 128>, dim3((unsigned)T_), dim3(128), smem, st, a);
  });
  return (int)cudaGetLastError();
}

extern "C" int b200_rotate_heads(void* q, const float* table, int64_t T_, int H, int D, int off, int pairs, int dtype,
                                 cudaStream_t st) {
  if (T_ == 0 || pairs == 0) return 0;
  if (off < 0 || off + 2 * pairs > D) return 2;
  const bool two = pairs % 2 == 0 && off % 2 == 0 && D % 2 == 0 && (uintptr_t)q % 16 == 0;
  const int64_t n = T_ * H * (pairs / (two ? 2 : 1));
  const dim3 grid((unsigned)((n + 255) / 256));
  B200_DISPATCH_DTYPE(dtype, {
    if (two) launch_pdl(rotate_heads_kernel<T, 2>, grid, dim3(256), 0, st, (T*)q, (const float2*)table, n, H, D, off, pairs);
    else launch_pdl(rotate_heads_kernel<T, 1>, grid, dim3(256), 0, st, (T*)q, (const float2*)table, n, H, D, off, pairs);
  });
  return (int)cudaGetLastError();
}

extern "C" int b200_absorb_query(void* out, const void* q, const void* w, int64_t w_head, const float* table, int64_t T_, int H,
                                 int D, int R, int C, int rot_off, int row, int pairs, int dtype, cudaStream_t st) {
  if (T_ == 0) return 0;
  if (H > 65535 || 2 * pairs > R || rot_off < C || rot_off + R > row) return 2;
  if (dtype != kF32 && D == kD && R == kR && C == kC && rot_off == kC && row == kRow && w_head % 8 == 0 &&
      ((uintptr_t)q | (uintptr_t)w | (uintptr_t)out) % 16 == 0 && T_ <= 64 * 65535) {
#define B200_ABSORB(MT)                                                                                              \
  return dtype == kBF16 ? launch_absorb<__nv_bfloat16, MT>(out, q, w, w_head, table, T_, H, pairs, st)                \
                        : launch_absorb<__half, MT>(out, q, w, w_head, table, T_, H, pairs, st)
    if (T_ <= 16) B200_ABSORB(1);
    if (T_ <= 32) B200_ABSORB(2);
    B200_ABSORB(4);
#undef B200_ABSORB
  }
  const size_t smem = (size_t)(D + R) * sizeof(float);
  if (smem > 46 * 1024) return 3;
  B200_DISPATCH_DTYPE(dtype, launch_pdl(absorb_query_generic_kernel<T>, dim3((unsigned)T_, H), dim3(128), smem, st, (T*)out,
                                       (const T*)q, (const T*)w, w_head, (const float2*)table, H, D, R, C, rot_off, row, pairs));
  return (int)cudaGetLastError();
}

extern "C" int b200_expand_value(void* out, int64_t out_stride, const void* o, const void* w, int64_t w_head, const void* gate,
                                 int64_t gate_stride, int64_t T_, int H, int Dv, int C, int dtype, cudaStream_t st) {
  if (T_ == 0) return 0;
  if (H > 65535) return 2;
  if (dtype != kF32 && Dv == kD && C == kC && out_stride == (int64_t)H * kD && w_head % 8 == 0 &&
      ((uintptr_t)o | (uintptr_t)w | (uintptr_t)out) % 16 == 0 && T_ <= 64 * 65535) {
#define B200_EXPAND(MT)                                                                                              \
  return dtype == kBF16 ? launch_expand<__nv_bfloat16, MT>(out, o, w, w_head, gate, gate_stride, T_, H, st)           \
                        : launch_expand<__half, MT>(out, o, w, w_head, gate, gate_stride, T_, H, st)
    if (T_ <= 16) B200_EXPAND(1);
    if (T_ <= 32) B200_EXPAND(2);
    B200_EXPAND(4);
#undef B200_EXPAND
  }
  const size_t smem = (size_t)C * sizeof(float);
  if (smem > 46 * 1024) return 3;
  B200_DISPATCH_DTYPE(dtype, launch_pdl(expand_value_generic_kernel<T>, dim3((unsigned)T_, H), dim3(128), smem, st, (T*)out,
                                       out_stride, (const T*)o, (const T*)w, w_head, (const T*)gate, gate_stride, H, Dv, C));
  return (int)cudaGetLastError();
}

extern "C" int b200_gather_window(void* out, const void* cache, const int* block_tables, const int* seq_lens, const int* starts,
                                  const int* lens, int B, int max_len, int64_t max_blocks, int block_size, int64_t num_blocks,
                                  int64_t row_bytes, int64_t total, cudaStream_t st) {
  if (B == 0 || max_len <= 0) return 0;
  if (row_bytes % 16 || B > 65535) return 2;
  launch_pdl(gather_window_kernel, dim3((unsigned)((max_len + 7) / 8), B), dim3(256), 0, st, (uint4*)out, (const uint4*)cache,
             block_tables, seq_lens, starts, lens, max_blocks, block_size, num_blocks, (int)(row_bytes / 16), total);
  return (int)cudaGetLastError();
}
