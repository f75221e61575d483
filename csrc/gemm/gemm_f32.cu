// fp32 GEMM on the CUDA cores for models served in 32-bit: out[T, N] = x[T, K] . w[N, K]^T (+ bias[N]), true fp32
// products and sums (the tensor cores have no such format).  Any T, N, K and row strides.
//   few rows   one warp per output feature, the weight row streamed once for up to kRows tokens
//   many rows  64 x 64 output tile per CTA, 16-wide K slices through shared memory, 4 x 4 outputs per thread
//   grouped    rows sorted by expert, w[E, N, K], lod[e] .. lod[e + 1] the rows of expert e: the tile kernel, a tile per
//              (expert, 64 rows); the tiles are counted off on the device
// `relu2`: outputs pass the square of relu.
#include "../api.h"
#include "../common/launch.cuh"
#include "../common/utils.cuh"

namespace b200 {
namespace {

constexpr int kRows = 8;

__device__ __forceinline__ float result(float v, int relu2) {
  if (!relu2) return v;
  v = fmaxf(v, 0.f);
  return v * v;
}

__global__ void __launch_bounds__(256) gemm_f32_rows_kernel(float* out, int64_t ldo, const float* x,
                                                            int64_t ldx, const float* w, int64_t ldw,
                                                            const float* bias, int64_t T_, int N, int K, int relu2) {
  griddep_launch();
  griddep_wait();
  const int n = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  const int64_t t0 = (int64_t)blockIdx.y * kRows;
  if (n >= N) return;
  const float* wr = w + (int64_t)n * ldw;
  float acc[kRows];
#pragma unroll
  for (int i = 0; i < kRows; ++i) acc[i] = 0.f;
  for (int c = lane; c < K; c += 32) {
    const float wv = wr[c];
#pragma unroll
    for (int i = 0; i < kRows; ++i)
      if (t0 + i < T_) acc[i] += wv * x[(t0 + i) * ldx + c];
  }
#pragma unroll
  for (int i = 0; i < kRows; ++i) {
    const float s = warp_sum(acc[i]);
    if (lane == 0 && t0 + i < T_) out[(t0 + i) * ldo + n] = result(s + (bias ? bias[n] : 0.f), relu2);
  }
}

__device__ __forceinline__ void gemm_f32_tile(float* out, int64_t ldo, const float* x, int64_t ldx, const float* w,
                                              int64_t ldw, const float* bias, int64_t t0, int64_t T_, int N, int K, int relu2) {
  __shared__ __align__(16) float sx[16][68], sw[16][68];
  const int n0 = blockIdx.x * 64, tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += 16) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int e = i * 256 + threadIdx.x, c = e & 15, r = e >> 4;
      sx[c][r] = (t0 + r < T_ && k0 + c < K) ? x[(t0 + r) * ldx + k0 + c] : 0.f;
      sw[c][r] = (n0 + r < N && k0 + c < K) ? w[(int64_t)(n0 + r) * ldw + k0 + c] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < 16; ++c) {
      const float4 a = *reinterpret_cast<const float4*>(&sx[c][ty * 4]);
      const float4 b = *reinterpret_cast<const float4*>(&sw[c][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] += av[i] * bv[j];
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int64_t t = t0 + ty * 4 + i;
      const int n = n0 + tx * 4 + j;
      if (t < T_ && n < N) out[t * ldo + n] = result(acc[i][j] + (bias ? bias[n] : 0.f), relu2);
    }
}

__global__ void __launch_bounds__(256) gemm_f32_tile_kernel(float* out, int64_t ldo, const float* x,
                                                            int64_t ldx, const float* w, int64_t ldw,
                                                            const float* bias, int64_t T_, int N, int K, int relu2) {
  griddep_launch();
  griddep_wait();
  gemm_f32_tile(out, ldo, x, ldx, w, ldw, bias, (int64_t)blockIdx.y * 64, T_, N, K, relu2);
}

__global__ void __launch_bounds__(256) gemm_f32_grouped_kernel(float* out, int64_t ldo, const float* x, int64_t ldx,
                                                               const float* w, const int* lod, int E, int N, int K, int relu2) {
  griddep_launch();
  griddep_wait();
  int tile = blockIdx.y;
  for (int e = 0; e < E; ++e) {
    const int lo = lod[e], hi = lod[e + 1], tiles = (hi - lo + 63) / 64;
    if (tile < tiles) {
      gemm_f32_tile(out, ldo, x, ldx, w + (int64_t)e * N * K, K, nullptr, lo + (int64_t)tile * 64, hi, N, K, relu2);
      return;
    }
    tile -= tiles;
  }
}

}  // namespace
}  // namespace b200

extern "C" int b200_gemm_f32(float* out, int64_t ldo, const float* x, int64_t ldx, const float* w, int64_t ldw,
                             const float* bias, int64_t T_, int N, int K, int relu2, cudaStream_t st) {
  using namespace b200;
  if (T_ == 0 || N == 0) return 0;
  if (T_ <= 32) {
    launch_pdl(gemm_f32_rows_kernel, dim3((N + 7) / 8, (unsigned)((T_ + kRows - 1) / kRows)), dim3(256), 0, st, out, ldo, x,
               ldx, w, ldw, bias, T_, N, K, relu2);
  } else {
    const int64_t ty = (T_ + 63) / 64;
    if (ty > 65535) return 3;
    launch_pdl(gemm_f32_tile_kernel, dim3((N + 63) / 64, (unsigned)ty), dim3(256), 0, st, out, ldo, x, ldx, w, ldw, bias, T_,
               N, K, relu2);
  }
  return (int)cudaGetLastError();
}

// M rows of x in expert order; a grid of ceil(M / 64) + E row tiles covers any split of them over the experts
extern "C" int b200_gemm_f32_grouped(float* out, int64_t ldo, const float* x, int64_t ldx, const float* w, const int* lod,
                                     int64_t M, int E, int N, int K, int relu2, cudaStream_t st) {
  using namespace b200;
  if (M == 0 || N == 0) return 0;
  const int64_t ty = (M + 63) / 64 + E;
  if (ty > 65535) return 3;
  launch_pdl(gemm_f32_grouped_kernel, dim3((N + 63) / 64, (unsigned)ty), dim3(256), 0, st, out, ldo, x, ldx, w, lod, E, N, K, relu2);
  return (int)cudaGetLastError();
}
