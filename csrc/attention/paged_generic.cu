// Paged attention for any head size and for fp32 models: causal, optional sliding window (with first keys that stay visible),
// sinks, score bias by distance, output gates, sigmoid weights instead of a softmax; over keys and
// values [block][2][head][slot][D], or over latent rows [block][slot][D] that all heads share and whose first `latent_dv`
// columns are the values (absorbed multi-head latent attention).  The
// tensor-core kernels (prefill_umma.cu, decode_umma.cu, paged_attention.cu, paged_decode.cu) serve 16-bit heads of 64,
// 128 and 256; this one serves the rest on the CUDA cores, in fp32 throughout.
// One CTA = one (query token, query head).  Each of its 4 warps walks 32-key tiles of the visible range: scores with a
// lane per key, an online softmax (or plain sigmoids) per warp, then P.V with the lanes over the value dims; the warps' states meet at the
// end.
#include <math.h>

#include "../api.h"
#include "../common/launch.cuh"
#include "../common/utils.cuh"

namespace b200 {
namespace {

constexpr int kGenWarps = 4;

template <typename T, int ND>  // ND: value dims per lane, Dv <= 32 ND
__global__ void __launch_bounds__(kGenWarps * 32) paged_attention_generic_kernel(
    T* out, const T* q, const T* cache, const int* block_tables,
    const int* seq_lens, const int* qsl, const float* sinks, const float* bias, int bias_len, const T* gate,
    int64_t gate_stride, int B, int Hq, int Hkv, int D, int Dv, int latent, int block_size, int max_blocks, int64_t num_blocks, int window, int keep_first,
    int sigmoid, float scale) {
  extern __shared__ float sm_gen[];
  float* sq = sm_gen;                       // [D]
  float* so = sq + D;                       // [kGenWarps][Dv]
  float* sml = so + kGenWarps * Dv;         // [kGenWarps][2]
  griddep_launch();
  griddep_wait();
  const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  if (t < qsl[0] || t >= qsl[B]) return;
  int lo = 0, hi = B;
  while (hi - lo > 1) {
    const int mid = (lo + hi) >> 1;
    if (qsl[mid] <= t) lo = mid; else hi = mid;
  }
  const int req = lo, kvh = h / (Hq / Hkv);
  const int pos = seq_lens[req] - (qsl[req + 1] - t);
  if (pos < 0) return;
  const int first = window > 0 ? max(0, pos - window + 1) : 0;
  const int kept = min(keep_first, first), visible = kept + pos + 1 - first;   // kept keys, then the window
  for (int i = tid; i < D; i += kGenWarps * 32) sq[i] = to_f(q[((int64_t)t * Hq + h) * D + i]) * scale;
  __syncthreads();
  const int* bt = block_tables + (int64_t)req * max_blocks;
  const int64_t v_off = latent ? 0 : (int64_t)Hkv * block_size * D;
  auto row_of = [&](int key) -> int64_t {
    const int bi = key / block_size;
    const int64_t blk = bi < max_blocks ? bt[bi] : -1;
    if (blk < 0 || blk >= num_blocks) return -1;
    const int64_t page = latent ? blk : (blk * 2) * Hkv + kvh;
    return (page * block_size + key % block_size) * (int64_t)D;
  };
  float m = -INFINITY, l = 0.f, acc[ND];
#pragma unroll
  for (int i = 0; i < ND; ++i) acc[i] = 0.f;
  for (int k0 = warp * 32; k0 < visible; k0 += kGenWarps * 32) {
    const int i = k0 + lane, key = i < kept ? i : first + i - kept;
    const int64_t off = i < visible ? row_of(key) : -1;
    float s = -INFINITY;
    if (off >= 0) {
      const T* kr = cache + off;
      float a0 = 0.f, a1 = 0.f;
      int d = 0;
      for (; d + 1 < D; d += 2) { a0 += sq[d] * to_f(kr[d]); a1 += sq[d + 1] * to_f(kr[d + 1]); }
      if (d < D) a0 += sq[d] * to_f(kr[d]);
      s = a0 + a1;
      if (bias != nullptr) s += bias[(int64_t)h * bias_len + min(pos - key, bias_len - 1)];
    }
    float pr;
    if (sigmoid) {
      pr = off >= 0 ? 1.f / (1.f + expf(-s)) : 0.f;
      m = 0.f;
      l = 1.f;
    } else {
      const float mn = fmaxf(m, warp_max(s));
      if (mn == -INFINITY) continue;
      const float corr = expf(m - mn);
      pr = expf(s - mn);
      m = mn;
      l = l * corr + warp_sum(pr);
#pragma unroll
      for (int j = 0; j < ND; ++j) acc[j] *= corr;
    }
    for (int j = 0; j < 32; ++j) {
      const float pj = __shfl_sync(0xffffffff, pr, j);
      const int64_t oj = __shfl_sync(0xffffffff, off, j);
      if (oj < 0) continue;
      const T* vr = cache + oj + v_off;
#pragma unroll
      for (int i = 0; i < ND; ++i) {
        const int d = i * 32 + lane;
        if (d < Dv) acc[i] += pj * to_f(vr[d]);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < ND; ++i)
    if (i * 32 + lane < Dv) so[warp * Dv + i * 32 + lane] = acc[i];
  if (lane == 0) { sml[warp * 2] = m; sml[warp * 2 + 1] = l; }
  __syncthreads();
  float M = sinks != nullptr ? sinks[h] : -INFINITY;
#pragma unroll
  for (int w = 0; w < kGenWarps; ++w) M = fmaxf(M, sml[w * 2]);
  float den = sinks != nullptr ? expf(sinks[h] - M) : 0.f, wg[kGenWarps];
#pragma unroll
  for (int w = 0; w < kGenWarps; ++w) { wg[w] = expf(sml[w * 2] - M); den += sml[w * 2 + 1] * wg[w]; }
  float inv = sigmoid ? 1.f : den > 0.f ? 1.f / den : 0.f;
  if (gate != nullptr) inv /= 1.f + expf(-to_f(gate[(int64_t)t * gate_stride + h]));
  for (int d = tid; d < Dv; d += kGenWarps * 32) {
    float a = 0.f;
#pragma unroll
    for (int w = 0; w < kGenWarps; ++w) a += so[w * Dv + d] * wg[w];
    out[((int64_t)t * Hq + h) * Dv + d] = from_f<T>(a * inv);
  }
}

}  // namespace
}  // namespace b200

extern "C" int b200_paged_attention_generic(void* out, const void* q, const void* kv_cache, const int* block_tables,
                                            const int* seq_lens, const int* qsl, const float* sinks, int64_t T_, int B,
                                            int Hq, int Hkv, int D, int block_size, int max_blocks, int64_t num_blocks,
                                            int latent_dv, int window, float scale, const float* bias, int bias_len,
                                            const void* gate, int64_t gate_stride, int keep_first, int sigmoid, int dtype,
                                            cudaStream_t st) {
  using namespace b200;
  const int Dv = latent_dv > 0 ? latent_dv : D;
  if (B == 0 || T_ == 0) return 0;
  if (Hq % Hkv || Hq > 65535 || window < 0 || Dv > D || (latent_dv > 0 && Hkv != 1) ||
      (bias != nullptr && bias_len < 1) || keep_first < 0 || (sigmoid && sinks != nullptr))
    return 2;
  const size_t smem = (size_t)(D + kGenWarps * (Dv + 2)) * sizeof(float);
  if (smem > 48 * 1024) return 3;
  dim3 grid((unsigned)T_, Hq);
#define B200_GEN_ATTN(ND)                                                                                                \
  B200_DISPATCH_DTYPE(dtype, launch_pdl(paged_attention_generic_kernel<T, ND>, grid, dim3(kGenWarps * 32), smem, st,        \
                                       (T*)out, (const T*)q, (const T*)kv_cache, block_tables, seq_lens, qsl, sinks, bias,  \
                                       bias_len, (const T*)gate, gate_stride, B, Hq, Hkv, D, Dv, latent_dv > 0, block_size, max_blocks, num_blocks, window, keep_first, sigmoid, scale))
  if (Dv <= 64) { B200_GEN_ATTN(2); }
  else if (Dv <= 128) { B200_GEN_ATTN(4); }
  else if (Dv <= 256) { B200_GEN_ATTN(8); }
  else if (Dv <= 512) { B200_GEN_ATTN(16); }
  else if (Dv <= 1024) { B200_GEN_ATTN(32); }
  else return 3;
#undef B200_GEN_ATTN
  return (int)cudaGetLastError();
}
