// Linear attention whose forget gate also decides what is written, chunked form for prompt portions (16-bit models):
//
//   S_t = diag(f_t) S_(t-1) + (1 - f_t) v_t^T,  o_t = S_t^T q_t        f_t = l + (1 - l) sigmoid(x_t + bias),  q = SiLU
//
// For a chunk of 16 tokens that starts from state S (k = 1 - f; products of gates per key channel d):
//   O[i] = sum_d q_i[d] (f_0 .. f_i)[d] S[d]  +  sum_(j <= i) A[i][j] v_j,   A[i][j] = sum_d q_i[d] k_j[d] (f_(j+1) .. f_i)[d]
//   S'   = diag(f_0 .. f_15) S + sum_j (k_j (f_(j+1) .. f_15)) v_j^T
// Every product of gates is formed by multiplication in fp32 (no logarithms, no quotients), so gates of any size are safe.
// One CTA = (16 NW value channels of a head, request), NW warps, chunks in order.  Warp r keeps S^T of its 16 value channels
// as fp32 MMA accumulators for the whole request: they are the A operand of S^T q without leaving registers.  fp32 operands
// (state, scores A, decayed writes) enter the 16-bit MMAs as a high and a low part, which keeps about 16 mantissa bits;
// accumulation is fp32.  The raw projections of the next chunk wait in registers meanwhile.
#include "../api.h"
#include "../attention/attn_common.cuh"
#include "../common/launch.cuh"

namespace b200 {
namespace {

constexpr int kCT = 16;   // tokens per chunk

__device__ __forceinline__ float lo_bf16(uint32_t x) { return __uint_as_float(x << 16); }
__device__ __forceinline__ float hi_bf16(uint32_t x) { return __uint_as_float(x & 0xffff0000u); }
// (a, b) -> packed bf16 high parts and packed bf16 remainders
__device__ __forceinline__ void split2(float a, float b, uint32_t& h, uint32_t& l) {
  h = MmaTraits<__nv_bfloat16>::pack(a, b);
  l = MmaTraits<__nv_bfloat16>::pack(a - lo_bf16(h), b - hi_bf16(h));
}

template <int DK, int NW>
struct GatedSmem {
  static constexpr int kVT = NW * 16;
  float q[kCT][DK], f[kCT][DK], k[kCT][DK];              // SiLU(q), forget gate, written share
  float decay[DK];                                       // product of the chunk's gates
  __nv_bfloat16 qd[kCT * DK];                            // q_i (f_0 .. f_i), swizzled rows
  __nv_bfloat16 kh[kCT * DK], kl[kCT * DK];              // k_j (f_(j+1) .. f_15), high and low part
  __nv_bfloat16 v[kCT * kVT];
  __nv_bfloat16 ah[kCT * 16], al[kCT * 16];              // A, rows of 16 (two 16-byte chunks, swapped by row parity)
};

// 16-byte chunk `chunk` (0, 1) of row `row` of a [16][16] 16-bit tile
__device__ __forceinline__ int swz16(int row, int chunk) { return row * 16 + ((chunk ^ ((row >> 2) & 1)) << 3); }

template <int DK, int NW>
__global__ void __launch_bounds__(NW * 32) chunk_gated_kernel(const RecurrenceArgs p) {
  using T = __nv_bfloat16;
  using MT = MmaTraits<T>;
  using Sm = GatedSmem<DK, NW>;
  constexpr int kThr = NW * 32, kVT = Sm::kVT, NT = DK / 8;
  constexpr int QV = kCT * DK / 8, VV = kCT * kVT / 8;                   // 16-byte vectors of a chunk
  constexpr int QPER = (QV + kThr - 1) / kThr, VPER = (VV + kThr - 1) / kThr;
  constexpr int SL = kThr / 16;                                          // threads that share a row of A (32 / SL <= lanes)
  static_assert(SL == 8 || SL == 16, "slices of a score row stay inside a warp");
  static_assert(DK % (4 * SL) == 0, "score slices");
  extern __shared__ __align__(128) uint8_t smem_cg[];
  Sm& sm = *reinterpret_cast<Sm*>(smem_cg);
  griddep_launch();
  griddep_wait();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t2 = (lane & 3) * 2;
  const int h = blockIdx.y, r = blockIdx.z, v0 = blockIdx.x * kVT;
  const int s = p.cu[r], L = p.cu[r + 1] - s, slot = p.slots[r];
  if (L <= 0 || slot < 0) return;
  const T* gq = reinterpret_cast<const T*>(p.q) + h * p.Dk;
  const T* ga = reinterpret_cast<const T*>(p.a) + h * p.Dk;
  const T* gv = reinterpret_cast<const T*>(p.v) + h * p.Dv + v0;
  const float* bias = p.dt_bias + h * p.Dk;
  const float* lower = p.lower + h * p.Dk;

  // S[nt][e]: value channel 16 warp + g (+ 8 for e >= 2), key channel 8 nt + t2 + (e & 1)
  float S[NT][4];
  const int va = v0 + warp * 16 + g, vb = va + 8;
  float* sp = p.states + ((int64_t)slot * p.H + h) * p.Dv * p.Dks;
  const bool init = p.has_init[r] != 0;
#pragma unroll
  for (int nt = 0; nt < NT; ++nt) {
    const int d = nt * 8 + t2;
    float2 a = make_float2(0.f, 0.f), b = a;
    if (init && d < p.Dks) {
      if (va < p.Dv) a = *reinterpret_cast<const float2*>(sp + (int64_t)va * p.Dks + d);
      if (vb < p.Dv) b = *reinterpret_cast<const float2*>(sp + (int64_t)vb * p.Dks + d);
    }
    S[nt][0] = a.x; S[nt][1] = a.y; S[nt][2] = b.x; S[nt][3] = b.y;
  }

  uint4 rq[QPER], ra[QPER], rv[VPER];
  const uint4 zero = make_uint4(0, 0, 0, 0);
  auto fetch = [&](int c0) {
#pragma unroll
    for (int i = 0; i < QPER; ++i) {
      const int c = i * kThr + tid, row = c / (DK / 8), ch = c % (DK / 8);
      const bool ok = c < QV && c0 + row < L && ch * 8 < p.Dk;
      rq[i] = ok ? *reinterpret_cast<const uint4*>(gq + (int64_t)(s + c0 + row) * p.qkv_stride + ch * 8) : zero;
      ra[i] = ok ? *reinterpret_cast<const uint4*>(ga + (int64_t)(s + c0 + row) * p.a_stride + ch * 8) : zero;
    }
#pragma unroll
    for (int i = 0; i < VPER; ++i) {
      const int c = i * kThr + tid, row = c / (kVT / 8), ch = c % (kVT / 8);
      const bool ok = c < VV && c0 + row < L && v0 + ch * 8 < p.Dv;
      rv[i] = ok ? *reinterpret_cast<const uint4*>(gv + (int64_t)(s + c0 + row) * p.qkv_stride + ch * 8) : zero;
    }
  };
  fetch(0);

  for (int c0 = 0; c0 < L; c0 += kCT) {
    const int n = min(kCT, L - c0);
    // ---- gates and SiLU in fp32.  Rows past the end: f = 1, k = 0 (the state stays as it is); padding channels: zeros
#pragma unroll
    for (int i = 0; i < QPER; ++i) {
      const int c = i * kThr + tid, row = c / (DK / 8), d0 = (c % (DK / 8)) * 8;
      if (c >= QV) continue;
      const uint32_t qw[4] = {rq[i].x, rq[i].y, rq[i].z, rq[i].w}, aw[4] = {ra[i].x, ra[i].y, ra[i].z, ra[i].w};
      float fq[8], ff[8], fk[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const float qv = (e & 1) ? hi_bf16(qw[e >> 1]) : lo_bf16(qw[e >> 1]);
        const float av = (e & 1) ? hi_bf16(aw[e >> 1]) : lo_bf16(aw[e >> 1]);
        fq[e] = __fdividef(qv, 1.f + __expf(-qv));
        ff[e] = row < n ? 0.f : 1.f;
        fk[e] = 0.f;
        if (row < n && d0 + e < p.Dk) {
          const float z = av + bias[d0 + e], low = lower[d0 + e];
          const float x = __expf(-fabsf(z)), big = __fdividef(1.f, 1.f + x), small = x * big;
          ff[e] = low + (1.f - low) * (z >= 0.f ? big : small);
          fk[e] = (1.f - low) * (z >= 0.f ? small : big);
        }
      }
#pragma unroll
      for (int e = 0; e < 8; e += 4) {
        *reinterpret_cast<float4*>(&sm.q[row][d0 + e]) = make_float4(fq[e], fq[e + 1], fq[e + 2], fq[e + 3]);
        *reinterpret_cast<float4*>(&sm.f[row][d0 + e]) = make_float4(ff[e], ff[e + 1], ff[e + 2], ff[e + 3]);
        *reinterpret_cast<float4*>(&sm.k[row][d0 + e]) = make_float4(fk[e], fk[e + 1], fk[e + 2], fk[e + 3]);
      }
    }
#pragma unroll
    for (int i = 0; i < VPER; ++i) {
      const int c = i * kThr + tid, row = c / (kVT / 8), ch = c % (kVT / 8);
      if (c < VV) *reinterpret_cast<uint4*>(sm.v + swz<kVT>(row, ch)) = rv[i];
    }
    __syncthreads();
    if (c0 + kCT < L) fetch(c0 + kCT);
    // ---- products of gates: forwards for the queries, backwards for the writes (two adjacent channels per thread; the
    // first half of the threads takes the queries, the second half the writes)
    {
      constexpr int HALF = kThr / 2;
      const bool fwd = tid < HALF;
      for (int d = (tid % HALF) * 2; d < DK; d += 2 * HALF) {
        float px = 1.f, py = 1.f;
        if (fwd) {
#pragma unroll
          for (int i = 0; i < kCT; ++i) {
            const float2 f = *reinterpret_cast<const float2*>(&sm.f[i][d]);
            const float2 q = *reinterpret_cast<const float2*>(&sm.q[i][d]);
            px *= f.x;
            py *= f.y;
            *reinterpret_cast<uint32_t*>(sm.qd + swz<DK>(i, d >> 3) + (d & 7)) = MT::pack(q.x * px, q.y * py);
          }
          *reinterpret_cast<float2*>(&sm.decay[d]) = make_float2(px, py);
        } else {
#pragma unroll
          for (int i = kCT - 1; i >= 0; --i) {
            const float2 f = *reinterpret_cast<const float2*>(&sm.f[i][d]);
            const float2 k = *reinterpret_cast<const float2*>(&sm.k[i][d]);
            uint32_t hi, lo;
            split2(k.x * px, k.y * py, hi, lo);
            *reinterpret_cast<uint32_t*>(sm.kh + swz<DK>(i, d >> 3) + (d & 7)) = hi;
            *reinterpret_cast<uint32_t*>(sm.kl + swz<DK>(i, d >> 3) + (d & 7)) = lo;
            px *= f.x;
            py *= f.y;
          }
        }
      }
    }
    // ---- A[i][j]: SL neighbouring threads share column j; each carries k_j (f_(j+1) .. f_i) of its channels along i
    {
      constexpr int W = DK / SL;
      const int j = tid / SL, sl = tid % SL;
      float w[W];
#pragma unroll
      for (int c = 0; c < W; c += 4) {
        const float4 k = *reinterpret_cast<const float4*>(&sm.k[j][(c / 4 * SL + sl) * 4]);
        w[c] = k.x; w[c + 1] = k.y; w[c + 2] = k.z; w[c + 3] = k.w;
      }
      const int jlo = (tid & ~31) / SL;       // first column of this warp
      for (int i = 0; i < kCT; ++i) {
        float a = 0.f;
        if (i >= jlo) {                        // warp-uniform
          float b = 0.f;
#pragma unroll
          for (int c = 0; c < W; c += 4) {
            const int d = (c / 4 * SL + sl) * 4;
            if (i > j) {
              const float4 f = *reinterpret_cast<const float4*>(&sm.f[i][d]);
              w[c] *= f.x; w[c + 1] *= f.y; w[c + 2] *= f.z; w[c + 3] *= f.w;
            }
            const float4 q = *reinterpret_cast<const float4*>(&sm.q[i][d]);
            a += q.x * w[c] + q.y * w[c + 1];
            b += q.z * w[c + 2] + q.w * w[c + 3];
          }
          a += b;
#pragma unroll
          for (int m = 1; m < SL; m <<= 1) a += __shfl_xor_sync(0xffffffff, a, m);
        }
        if (sl == 0) {
          a = i >= j ? a : 0.f;
          const T hi = __float2bfloat16(a);
          sm.ah[swz16(i, j >> 3) + (j & 7)] = hi;
          sm.al[swz16(i, j >> 3) + (j & 7)] = __float2bfloat16(a - __bfloat162float(hi));
        }
      }
    }
    __syncthreads();
    // ---- O^T (16 value channels x 16 tokens of this warp): state part, then the chunk's own tokens
    float acc[2][4] = {};
    float acl[2][4] = {};
#pragma unroll
    for (int ks = 0; ks < DK / 16; ++ks) {
      uint32_t ah[4], al[4], b[4];
      split2(S[2 * ks][0], S[2 * ks][1], ah[0], al[0]);
      split2(S[2 * ks][2], S[2 * ks][3], ah[1], al[1]);
      split2(S[2 * ks + 1][0], S[2 * ks + 1][1], ah[2], al[2]);
      split2(S[2 * ks + 1][2], S[2 * ks + 1][3], ah[3], al[3]);
      ldmatrix_x4(b, sm.qd + swz<DK>((lane & 7) + (lane >> 4) * 8, ks * 2 + ((lane >> 3) & 1)));
      MT::mma(acc[0], ah, b[0], b[1]);
      MT::mma(acc[1], ah, b[2], b[3]);
      MT::mma(acl[0], al, b[0], b[1]);
      MT::mma(acl[1], al, b[2], b[3]);
    }
    uint32_t a[4];      // V^T: this warp's value channels x the chunk's tokens
    ldmatrix_x4_trans(a, sm.v + swz<kVT>((lane & 7) + (lane >> 4) * 8, warp * 2 + ((lane >> 3) & 1)));
    {
      uint32_t b[4], c[4];
      const int off = swz16((lane & 7) + (lane >> 4) * 8, (lane >> 3) & 1);
      ldmatrix_x4(b, sm.ah + off);
      ldmatrix_x4(c, sm.al + off);
      MT::mma(acc[0], a, b[0], b[1]);
      MT::mma(acc[1], a, b[2], b[3]);
      MT::mma(acl[0], a, c[0], c[1]);
      MT::mma(acl[1], a, c[2], c[3]);
    }
    // ---- S^T <- S^T diag(decay) + V^T (decayed writes)
#pragma unroll
    for (int dp = 0; dp < NT / 2; ++dp) {
      const float2 w0 = *reinterpret_cast<const float2*>(&sm.decay[dp * 16 + t2]);
      const float2 w1 = *reinterpret_cast<const float2*>(&sm.decay[dp * 16 + 8 + t2]);
      S[2 * dp][0] *= w0.x; S[2 * dp][1] *= w0.y; S[2 * dp][2] *= w0.x; S[2 * dp][3] *= w0.y;
      S[2 * dp + 1][0] *= w1.x; S[2 * dp + 1][1] *= w1.y; S[2 * dp + 1][2] *= w1.x; S[2 * dp + 1][3] *= w1.y;
      uint32_t b[4], c[4];
      const int off = swz<DK>((lane & 7) + ((lane >> 3) & 1) * 8, dp * 2 + (lane >> 4));
      ldmatrix_x4_trans(b, sm.kh + off);
      ldmatrix_x4_trans(c, sm.kl + off);
      MT::mma(S[2 * dp], a, b[0], b[1]);
      MT::mma(S[2 * dp + 1], a, b[2], b[3]);
      MT::mma(S[2 * dp], a, c[0], c[1]);
      MT::mma(S[2 * dp + 1], a, c[2], c[3]);
    }
    float* out = p.out + (int64_t)(s + c0) * p.out_stride + h * p.Dv;
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int tok = nt * 8 + t2 + (e & 1), v = e < 2 ? va : vb;
        if (tok < n && v < p.Dv) out[(int64_t)tok * p.out_stride + v] = acc[nt][e] + acl[nt][e];
      }
    __syncthreads();   // everyone has read this chunk before the next one overwrites it
  }
#pragma unroll
  for (int nt = 0; nt < NT; ++nt) {
    const int d = nt * 8 + t2;
    if (d >= p.Dks) continue;
    if (va < p.Dv) *reinterpret_cast<float2*>(sp + (int64_t)va * p.Dks + d) = make_float2(S[nt][0], S[nt][1]);
    if (vb < p.Dv) *reinterpret_cast<float2*>(sp + (int64_t)vb * p.Dks + d) = make_float2(S[nt][2], S[nt][3]);
  }
}

template <int DK, int NW>
int launch_gated(const RecurrenceArgs& a, cudaStream_t st) {
  auto kern = chunk_gated_kernel<DK, NW>;
  constexpr int smem = (int)sizeof(GatedSmem<DK, NW>);
  cudaError_t e = ensure_dynamic_smem((const void*)kern, smem);
  if (e != cudaSuccess) return (int)e;
  launch_pdl(kern, dim3((a.Dv + NW * 16 - 1) / (NW * 16), a.H, a.R), dim3(NW * 32), smem, st, a);
  return (int)cudaGetLastError();
}

}  // namespace
}  // namespace b200

// Prompt portions (kind 2, bf16): head sizes up to 128 that are multiples of 8, 16-byte aligned rows.
extern "C" int b200_chunk_gated_write(const RecurrenceArgs* a, int dtype, cudaStream_t st) {
  if (a->R == 0) return 0;
  const uintptr_t al = (uintptr_t)a->q | (uintptr_t)a->v | (uintptr_t)a->a;
  if (dtype != b200::kBF16 || a->kind != 2 || a->H != a->Hk || a->Dk % 8 || a->Dv % 8 || a->Dk > 128 || a->qkv_stride % 8 ||
      a->a_stride % 8 || al % 16 || a->Dks % 4 || a->Dks < a->Dk || a->R > 65535 || a->H > 65535)
    return 3;
  // eight warps share a chunk's gates and scores between 128 value channels; few heads and requests are spread thinner
  const bool wide = a->Dv > 64 && (int64_t)a->R * a->H * ((a->Dv + 127) / 128) >= 100;
  if (a->Dk <= 64) return wide ? b200::launch_gated<64, 8>(*a, st) : b200::launch_gated<64, 4>(*a, st);
  return wide ? b200::launch_gated<128, 8>(*a, st) : b200::launch_gated<128, 4>(*a, st);
}
