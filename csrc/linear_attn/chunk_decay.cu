// Linear attention with a fixed decay per head, chunked form for prompt portions (16-bit models):
//
//   S_t = decay S_(t-1) + k_t v_t^T,  o_t = S_t^T q_t        (q, k, v = SiLU of the projections)
//
// For a chunk of 64 tokens that starts from state S (w = decay):
//   O[i] = w^(i+1) S^T q_i + sum_(j <= i) w^(i-j) (q_i . k_j) v_j
//   S'   = w^n S + sum_j w^(n-1-j) k_j v_j^T
// One CTA = (64 value channels of a head, request), 4 warps, chunks in order.  Warp r keeps S^T of its 16 value
// channels as fp32 MMA accumulators for the whole request: they are the A operand of S^T q without leaving registers.
// fp32 operands (state, decayed scores, decayed values) enter the 16-bit MMAs as a high and a low part, which keeps
// about 16 mantissa bits; accumulation is fp32.  q, k, v of the next chunk arrive by cp.async meanwhile.
#include "../api.h"
#include "../attention/attn_common.cuh"
#include "../common/launch.cuh"

namespace b200 {
namespace {

constexpr int kC = 64;    // tokens per chunk
constexpr int kVT = 64;   // value channels per CTA
constexpr int kThr = 128;

__device__ __forceinline__ float lo_bf16(uint32_t x) { return __uint_as_float(x << 16); }
__device__ __forceinline__ float hi_bf16(uint32_t x) { return __uint_as_float(x & 0xffff0000u); }
// (a, b) -> packed bf16 high parts and packed bf16 remainders
__device__ __forceinline__ void split2(float a, float b, uint32_t& h, uint32_t& l) {
  h = MmaTraits<__nv_bfloat16>::pack(a, b);
  l = MmaTraits<__nv_bfloat16>::pack(a - lo_bf16(h), b - hi_bf16(h));
}
__device__ __forceinline__ uint32_t silu2(uint32_t x) {
  const float a = lo_bf16(x), b = hi_bf16(x);
  return MmaTraits<__nv_bfloat16>::pack(__fdividef(a, 1.f + __expf(-a)), __fdividef(b, 1.f + __expf(-b)));
}

template <int DK>
struct ChunkSmem {
  static constexpr int kQ = kC * DK, kV = kC * kVT, kStage = 2 * kQ + kV;                 // elements
  static constexpr size_t kBytes = (2 * kStage + 2 * kC * kC) * sizeof(__nv_bfloat16) + (kC + 1) * sizeof(float) + 12;
};

template <int DK>
__global__ void __launch_bounds__(kThr, 2) chunk_decay_kernel(const RecurrenceArgs p) {
  using T = __nv_bfloat16;
  using MT = MmaTraits<T>;
  using L_ = ChunkSmem<DK>;
  constexpr int NT = DK / 8, CH = DK / 8;
  extern __shared__ __align__(128) uint8_t smem_cd[];
  T* stage0 = reinterpret_cast<T*>(smem_cd);
  T* sPh = stage0 + 2 * L_::kStage;
  T* sPl = sPh + kC * kC;
  float* lam = reinterpret_cast<float*>(sPl + kC * kC);  // [kC + 1] powers of the decay
  griddep_launch();
  griddep_wait();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t2 = (lane & 3) * 2;
  const int h = blockIdx.y, r = blockIdx.z, v0 = blockIdx.x * kVT;
  const int s = p.cu[r], L = p.cu[r + 1] - s, slot = p.slots[r];
  if (L <= 0 || slot < 0) return;
  const T* gq = reinterpret_cast<const T*>(p.q) + h * p.Dk;
  const T* gk = reinterpret_cast<const T*>(p.k) + h * p.Dk;
  const T* gv = reinterpret_cast<const T*>(p.v) + h * p.Dv + v0;

  auto load = [&](int c0, int st) {
    T* sQ = stage0 + st * L_::kStage;
    T* sK = sQ + L_::kQ;
    T* sV = sK + L_::kQ;
    for (int c = tid; c < kC * CH; c += kThr) {
      const int row = c / CH, ch = c % CH;
      const bool ok = c0 + row < L && ch * 8 < p.Dk;
      const int64_t off = ok ? (int64_t)(s + c0 + row) * p.qkv_stride + ch * 8 : 0;
      cp_async16(sQ + swz<DK>(row, ch), gq + off, ok);
      cp_async16(sK + swz<DK>(row, ch), gk + off, ok);
    }
    for (int c = tid; c < kC * (kVT / 8); c += kThr) {
      const int row = c / (kVT / 8), ch = c % (kVT / 8);
      const bool ok = c0 + row < L && v0 + ch * 8 < p.Dv;
      cp_async16(sV + swz<kVT>(row, ch), gv + (ok ? (int64_t)(s + c0 + row) * p.qkv_stride + ch * 8 : 0), ok);
    }
    cp_async_commit();
  };
  load(0, 0);
  if (tid <= kC) lam[tid] = powf(p.decay[h], (float)tid);

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

  for (int c0 = 0, it = 0; c0 < L; c0 += kC, ++it) {
    T* sQ = stage0 + (it & 1) * L_::kStage;
    T* sK = sQ + L_::kQ;
    T* sV = sK + L_::kQ;
    const int n = min(kC, L - c0);
    cp_async_wait<0>();
    __syncthreads();  // this chunk has arrived; everyone is done with the other stage and with P
    if (c0 + kC < L) load(c0 + kC, (it + 1) & 1);
    for (int c = tid; c < L_::kStage / 8; c += kThr) {
      uint4* x = reinterpret_cast<uint4*>(sQ) + c;
      uint4 y = *x;
      y.x = silu2(y.x); y.y = silu2(y.y); y.z = silu2(y.z); y.w = silu2(y.w);
      *x = y;
    }
    __syncthreads();
    // ---- P[i][j] = w^(i-j) q_i . k_j for this warp's 16 queries, key tiles up to the diagonal
    {
      float acc[8][4];
#pragma unroll
      for (int i = 0; i < 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
      for (int ks = 0; ks < DK / 16; ++ks) {
        uint32_t a[4];
        ldmatrix_x4(a, sQ + swz<DK>(warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, ks * 2 + (lane >> 4)));
#pragma unroll
        for (int np = 0; np < 4; ++np) {
          if (np > warp) break;
          uint32_t b[4];
          ldmatrix_x4(b, sK + swz<DK>(np * 16 + (lane & 7) + (lane >> 4) * 8, ks * 2 + ((lane >> 3) & 1)));
          MT::mma(acc[2 * np], a, b[0], b[1]);
          MT::mma(acc[2 * np + 1], a, b[2], b[3]);
        }
      }
#pragma unroll
      for (int nt = 0; nt < 8; ++nt) {
        if (nt > 2 * warp + 1) break;
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int i = warp * 16 + g + half * 8, j = nt * 8 + t2;
          const float x = j <= i ? acc[nt][half * 2] * lam[i - j] : 0.f;
          const float y = j + 1 <= i ? acc[nt][half * 2 + 1] * lam[i - j - 1] : 0.f;
          uint32_t hi, lo;
          split2(x, y, hi, lo);
          *reinterpret_cast<uint32_t*>(sPh + swz<kC>(i, nt) + t2) = hi;
          *reinterpret_cast<uint32_t*>(sPl + swz<kC>(i, nt) + t2) = lo;
        }
      }
    }
    __syncthreads();
    // ---- O^T (16 value channels x 64 tokens of this warp): state part, then the chunk's own tokens
    float acc[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
    for (int ks = 0; ks < DK / 16; ++ks) {
      uint32_t ah[4], al[4];
      split2(S[2 * ks][0], S[2 * ks][1], ah[0], al[0]);
      split2(S[2 * ks][2], S[2 * ks][3], ah[1], al[1]);
      split2(S[2 * ks + 1][0], S[2 * ks + 1][1], ah[2], al[2]);
      split2(S[2 * ks + 1][2], S[2 * ks + 1][3], ah[3], al[3]);
#pragma unroll
      for (int np = 0; np < 4; ++np) {
        uint32_t b[4];
        ldmatrix_x4(b, sQ + swz<DK>(np * 16 + (lane & 7) + (lane >> 4) * 8, ks * 2 + ((lane >> 3) & 1)));
        MT::mma(acc[2 * np], ah, b[0], b[1]);
        MT::mma(acc[2 * np + 1], ah, b[2], b[3]);
        MT::mma(acc[2 * np], al, b[0], b[1]);
        MT::mma(acc[2 * np + 1], al, b[2], b[3]);
      }
    }
#pragma unroll
    for (int nt = 0; nt < 8; ++nt) {
      const float w0 = lam[nt * 8 + t2 + 1], w1 = lam[nt * 8 + t2 + 2 > kC ? kC : nt * 8 + t2 + 2];
      acc[nt][0] *= w0; acc[nt][1] *= w1; acc[nt][2] *= w0; acc[nt][3] *= w1;
    }
    const float wn = lam[n];
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) { S[nt][0] *= wn; S[nt][1] *= wn; S[nt][2] *= wn; S[nt][3] *= wn; }
#pragma unroll
    for (int kt = 0; kt < kC / 16; ++kt) {
      if (kt * 16 >= n) break;
      uint32_t a[4], ah[4], al[4];
      ldmatrix_x4_trans(a, sV + swz<kVT>(kt * 16 + (lane & 7) + (lane >> 4) * 8, warp * 2 + ((lane >> 3) & 1)));
#pragma unroll
      for (int np = 0; np < 4; ++np) {
        if (np < kt) continue;
        uint32_t b[4], c[4];
        const int off = swz<kC>(np * 16 + (lane & 7) + (lane >> 4) * 8, kt * 2 + ((lane >> 3) & 1));
        ldmatrix_x4(b, sPh + off);
        ldmatrix_x4(c, sPl + off);
        MT::mma(acc[2 * np], a, b[0], b[1]);
        MT::mma(acc[2 * np + 1], a, b[2], b[3]);
        MT::mma(acc[2 * np], a, c[0], c[1]);
        MT::mma(acc[2 * np + 1], a, c[2], c[3]);
      }
      // S^T += (V^T w^(n-1-j)) K
      const int j = kt * 16 + t2;
      const float f0 = lam[max(0, n - 1 - j)], f1 = lam[max(0, n - 2 - j)], f8 = lam[max(0, n - 9 - j)],
                  f9 = lam[max(0, n - 10 - j)];
      split2(lo_bf16(a[0]) * f0, hi_bf16(a[0]) * f1, ah[0], al[0]);
      split2(lo_bf16(a[1]) * f0, hi_bf16(a[1]) * f1, ah[1], al[1]);
      split2(lo_bf16(a[2]) * f8, hi_bf16(a[2]) * f9, ah[2], al[2]);
      split2(lo_bf16(a[3]) * f8, hi_bf16(a[3]) * f9, ah[3], al[3]);
#pragma unroll
      for (int dp = 0; dp < NT / 2; ++dp) {
        uint32_t b[4];
        ldmatrix_x4_trans(b, sK + swz<DK>(kt * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, dp * 2 + (lane >> 4)));
        MT::mma(S[2 * dp], ah, b[0], b[1]);
        MT::mma(S[2 * dp + 1], ah, b[2], b[3]);
        MT::mma(S[2 * dp], al, b[0], b[1]);
        MT::mma(S[2 * dp + 1], al, b[2], b[3]);
      }
    }
    float* out = p.out + (int64_t)(s + c0) * p.out_stride + h * p.Dv;
#pragma unroll
    for (int nt = 0; nt < 8; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int tok = nt * 8 + t2 + (e & 1), v = e < 2 ? va : vb;
        if (tok < n && v < p.Dv) out[(int64_t)tok * p.out_stride + v] = acc[nt][e];
      }
  }
#pragma unroll
  for (int nt = 0; nt < NT; ++nt) {
    const int d = nt * 8 + t2;
    if (d >= p.Dks) continue;
    if (va < p.Dv) *reinterpret_cast<float2*>(sp + (int64_t)va * p.Dks + d) = make_float2(S[nt][0], S[nt][1]);
    if (vb < p.Dv) *reinterpret_cast<float2*>(sp + (int64_t)vb * p.Dks + d) = make_float2(S[nt][2], S[nt][3]);
  }
}

template <int DK>
int launch_chunk(const RecurrenceArgs& a, cudaStream_t st) {
  auto kern = chunk_decay_kernel<DK>;
  constexpr int smem = (int)ChunkSmem<DK>::kBytes;
  cudaError_t e = ensure_dynamic_smem((const void*)kern, smem);
  if (e != cudaSuccess) return (int)e;
  launch_pdl(kern, dim3((a.Dv + kVT - 1) / kVT, a.H, a.R), dim3(kThr), smem, st, a);
  return (int)cudaGetLastError();
}

}  // namespace
}  // namespace b200

// Prompt portions (kind 1, bf16): head sizes up to 128 that are multiples of 8, 16-byte aligned rows.
extern "C" int b200_chunk_decay(const RecurrenceArgs* a, int dtype, cudaStream_t st) {
  if (a->R == 0) return 0;
  const uintptr_t al = (uintptr_t)a->q | (uintptr_t)a->k | (uintptr_t)a->v;
  if (dtype != b200::kBF16 || a->kind != 1 || a->H != a->Hk || a->Dk % 8 || a->Dv % 8 || a->Dk > 128 || a->qkv_stride % 8 ||
      al % 16 || a->Dks % 4 || a->Dks < a->Dk || a->R > 65535 || a->H > 65535)
    return 3;
  return a->Dk <= 64 ? b200::launch_chunk<64>(*a, st) : b200::launch_chunk<128>(*a, st);
}
