// The gated delta rule with ONE decay per token and head,
//
//   S <- g_t S;   u_t = beta_t (v_t - S^T k_t);   S <- S + k_t u_t^T;   o_t = S^T q_t          (q, k unit vectors, q times q_scale)
//
// for bf16 prompt portions in chunks of 64 tokens on the tensor cores, and for steps of one token per sequence.
//
// Chunks.  With l_t the running sum of log decays inside a chunk and S the fp32 state at its start, the writes solve a unit lower
// triangular system, (1 + A) U = diag(beta) (V - diag(e^l) K S) with A_ts = beta_t e^(l_t - l_s) k_t.k_s for s < t, and
//
//   o_t = e^(l_t) S^T q_t + sum_(s <= t) e^(l_t - l_s) (k_s . q_t) u_s,      S <- e^(l_64) S + sum_s e^(l_64 - l_s) k_s u_s^T.
//
// delta_prepare_kernel inverts 1 + A for every (chunk, head) of a step at once - the inverse does not depend on the state - and
// leaves M = (1 + A)^-1 diag(beta) with the tokens' scalars in a workspace; delta_chunk_scan_kernel then walks the chunks of a
// (sequence, head, block of value columns) in order.
//
// Precision.  q and k enter the products as the bf16 numbers the convolution left, their unit-norm factors stay with the fp32
// scalars; every fp32 operand (state, M, V - ..., U, the pair weights) is split into two bf16 numbers (relative remainder 2^-17)
// and multiplied part by part with fp32 accumulation.  The state stays fp32 in accumulator registers for the whole portion.
// Running sums of logs are formed in double and kept as two floats; every exponent is a difference <= 0.
#include <algorithm>
#include <type_traits>

#include "../../include/b200_mixers.h"
#include "b200_common.cuh"

namespace b200 {
namespace {

constexpr int kChunk = 64;
constexpr int kMld = kChunk + 8;           // row length of M in shared memory
constexpr float kLogFloor = -200.0f;       // e^-200 is 0 in fp32: slower forgetting is kept exactly, faster is "everything"

struct DeltaSeq {
  int tok0, count, slot, fresh;
};

// Workspace of one (chunk, head): M as two bf16 matrices, then per token (l high, l low, 1/|k|, q_scale/|q|).
constexpr size_t kWsMat = sizeof(__nv_bfloat16) * kChunk * kChunk;
constexpr size_t kWsBytes = 2 * kWsMat + sizeof(float4) * kChunk;

struct DeltaChunkArgs {
  float* o;
  const __nv_bfloat16* q;
  const __nv_bfloat16* k;
  const __nv_bfloat16* v;
  int64_t stride;
  const __nv_bfloat16* beta;
  int64_t beta_stride;
  const __nv_bfloat16* a;
  int64_t a_stride;
  const __nv_bfloat16* dt_bias;
  const __nv_bfloat16* a_log;
  float* state;
  const DeltaSeq* seqs;
  int H, G, dk, dv;
  float unit_eps, q_scale;
  unsigned char* ws;
  int vec;                                 // rows of q, k and v may be copied in 16-byte pieces
};

// first chunk of a sequence: unique for any packing in row order, since a sequence of n tokens has at most n / 64 + 1 chunks
__device__ __forceinline__ int64_t first_chunk(const DeltaSeq& sq, int seq) { return sq.tok0 / kChunk + seq; }

__device__ __forceinline__ uint32_t smem_at(const void* p) { return static_cast<uint32_t>(__cvta_generic_to_shared(p)); }
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void copy16(void* dst, const void* src, bool valid) {
  const int bytes = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_at(dst)), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - f.x, y - f.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ float sigm(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float softp(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// ---- M and the scalars of every chunk ----------------------------------------------------------------------------------
// One CTA of four warps per (chunk, head, sequence).  1 + A in 32 x 32 blocks: the two diagonal blocks are inverted by forward
// substitution (one column per lane, two warps), the block below is -T22 (A21 T11).
constexpr int kALd = 68;

template <int DKP>
__global__ void __launch_bounds__(128)
delta_prepare_kernel(const DeltaChunkArgs A) {
  constexpr int LDK = DKP + 8;
  extern __shared__ __align__(16) unsigned char dp_raw[];
  __nv_bfloat16* k_s = reinterpret_cast<__nv_bfloat16*>(dp_raw);
  float* a_s = reinterpret_cast<float*>(k_s + kChunk * LDK);      // A [64][kALd]
  float* t_s = a_s + kChunk * kALd;                               // inverse [64][kALd]
  float* m_s = t_s + kChunk * kALd;                               // A21 T11 [32][33]
  float* lh_s = m_s + 32 * 33;
  float* ll_s = lh_s + kChunk;
  float* b_s = ll_s + kChunk;
  float* ik_s = b_s + kChunk;
  float* iq_s = ik_s + kChunk;
  const DeltaSeq sq = A.seqs[blockIdx.z];
  const int t0 = blockIdx.x * kChunk;
  if (t0 >= sq.count) return;
  const int h = blockIdx.y, g = h / (A.H / A.G), dk = A.dk;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gr = lane >> 2, tq = lane & 3;
  const int nt = min(kChunk, sq.count - t0);
  const int64_t tok = static_cast<int64_t>(sq.tok0) + t0;
  const __nv_bfloat16* kp = A.k + tok * A.stride + static_cast<int64_t>(g) * dk;
  const __nv_bfloat16* qp = A.q + tok * A.stride + static_cast<int64_t>(g) * dk;
  const __nv_bfloat16 zero = __float2bfloat16_rn(0.f);
  if (A.vec) {
    constexpr int pieces = DKP / 8;
    for (int e = tid; e < kChunk * pieces; e += 128) {
      const int t = e / pieces, c = (e - t * pieces) * 8;
      const bool ok = t < nt && c < dk;
      copy16(k_s + t * LDK + c, ok ? kp + static_cast<int64_t>(t) * A.stride + c : kp, ok);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  } else {
    for (int e = tid; e < kChunk * DKP; e += 128) {
      const int t = e / DKP, c = e - t * DKP;
      k_s[t * LDK + c] = (t < nt && c < dk) ? kp[static_cast<int64_t>(t) * A.stride + c] : zero;
    }
  }
  // 1/|q|: four lanes per token
  for (int r = warp * 16 + gr; r < warp * 16 + 16; r += 8) {
    float s = 0.f;
    if (r < nt) {
      const __nv_bfloat16* row = qp + static_cast<int64_t>(r) * A.stride;
      if (A.vec) {
        for (int c = tq * 8; c < dk; c += 32) {
          const int4 raw = *reinterpret_cast<const int4*>(row + c);
          const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const float2 f = __bfloat1622float2(p[i]);
            s = fmaf(f.x, f.x, fmaf(f.y, f.y, s));
          }
        }
      } else {
        for (int c = tq; c < dk; c += 4) {
          const float f = __bfloat162float(row[c]);
          s = fmaf(f, f, s);
        }
      }
    }
    s += __shfl_xor_sync(0xffffffffu, s, 1);
    s += __shfl_xor_sync(0xffffffffu, s, 2);
    if (tq == 0) iq_s[r] = rsqrtf(s + A.unit_eps) * A.q_scale;
  }
  if (warp == 0) {                           // write strengths, running log decays; two tokens per lane
    const float rate = expf(__bfloat162float(A.a_log[h])), bias = __bfloat162float(A.dt_bias[h]);
    float ld[2];
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int t = 2 * lane + j;
      ld[j] = 0.f;
      float b = 0.f;
      if (t < nt) {
        ld[j] = fmaxf(-rate * softp(__bfloat162float(A.a[(tok + t) * A.a_stride + h]) + bias), kLogFloor);
        b = sigm(__bfloat162float(A.beta[(tok + t) * A.beta_stride + h]));
      }
      b_s[t] = b;
    }
    double s = static_cast<double>(ld[0]) + static_cast<double>(ld[1]);
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const double p = __shfl_up_sync(0xffffffffu, s, o);
      if (lane >= o) s += p;
    }
    const double l0 = s - static_cast<double>(ld[1]);
    lh_s[2 * lane] = static_cast<float>(l0);
    ll_s[2 * lane] = static_cast<float>(l0 - static_cast<double>(lh_s[2 * lane]));
    lh_s[2 * lane + 1] = static_cast<float>(s);
    ll_s[2 * lane + 1] = static_cast<float>(s - static_cast<double>(lh_s[2 * lane + 1]));
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  {                                          // 1/|k|: two threads per token
    const int r = tid >> 1;
    const __nv_bfloat162* row = reinterpret_cast<const __nv_bfloat162*>(k_s + r * LDK) + (tid & 1) * (DKP / 4);
    float s = 0.f;
#pragma unroll 8
    for (int i = 0; i < DKP / 4; ++i) {
      const float2 f = __bfloat1622float2(row[i]);
      s = fmaf(f.x, f.x, fmaf(f.y, f.y, s));
    }
    s += __shfl_xor_sync(0xffffffffu, s, 1);
    if ((tid & 1) == 0) ik_s[r] = rsqrtf(s + A.unit_eps);
  }
  __syncthreads();
  {
    float P[8][4];
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) P[n][e] = 0.f;
    const int a_row = lane & 15, a_col = (lane >> 4) * 8;
    const int b_row = (lane & 7) + ((lane >> 4) << 3), b_col = ((lane >> 3) & 1) * 8;
    const uint32_t a_at = smem_at(k_s + (warp * 16 + a_row) * LDK + a_col);
    const uint32_t b_at = smem_at(k_s + b_row * LDK + b_col);
#pragma unroll 4
    for (int ks = 0; ks < DKP / 16; ++ks) {
      uint32_t a[4];
      ldsm4(a, a_at + ks * 32);
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (j <= warp) {
          uint32_t b[4];
          ldsm4(b, b_at + j * 16 * LDK * 2 + ks * 32);
          mma(P[2 * j], a, b[0], b[1]);
          mma(P[2 * j + 1], a, b[2], b[3]);
        }
    }
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int t = warp * 16 + gr + half * 8;
      const float lh = lh_s[t], ll = ll_s[t], f = b_s[t] * ik_s[t];
#pragma unroll
      for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int s = n * 8 + 2 * tq + e;
          a_s[t * kALd + s] = s < t ? P[n][2 * half + e] * (f * ik_s[s] * __expf((lh - lh_s[s]) + (ll - ll_s[s]))) : 0.f;
        }
    }
  }
  __syncthreads();
  if (warp < 2) {
    float x[32];
    const float* blk = a_s + (warp * 32) * kALd + warp * 32;
#pragma unroll
    for (int i = 0; i < 32; ++i) {
      float acc[4] = {i == lane ? 1.f : 0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int j = 0; j < i; j += 4) {
        const float4 r = *reinterpret_cast<const float4*>(blk + i * kALd + j);   // entries from the diagonal on are zero
        acc[0] = fmaf(-r.x, x[j], acc[0]);
        if (j + 1 < i) acc[1] = fmaf(-r.y, x[j + 1], acc[1]);
        if (j + 2 < i) acc[2] = fmaf(-r.z, x[j + 2], acc[2]);
        if (j + 3 < i) acc[3] = fmaf(-r.w, x[j + 3], acc[3]);
      }
      x[i] = (acc[0] + acc[1]) + (acc[2] + acc[3]);
      t_s[(warp * 32 + i) * kALd + warp * 32 + lane] = x[i];
    }
  } else {
    for (int e = tid - 64; e < 32 * 32; e += 64) t_s[(e >> 5) * kALd + 32 + (e & 31)] = 0.f;
  }
  __syncthreads();
  {
    float acc[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i] = 0.f;
    for (int j = 0; j < 32; j += 4) {
      float x[4];
#pragma unroll
      for (int u = 0; u < 4; ++u) x[u] = t_s[(j + u) * kALd + lane];
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const float4 r = *reinterpret_cast<const float4*>(a_s + (32 + warp * 8 + i) * kALd + j);
        acc[i] = fmaf(r.x, x[0], fmaf(r.y, x[1], fmaf(r.z, x[2], fmaf(r.w, x[3], acc[i]))));
      }
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) m_s[(warp * 8 + i) * 33 + lane] = acc[i];
  }
  __syncthreads();
  {
    float acc[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i] = 0.f;
    for (int j = 0; j < 32; j += 4) {
      float x[4];
#pragma unroll
      for (int u = 0; u < 4; ++u) x[u] = m_s[(j + u) * 33 + lane];
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const float4 r = *reinterpret_cast<const float4*>(t_s + (32 + warp * 8 + i) * kALd + 32 + j);
        acc[i] = fmaf(-r.x, x[0], fmaf(-r.y, x[1], fmaf(-r.z, x[2], fmaf(-r.w, x[3], acc[i]))));
      }
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) t_s[(32 + warp * 8 + i) * kALd + lane] = acc[i];
  }
  __syncthreads();
  unsigned char* ws = A.ws + ((first_chunk(sq, blockIdx.z) + blockIdx.x) * A.H + h) * kWsBytes;
  uint32_t* mh = reinterpret_cast<uint32_t*>(ws);
  uint32_t* ml = reinterpret_cast<uint32_t*>(ws + kWsMat);
  for (int e = tid; e < kChunk * kChunk / 2; e += 128) {
    const int t = e >> 5, s = (e & 31) * 2;
    uint32_t hi, lo;
    split2(t_s[t * kALd + s] * b_s[s], t_s[t * kALd + s + 1] * b_s[s + 1], hi, lo);
    mh[e] = hi;
    ml[e] = lo;
  }
  if (tid < kChunk) reinterpret_cast<float4*>(ws + 2 * kWsMat)[tid] = make_float4(lh_s[tid], ll_s[tid], ik_s[tid], iq_s[tid]);
}

template <int DKP>
constexpr size_t prepare_smem() {
  return sizeof(__nv_bfloat16) * kChunk * (DKP + 8) + sizeof(float) * (2 * kChunk * kALd + 32 * 33 + 5 * kChunk);
}

// ---- the walk over a sequence's chunks -----------------------------------------------------------------------------------
// One CTA per (sequence, head, DVB value columns), 4 row warps (16 tokens each) times NC column warps; the state's rows are dealt
// over all warps.  Between a chunk's first product and its end the split copy of the state is not needed: V - e^l K S, then U,
// live in its place.  q and v of the next chunk arrive while U is formed, M while the read-outs are, k at the end.
template <int DKP, int DVB, int NC>
struct DeltaShape {
  static constexpr int NW = 4 * NC, NT = 32 * NW;
  static constexpr int LDK = DKP + 8, LDV = DVB + 8;
  static constexpr int SR = DKP < 2 * kChunk ? 2 * kChunk : DKP;          // rows of the state's copy
  static constexpr size_t kBytes = sizeof(__nv_bfloat16) * (2ull * kChunk * LDK + kChunk * LDV + 2ull * SR * LDV + 2ull * kChunk * kMld) +
                                   sizeof(float4) * 2 * kChunk + sizeof(float) * 4 * kChunk;
  static constexpr int kPerSm = 2 * kBytes + 2048 <= 227 * 1024 ? 2 : 1;
};

template <int DKP, int DVB, int NC>
__global__ void __launch_bounds__(128 * NC, DeltaShape<DKP, DVB, NC>::kPerSm)
delta_chunk_scan_kernel(const DeltaChunkArgs A) {
  using Sh = DeltaShape<DKP, DVB, NC>;
  constexpr int NT = Sh::NT, LDK = Sh::LDK, LDV = Sh::LDV, SR = Sh::SR;
  constexpr int MT = DKP / (16 * Sh::NW);       // 16-row tiles of the state per warp
  constexpr int SN = DVB / 8;                   // 8-column tiles of the state
  constexpr int ON = DVB / 8 / NC;              // 8-column tiles of a warp's read-outs
  static_assert(MT >= 1 && ON >= 2, "shape");
  extern __shared__ __align__(16) unsigned char dc_raw[];
  __nv_bfloat16* q_s = reinterpret_cast<__nv_bfloat16*>(dc_raw);
  __nv_bfloat16* k_s = q_s + kChunk * LDK;
  __nv_bfloat16* v_s = k_s + kChunk * LDK;
  __nv_bfloat16* sh_s = v_s + kChunk * LDV;     // state, high parts [SR][LDV]; rows 0..63 also R, then weighted U; 64..127 U
  __nv_bfloat16* sl_s = sh_s + SR * LDV;        // low parts
  __nv_bfloat16* mh_s = sl_s + SR * LDV;        // M [64][kMld]
  __nv_bfloat16* ml_s = mh_s + kChunk * kMld;
  float4* sc_s = reinterpret_cast<float4*>(ml_s + kChunk * kMld);   // [2][64] (l high, l low, 1/|k|, q_scale/|q|)
  float* ek_s = reinterpret_cast<float*>(sc_s + 2 * kChunk);        // e^(l_t) / |k_t|
  float* eq_s = ek_s + kChunk;                                      // e^(l_t) q_scale / |q_t|
  float* w_s = eq_s + kChunk;                                       // e^(l_64 - l_t) / |k_t|
  float* end_s = w_s + kChunk;                                      // [0] = e^(l_64)

  const DeltaSeq sq = A.seqs[blockIdx.x];
  if (sq.count <= 0) return;
  const int h = blockIdx.y, g = h / (A.H / A.G), dk = A.dk, dv = A.dv;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int wr = warp & 3, wc = warp >> 2;
  const int gr = lane >> 2, tq = lane & 3;
  const int col0 = blockIdx.z * DVB, ncol = min(DVB, dv - col0);
  float* st = A.state + (static_cast<int64_t>(sq.slot) * A.H + h) * dk * dv + col0;
  const __nv_bfloat16* q = A.q + static_cast<int64_t>(sq.tok0) * A.stride + static_cast<int64_t>(g) * dk;
  const __nv_bfloat16* k = A.k + static_cast<int64_t>(sq.tok0) * A.stride + static_cast<int64_t>(g) * dk;
  const __nv_bfloat16* v = A.v + static_cast<int64_t>(sq.tok0) * A.stride + static_cast<int64_t>(h) * dv + col0;
  const unsigned char* ws = A.ws + (first_chunk(sq, blockIdx.x) * A.H + h) * kWsBytes;
  const int64_t ws_step = static_cast<int64_t>(A.H) * kWsBytes;
  const __nv_bfloat16 zero = __float2bfloat16_rn(0.f);

  auto load_rows = [&](__nv_bfloat16* dst, int ldd, int cols, const __nv_bfloat16* src, int width, int t0) {
    if (A.vec) {
      const int pieces = cols / 8;
      for (int e = tid; e < kChunk * pieces; e += NT) {
        const int t = e / pieces, c = (e - t * pieces) * 8;
        const bool ok = t0 + t < sq.count && c < width;
        copy16(dst + t * ldd + c, ok ? src + static_cast<int64_t>(t0 + t) * A.stride + c : src, ok);
      }
    } else {
      for (int e = tid; e < kChunk * cols; e += NT) {
        const int t = e / cols, c = e - t * cols;
        dst[t * ldd + c] = (t0 + t < sq.count && c < width) ? src[static_cast<int64_t>(t0 + t) * A.stride + c] : zero;
      }
    }
  };
  auto load_m = [&](const unsigned char* src, int buf) {
    for (int e = tid; e < 2 * kChunk * 8; e += NT) {
      const int part = e >> 9, r = (e >> 3) & 63, c = (e & 7) * 8;
      copy16((part ? ml_s : mh_s) + r * kMld + c, src + part * kWsMat + (r * kChunk + c) * sizeof(__nv_bfloat16), true);
    }
    if (tid < kChunk) copy16(sc_s + buf * kChunk + tid, src + 2 * kWsMat + tid * sizeof(float4), true);
  };
  auto commit = [] { asm volatile("cp.async.commit_group;" ::: "memory"); };

  float S[MT][SN][4];
  const int srow = warp * MT * 16;
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < SN; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = srow + m * 16 + gr + (e >> 1) * 8, c = n * 8 + 2 * tq + (e & 1);
        S[m][n][e] = (!sq.fresh && r < dk && c < ncol) ? st[static_cast<int64_t>(r) * dv + c] : 0.f;
      }
  auto publish_state = [&]() {
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < SN; ++n)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int r = srow + m * 16 + gr + half * 8, c = n * 8 + 2 * tq;
          uint32_t hi, lo;
          split2(S[m][n][2 * half], S[m][n][2 * half + 1], hi, lo);
          *reinterpret_cast<uint32_t*>(sh_s + r * LDV + c) = hi;
          *reinterpret_cast<uint32_t*>(sl_s + r * LDV + c) = lo;
        }
  };
  publish_state();
  load_rows(q_s, LDK, DKP, q, dk, 0);
  load_rows(k_s, LDK, DKP, k, dk, 0);
  load_rows(v_s, LDV, DVB, v, ncol, 0);
  load_m(ws, 0);
  commit();

  const int a_row = lane & 15, a_col = (lane >> 4) * 8;                                 // A [m][k], and B [k][n] transposed
  const int b_row = (lane & 7) + ((lane >> 4) << 3), b_col = ((lane >> 3) & 1) * 8;     // B [n][k], and A [k][m] transposed
  const uint32_t q_at = smem_at(q_s + (wr * 16 + a_row) * LDK + a_col);
  const uint32_t kr_at = smem_at(k_s + (wr * 16 + a_row) * LDK + a_col);
  const uint32_t k_at = smem_at(k_s + b_row * LDK + b_col);
  const uint32_t sh_at = smem_at(sh_s + a_row * LDV + wc * ON * 8 + a_col);
  const uint32_t sl_at = smem_at(sl_s + a_row * LDV + wc * ON * 8 + a_col);
  const uint32_t mh_at = smem_at(mh_s + (wr * 16 + a_row) * kMld + a_col);
  const uint32_t ml_at = smem_at(ml_s + (wr * 16 + a_row) * kMld + a_col);
  const uint32_t uh_at = smem_at(sh_s + a_row * LDV + a_col);                           // weighted U, all columns
  const uint32_t ul_at = smem_at(sl_s + a_row * LDV + a_col);
  const uint32_t kt_at = smem_at(k_s + b_row * LDK + srow + b_col);
  const int ra = wr * 16 + gr, rb = ra + 8;     // the thread's two tokens

  int buf = 0;
  for (int t0 = 0; t0 < sq.count; t0 += kChunk, buf ^= 1, ws += ws_step) {
    const bool more = t0 + kChunk < sq.count;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    const float4* sc = sc_s + buf * kChunk;
    if (tid < kChunk) {
      const float4 x = sc[tid], e = sc[kChunk - 1];
      const float el = expf(x.x + x.y);
      ek_s[tid] = el * x.z;
      eq_s[tid] = el * x.w;
      w_s[tid] = expf((e.x - x.x) + (e.y - x.y)) * x.z;
      if (tid == 0) end_s[0] = expf(e.x + e.y);
    }
    // ---- K S, Q S and Q K^T of the warp's 16 tokens
    float O[ON][4], W[ON][4], P[8][4];
#pragma unroll
    for (int n = 0; n < ON; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) O[n][e] = W[n][e] = 0.f;
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) P[n][e] = 0.f;
#pragma unroll 2
    for (int ks = 0; ks < DKP / 16; ++ks) {
      uint32_t aq[4], ak[4];
      ldsm4(aq, q_at + ks * 32);
      ldsm4(ak, kr_at + ks * 32);
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (j <= wr) {
          uint32_t b[4];
          ldsm4(b, k_at + j * 16 * LDK * 2 + ks * 32);
          mma(P[2 * j], aq, b[0], b[1]);
          mma(P[2 * j + 1], aq, b[2], b[3]);
        }
#pragma unroll
      for (int j = 0; j < ON / 2; ++j) {
        uint32_t b[4];
        ldsm4t(b, sh_at + ks * 16 * LDV * 2 + j * 32);
        mma(O[2 * j], aq, b[0], b[1]);
        mma(O[2 * j + 1], aq, b[2], b[3]);
        mma(W[2 * j], ak, b[0], b[1]);
        mma(W[2 * j + 1], ak, b[2], b[3]);
        ldsm4t(b, sl_at + ks * 16 * LDV * 2 + j * 32);
        mma(O[2 * j], aq, b[0], b[1]);
        mma(O[2 * j + 1], aq, b[2], b[3]);
        mma(W[2 * j], ak, b[0], b[1]);
        mma(W[2 * j + 1], ak, b[2], b[3]);
      }
    }
    __syncthreads();                            // q, the split state have been read; the chunk's factors are there
    {
      const float ka = ek_s[ra], kb = ek_s[rb], qa = eq_s[ra], qb = eq_s[rb];
#pragma unroll
      for (int n = 0; n < ON; ++n) {            // R = V - e^l K S
        const int c = (wc * ON + n) * 8 + 2 * tq;
        const float2 va = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(v_s + ra * LDV + c));
        const float2 vb = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(v_s + rb * LDV + c));
        uint32_t hi, lo;
        split2(fmaf(-ka, W[n][0], va.x), fmaf(-ka, W[n][1], va.y), hi, lo);
        *reinterpret_cast<uint32_t*>(sh_s + ra * LDV + c) = hi;
        *reinterpret_cast<uint32_t*>(sl_s + ra * LDV + c) = lo;
        split2(fmaf(-kb, W[n][2], vb.x), fmaf(-kb, W[n][3], vb.y), hi, lo);
        *reinterpret_cast<uint32_t*>(sh_s + rb * LDV + c) = hi;
        *reinterpret_cast<uint32_t*>(sl_s + rb * LDV + c) = lo;
        O[n][0] *= qa;
        O[n][1] *= qa;
        O[n][2] *= qb;
        O[n][3] *= qb;
      }
      const float4 xa = sc[ra], xb = sc[rb];
#pragma unroll
      for (int n = 0; n < 8; ++n)
        if (n / 2 <= wr) {
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int s = n * 8 + 2 * tq + e;
            const float4 x = sc[s];
            P[n][e] = s <= ra ? P[n][e] * (__expf((xa.x - x.x) + (xa.y - x.y)) * xa.w * x.z) : 0.f;
            P[n][2 + e] = s <= rb ? P[n][2 + e] * (__expf((xb.x - x.x) + (xb.y - x.y)) * xb.w * x.z) : 0.f;
          }
        }
    }
    __syncthreads();                            // R is there; q and v have been read
    if (more) {
      load_rows(q_s, LDK, DKP, q, dk, t0 + kChunk);
      load_rows(v_s, LDV, DVB, v, ncol, t0 + kChunk);
      commit();
    }
    // ---- U = M R
    float U[ON][4];
#pragma unroll
    for (int n = 0; n < ON; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) U[n][e] = 0.f;
#pragma unroll
    for (int ks = 0; ks < 4; ++ks)
      if (ks <= wr) {
        uint32_t ah[4], al[4];
        ldsm4(ah, mh_at + ks * 32);
        ldsm4(al, ml_at + ks * 32);
#pragma unroll
        for (int j = 0; j < ON / 2; ++j) {
          uint32_t b[4];
          ldsm4t(b, sh_at + ks * 16 * LDV * 2 + j * 32);
          mma(U[2 * j], ah, b[0], b[1]);
          mma(U[2 * j + 1], ah, b[2], b[3]);
          mma(U[2 * j], al, b[0], b[1]);
          mma(U[2 * j + 1], al, b[2], b[3]);
          ldsm4t(b, sl_at + ks * 16 * LDV * 2 + j * 32);
          mma(U[2 * j], ah, b[0], b[1]);
          mma(U[2 * j + 1], ah, b[2], b[3]);
        }
      }
#pragma unroll
    for (int n = 0; n < ON; ++n)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int r = kChunk + (half ? rb : ra), c = (wc * ON + n) * 8 + 2 * tq;
        uint32_t hi, lo;
        split2(U[n][2 * half], U[n][2 * half + 1], hi, lo);
        *reinterpret_cast<uint32_t*>(sh_s + r * LDV + c) = hi;
        *reinterpret_cast<uint32_t*>(sl_s + r * LDV + c) = lo;
      }
    __syncthreads();                            // U is there; R and M have been read
    if (more) {
      load_m(ws + ws_step, buf ^ 1);
      commit();
    }
    // ---- read-outs, and U weighted for the state
    const float wa = w_s[ra], wb = w_s[rb];
#pragma unroll
    for (int n = 0; n < ON; ++n)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int r = half ? rb : ra, c = (wc * ON + n) * 8 + 2 * tq;
        const float w = half ? wb : wa;
        uint32_t hi, lo;
        split2(U[n][2 * half] * w, U[n][2 * half + 1] * w, hi, lo);
        *reinterpret_cast<uint32_t*>(sh_s + r * LDV + c) = hi;
        *reinterpret_cast<uint32_t*>(sl_s + r * LDV + c) = lo;
      }
#pragma unroll
    for (int ks = 0; ks < 4; ++ks)
      if (ks <= wr) {
        uint32_t hi[4], lo[4];
        split2(P[2 * ks][0], P[2 * ks][1], hi[0], lo[0]);
        split2(P[2 * ks][2], P[2 * ks][3], hi[1], lo[1]);
        split2(P[2 * ks + 1][0], P[2 * ks + 1][1], hi[2], lo[2]);
        split2(P[2 * ks + 1][2], P[2 * ks + 1][3], hi[3], lo[3]);
#pragma unroll
        for (int j = 0; j < ON / 2; ++j) {
          uint32_t b[4];
          ldsm4t(b, sh_at + (kChunk + ks * 16) * LDV * 2 + j * 32);
          mma(O[2 * j], hi, b[0], b[1]);
          mma(O[2 * j + 1], hi, b[2], b[3]);
          mma(O[2 * j], lo, b[0], b[1]);
          mma(O[2 * j + 1], lo, b[2], b[3]);
          ldsm4t(b, sl_at + (kChunk + ks * 16) * LDV * 2 + j * 32);
          mma(O[2 * j], hi, b[0], b[1]);
          mma(O[2 * j + 1], hi, b[2], b[3]);
        }
      }
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int r = half ? rb : ra;
      if (t0 + r >= sq.count) continue;
      float* orow = A.o + (static_cast<int64_t>(sq.tok0 + t0 + r) * A.H + h) * dv + col0;
      const bool pair = (dv & 1) == 0;          // an even row length keeps every pair 8-byte aligned
#pragma unroll
      for (int n = 0; n < ON; ++n) {
        const int c = (wc * ON + n) * 8 + 2 * tq;
        if (pair && c + 1 < ncol) *reinterpret_cast<float2*>(orow + c) = make_float2(O[n][2 * half], O[n][2 * half + 1]);
        else {
          if (c < ncol) orow[c] = O[n][2 * half];
          if (c + 1 < ncol) orow[c + 1] = O[n][2 * half + 1];
        }
      }
    }
    __syncthreads();                            // the weighted U is there
    // ---- the state past this chunk
    const float end = end_s[0];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < SN; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[m][n][e] *= end;
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      uint32_t a[MT][4];
#pragma unroll
      for (int m = 0; m < MT; ++m) ldsm4t(a[m], kt_at + ks * 16 * LDK * 2 + m * 32);
#pragma unroll
      for (int j = 0; j < SN / 2; ++j) {
        uint32_t b[4];
        ldsm4t(b, uh_at + ks * 16 * LDV * 2 + j * 32);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          mma(S[m][2 * j], a[m], b[0], b[1]);
          mma(S[m][2 * j + 1], a[m], b[2], b[3]);
        }
        ldsm4t(b, ul_at + ks * 16 * LDV * 2 + j * 32);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          mma(S[m][2 * j], a[m], b[0], b[1]);
          mma(S[m][2 * j + 1], a[m], b[2], b[3]);
        }
      }
    }
    __syncthreads();                            // k and the weighted U have been read
    if (more) {
      load_rows(k_s, LDK, DKP, k, dk, t0 + kChunk);
      commit();
      publish_state();
    }
  }
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < SN; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = srow + m * 16 + gr + (e >> 1) * 8, c = n * 8 + 2 * tq + (e & 1);
        if (r < dk && c < ncol) st[static_cast<int64_t>(r) * dv + c] = S[m][n][e];
      }
}

// ---- one token per sequence ------------------------------------------------------------------------------------------------
// Bound by the state's bytes: a CTA (256 threads) holds its (sequence, head, LPR * V value columns) in registers between the one
// read and the one write.  r = S^T k and p = S^T q come from one pass; u = beta (v - g r), o = g p + (k.q) u, S <- g S + k u^T.
struct DeltaStepArgs {
  float* o;
  const void* q; const void* k; const void* v; int64_t stride;
  const void* beta; int64_t beta_stride;
  const void* a; int64_t a_stride;
  const void* dt_bias; const void* a_log;
  float* state;
  const DeltaSeq* seqs;
  int H, G, dk, dv;
  float unit_eps, q_scale;
};

template <typename T, int V, int LPR, int RPT>
__global__ void __launch_bounds__(256)
delta_step_kernel(const DeltaStepArgs A) {
  constexpr int RPI = 256 / LPR, COLS = LPR * V;
  extern __shared__ __align__(16) float ds_sm[];     // q[dk] | k[dk] | partial r, p [2][8 warps][COLS] | u[COLS]
  __shared__ float sums[3];
  const DeltaSeq sq = A.seqs[blockIdx.x];
  const int h = blockIdx.y, g = h / (A.H / A.G), dk = A.dk, dv = A.dv, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int64_t n = sq.tok0;
  float* qs = ds_sm;
  float* ks = qs + dk;
  float* ps = ds_sm + ((2 * dk + 3) & ~3);
  float* us = ps + 2 * 8 * COLS;
  const int lr = tid % LPR, row0 = tid / LPR, c0 = blockIdx.z * COLS, col = c0 + lr * V;
  const bool has = col < dv;
  float* st = A.state + (static_cast<int64_t>(sq.slot) * A.H + h) * dk * dv + col;
  float s[RPT][V];
#pragma unroll
  for (int j = 0; j < RPT; ++j) {
    const int i = row0 + j * RPI;
#pragma unroll
    for (int u = 0; u < V; ++u) s[j][u] = 0.f;
    if (has && i < dk && !sq.fresh) {
      if constexpr (V == 4) {
        const float4 x = *reinterpret_cast<const float4*>(st + static_cast<int64_t>(i) * dv);
        s[j][0] = x.x;
        s[j][1] = x.y;
        s[j][2] = x.z;
        s[j][3] = x.w;
      } else {
        s[j][0] = st[static_cast<int64_t>(i) * dv];
      }
    }
  }
  const T* q = static_cast<const T*>(A.q) + n * A.stride + static_cast<int64_t>(g) * dk;
  const T* k = static_cast<const T*>(A.k) + n * A.stride + static_cast<int64_t>(g) * dk;
  if (warp < 3) {                                     // |q|^2, |k|^2, k.q
    float t = 0.f;
    for (int i = lane; i < dk; i += 32) {
      const float x = Cvt<T>::to_f32(warp == 1 ? k[i] : q[i]), y = Cvt<T>::to_f32(warp == 0 ? q[i] : k[i]);
      t = fmaf(x, y, t);
      if (warp == 0) qs[i] = x;
      if (warp == 1) ks[i] = x;
    }
    t = warp_sum(t);
    if (lane == 0) sums[warp] = t;
  }
  // the decay as g - 1: one just below 1 is not rounded alike token after token
  const float lost = expm1f(-expf(Cvt<T>::to_f32(static_cast<const T*>(A.a_log)[h])) *
                            softp(Cvt<T>::to_f32(static_cast<const T*>(A.a)[n * A.a_stride + h]) +
                                  Cvt<T>::to_f32(static_cast<const T*>(A.dt_bias)[h])));
  const float decay = 1.0f + lost;
  const float beta = sigm(Cvt<T>::to_f32(static_cast<const T*>(A.beta)[n * A.beta_stride + h]));
  __syncthreads();
  const float iq = rsqrtf(sums[0] + A.unit_eps) * A.q_scale, ik = rsqrtf(sums[1] + A.unit_eps), kq = sums[2] * iq * ik;
  float r[V], p[V];
#pragma unroll
  for (int u = 0; u < V; ++u) r[u] = p[u] = 0.f;
#pragma unroll
  for (int j = 0; j < RPT; ++j) {
    const int i = row0 + j * RPI;
    if (i < dk) {
      const float ki = ks[i], qi = qs[i];
#pragma unroll
      for (int u = 0; u < V; ++u) {
        r[u] = fmaf(s[j][u], ki, r[u]);
        p[u] = fmaf(s[j][u], qi, p[u]);
      }
    }
  }
#pragma unroll
  for (int u = 0; u < V; ++u) {
#pragma unroll
    for (int o = LPR; o < 32; o <<= 1) {
      r[u] += __shfl_xor_sync(0xffffffffu, r[u], o);
      p[u] += __shfl_xor_sync(0xffffffffu, p[u], o);
    }
    if (lane < LPR) {
      ps[warp * COLS + lr * V + u] = r[u];
      ps[(8 + warp) * COLS + lr * V + u] = p[u];
    }
  }
  __syncthreads();
  if (tid < COLS) {
    float rr = 0.f, pp = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) {
      rr += ps[w * COLS + tid];
      pp += ps[(8 + w) * COLS + tid];
    }
    float u = 0.f;
    if (c0 + tid < dv) {
      const float vv = Cvt<T>::to_f32(static_cast<const T*>(A.v)[n * A.stride + static_cast<int64_t>(h) * dv + c0 + tid]);
      u = beta * fmaf(-decay * ik, rr, vv);
      A.o[(n * A.H + h) * dv + c0 + tid] = fmaf(decay * iq, pp, kq * u);
    }
    us[tid] = u * ik;
  }
  __syncthreads();
  if (!has) return;
#pragma unroll
  for (int j = 0; j < RPT; ++j) {
    const int i = row0 + j * RPI;
    if (i < dk) {
      const float ki = ks[i];
      if constexpr (V == 4) {
        const float4 u = *reinterpret_cast<const float4*>(us + lr * 4);
        *reinterpret_cast<float4*>(st + static_cast<int64_t>(i) * dv) =
            make_float4(s[j][0] + fmaf(lost, s[j][0], ki * u.x), s[j][1] + fmaf(lost, s[j][1], ki * u.y),
                        s[j][2] + fmaf(lost, s[j][2], ki * u.z), s[j][3] + fmaf(lost, s[j][3], ki * u.w));
      } else {
        st[static_cast<int64_t>(i) * dv] = s[j][0] + fmaf(lost, s[j][0], ki * us[lr]);
      }
    }
  }
}

template <typename F>
int delta_by_dtype(int dtype, const char* name, F&& f) {
  switch (dtype) {
    case B200_DTYPE_F16:
      return f(static_cast<__half*>(nullptr));
    case B200_DTYPE_BF16:
      return f(static_cast<__nv_bfloat16*>(nullptr));
    case B200_DTYPE_F32:
      return f(static_cast<float*>(nullptr));
    default:
      return fail(B200_EINVAL, "%s: unsupported dtype %d", name, dtype);
  }
}

}  // namespace
}  // namespace b200

using namespace b200;

extern "C" {

int b200_delta_chunk_scan_supported(int dk, int dv, int dtype) {
  return dtype == B200_DTYPE_BF16 && dk >= 1 && dk <= 256 && dv >= 1;
}

size_t b200_delta_chunk_workspace(int n_tok, int n_seqs, int H) {
  if (n_tok <= 0 || n_seqs <= 0 || H <= 0) return 0;
  return (static_cast<size_t>(n_tok / kChunk) + n_seqs + 1) * H * kWsBytes;
}

int b200_delta_chunk_scan(float* o_raw, const void* q, const void* k, const void* v, int64_t in_stride, const void* beta_logit,
                          int64_t beta_stride, const void* a_logit, int64_t a_stride, const void* dt_bias, const void* a_log,
                          float* state, const int32_t* seqs, int n_seqs, int max_count, int H, int G, int dk, int dv,
                          float unit_eps, float q_scale, void* workspace, int dtype, void* stream) {
  if (n_seqs < 0 || max_count < 0 || H <= 0 || G <= 0 || H % G || dk <= 0 || dv <= 0)
    return fail(B200_EINVAL, "b200_delta_chunk_scan: bad sizes");
  if (!b200_delta_chunk_scan_supported(dk, dv, dtype))
    return fail(B200_ESHAPE, "b200_delta_chunk_scan: dtype %d, key size %d not supported", dtype, dk);
  if (n_seqs == 0 || max_count == 0) return 0;
  if (!o_raw || !q || !k || !v || !beta_logit || !a_logit || !dt_bias || !a_log || !state || !seqs || !workspace ||
      !aligned16(workspace))
    return fail(B200_EINVAL, "b200_delta_chunk_scan: null pointer or unaligned workspace");
  if (n_seqs > 65535 || H > 65535) return fail(B200_ESHAPE, "b200_delta_chunk_scan: too many sequences or heads");
  using B = __nv_bfloat16;
  const int vec = dk % 8 == 0 && dv % 8 == 0 && in_stride % 8 == 0 && aligned16(q) && aligned16(k) && aligned16(v);
  const DeltaChunkArgs A{o_raw, static_cast<const B*>(q), static_cast<const B*>(k), static_cast<const B*>(v), in_stride,
                         static_cast<const B*>(beta_logit), beta_stride, static_cast<const B*>(a_logit), a_stride,
                         static_cast<const B*>(dt_bias), static_cast<const B*>(a_log), state,
                         reinterpret_cast<const DeltaSeq*>(seqs), H, G, dk, dv, unit_eps, q_scale,
                         static_cast<unsigned char*>(workspace), vec};
  auto s = static_cast<cudaStream_t>(stream);
  auto run = [&](auto kern, size_t smem, dim3 grid, int nt) {
    cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    kern<<<grid, nt, smem, s>>>(A);
  };
  const dim3 pg((max_count + kChunk - 1) / kChunk, H, n_seqs);
  if (dk <= 64) run(delta_prepare_kernel<64>, prepare_smem<64>(), pg, 128);
  else if (dk <= 128) run(delta_prepare_kernel<128>, prepare_smem<128>(), pg, 128);
  else run(delta_prepare_kernel<256>, prepare_smem<256>(), pg, 128);
  if (const int rc = check_launch("b200_delta_chunk_scan (prepare)")) return rc;
  auto scan = [&](auto kern, size_t smem, int dvb, int nt) { run(kern, smem, dim3(n_seqs, H, (dv + dvb - 1) / dvb), nt); };
  // blocks of 32 value columns also where blocks of 64 would leave SMs idle: the walk is a chain, and theirs is shorter
  const bool narrow = dv <= 32 || static_cast<int64_t>(n_seqs) * H * ((dv + 63) / 64) <= kNumSMs;
  if (dk <= 64) {
    if (narrow) scan(delta_chunk_scan_kernel<64, 32, 1>, DeltaShape<64, 32, 1>::kBytes, 32, 128);
    else scan(delta_chunk_scan_kernel<64, 64, 1>, DeltaShape<64, 64, 1>::kBytes, 64, 128);
  } else if (dk <= 128) {
    if (narrow) scan(delta_chunk_scan_kernel<128, 32, 1>, DeltaShape<128, 32, 1>::kBytes, 32, 128);
    else scan(delta_chunk_scan_kernel<128, 64, 2>, DeltaShape<128, 64, 2>::kBytes, 64, 256);
  } else {
    if (narrow) scan(delta_chunk_scan_kernel<256, 32, 2>, DeltaShape<256, 32, 2>::kBytes, 32, 256);
    else scan(delta_chunk_scan_kernel<256, 64, 2>, DeltaShape<256, 64, 2>::kBytes, 64, 256);
  }
  return check_launch("b200_delta_chunk_scan");
}

int b200_delta_step(float* o_raw, const void* q, const void* k, const void* v, int64_t in_stride, const void* beta_logit,
                    int64_t beta_stride, const void* a_logit, int64_t a_stride, const void* dt_bias, const void* a_log,
                    float* state, const int32_t* seqs, int n_seqs, int H, int G, int dk, int dv, float unit_eps, float q_scale,
                    int dtype, void* stream) {
  if (n_seqs < 0 || H <= 0 || G <= 0 || H % G || dk <= 0 || dv <= 0) return fail(B200_EINVAL, "b200_delta_step: bad sizes");
  if (dk > 256) return fail(B200_ESHAPE, "b200_delta_step: key size %d beyond 256", dk);
  if (n_seqs == 0) return 0;
  if (!o_raw || !q || !k || !v || !beta_logit || !a_logit || !dt_bias || !a_log || !state || !seqs)
    return fail(B200_EINVAL, "b200_delta_step: null pointer");
  const DeltaStepArgs A{o_raw, q, k, v, in_stride, beta_logit, beta_stride, a_logit, a_stride, dt_bias, a_log, state,
                        reinterpret_cast<const DeltaSeq*>(seqs), H, G, dk, dv, unit_eps, q_scale};
  return delta_by_dtype(dtype, "b200_delta_step", [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    auto launch = [&](auto kern, int cols) {
      const size_t smem = sizeof(float) * (((2 * static_cast<size_t>(dk) + 3) & ~size_t{3}) + 17 * static_cast<size_t>(cols));
      kern<<<dim3(n_seqs, H, (dv + cols - 1) / cols), 256, smem, static_cast<cudaStream_t>(stream)>>>(A);
    };
    if (dv % 4 || !aligned16(state)) launch(delta_step_kernel<T, 1, 32, 32>, 32);
    else if (dv <= 32) {
      if (dk <= 128) launch(delta_step_kernel<T, 4, 8, 4>, 32);
      else launch(delta_step_kernel<T, 4, 8, 8>, 32);
    } else {
      if (dk <= 64) launch(delta_step_kernel<T, 4, 16, 4>, 64);
      else if (dk <= 128) launch(delta_step_kernel<T, 4, 16, 8>, 64);
      else launch(delta_step_kernel<T, 4, 16, 16>, 64);
    }
    return check_launch("b200_delta_step");
  });
}

}  // extern "C"
