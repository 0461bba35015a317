// The decayed outer-product state (see b200_recurrent_ops.cu) over prompt portions in chunks of 64 tokens on the tensor cores,
// for bf16 inputs.  With l_t the running sum of log decays inside a chunk, c the write coefficients and S the fp32 state at the
// chunk's start,
//
//   o_t = q_scale [ e^(l_t) S^T q_t + sum_(s <= t) e^(l_t - l_s) c_s (k_s . q_t) v_s ] + skip v_t
//   S  <- e^(l_64) S + sum_s e^(l_64 - l_s) c_s k_s v_s^T
//
// and the same without v for the vector recurrence n (its product with q is the row sum of the second term's weights).
//
// q, k and v enter the products as they are (bf16); every fp32 operand - the state, the weights of the second term, the
// weighted keys - is split into two bf16 numbers (x = hi + lo, relative remainder 2^-17) and multiplied twice, with fp32
// accumulation; the state itself stays fp32 in accumulator registers for the whole portion.  Exponents are differences of
// running sums formed in double and kept as two floats, always of sums <= 0, so nothing overflows however fast a head forgets.
//
// One CTA per (sequence, head, DVB value columns), 4 row warps (16 tokens each) times NC column warps; the state's rows are
// dealt over all warps.  q, k, v arrive by cp.async (plain loads when rows are not 16-byte aligned): q of the next chunk while
// the state is updated, k and v behind it; other CTAs of the SM fill the rest.
#include <algorithm>

#include "../../include/b200_mixers.h"
#include "b200_common.cuh"

namespace b200 {
namespace {

constexpr int kChunk = 64;
constexpr float kLogFloor = -200.0f;   // e^-200 is 0 in fp32: slower forgetting is kept exactly, faster is "everything"

struct ChunkSeq {
  int tok0, count, slot, fresh;
};

struct ChunkArgs {
  float* o;
  float* nq;
  const __nv_bfloat16* q;
  const __nv_bfloat16* k;
  const __nv_bfloat16* v;
  int64_t q_stride, k_stride, v_stride;
  const float* log_decay;
  const float* coef;
  const float* skip;
  float q_scale;
  float* state;
  float* nstate;
  const ChunkSeq* seqs;
  int H, G, dk, dv, vec;   // vec: rows of q, k and v may be copied in 16-byte pieces
};

__device__ __forceinline__ uint32_t smem_addr(const void* p) { return static_cast<uint32_t>(__cvta_generic_to_shared(p)); }
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
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_addr(dst)), "l"(src), "r"(bytes) : "memory");
}

// x, y -> (hi pair, lo pair), packed for an MMA operand
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - f.x, y - f.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}

template <int DKP, int DVB, int NC>
struct ChunkShape {
  static constexpr int NW = 4 * NC, NT = 32 * NW;
  static constexpr int LDK = DKP + 8, LDV = DVB + 8;             // padded rows: ldmatrix without bank conflicts
  static constexpr size_t kBytes = sizeof(__nv_bfloat16) * (2ull * kChunk * LDK + kChunk * LDV + 2ull * DKP * LDV) +
                                   sizeof(float) * (6 * kChunk + DKP);
};

template <int DKP, int DVB, int NC>
__global__ void __launch_bounds__(128 * NC)
decay_chunk_scan_kernel(const ChunkArgs A) {
  using Sh = ChunkShape<DKP, DVB, NC>;
  constexpr int NT = Sh::NT, LDK = Sh::LDK, LDV = Sh::LDV;
  constexpr int MT = DKP / (16 * Sh::NW);       // 16-row tiles of the state per warp
  constexpr int SN = DVB / 8;                   // 8-column tiles of the state
  constexpr int ON = DVB / 8 / NC;              // 8-column tiles of a warp's read-outs
  static_assert(MT >= 1 && ON >= 2, "shape");
  extern __shared__ __align__(16) unsigned char cs_raw[];
  __nv_bfloat16* q_s = reinterpret_cast<__nv_bfloat16*>(cs_raw);
  __nv_bfloat16* k_s = q_s + kChunk * LDK;
  __nv_bfloat16* v_s = k_s + kChunk * LDK;
  __nv_bfloat16* sh_s = v_s + kChunk * LDV;     // state, high parts [DKP][LDV]
  __nv_bfloat16* sl_s = sh_s + DKP * LDV;       // state, low parts
  float* lh_s = reinterpret_cast<float*>(sl_s + DKP * LDV);   // running log decay, two floats
  float* ll_s = lh_s + kChunk;
  float* c_s = ll_s + kChunk;                   // write coefficient
  float* el_s = c_s + kChunk;                   // e^(l_t)
  float* w_s = el_s + kChunk;                   // e^(l_64 - l_s) c_s
  float* end_s = w_s + kChunk;                  // [0] = e^(l_64)
  float* n_s = end_s + kChunk;                  // n [DKP]

  const ChunkSeq sq = A.seqs[blockIdx.x];
  const int h = blockIdx.y, g = h / (A.H / A.G), dk = A.dk, dv = A.dv;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int wr = warp & 3, wc = warp >> 2;      // rows 16 wr .. of a chunk; columns ON*8*wc ..
  const int gr = lane >> 2, tq = lane & 3;
  const int col0 = blockIdx.z * DVB, ncol = min(DVB, dv - col0);
  const bool has_n = A.nstate != nullptr && blockIdx.z == 0;
  float* st = A.state + (static_cast<int64_t>(sq.slot) * A.H + h) * dk * dv + col0;
  float* nst = A.nstate ? A.nstate + (static_cast<int64_t>(sq.slot) * A.H + h) * dk : nullptr;
  const __nv_bfloat16* q = A.q + static_cast<int64_t>(sq.tok0) * A.q_stride + static_cast<int64_t>(g) * dk;
  const __nv_bfloat16* k = A.k + static_cast<int64_t>(sq.tok0) * A.k_stride + static_cast<int64_t>(g) * dk;
  const __nv_bfloat16* v = A.v + static_cast<int64_t>(sq.tok0) * A.v_stride + static_cast<int64_t>(h) * dv + col0;
  const float* ld = A.log_decay + static_cast<int64_t>(sq.tok0) * A.H + h;
  const float* cf = A.coef + static_cast<int64_t>(sq.tok0) * A.H + h;
  const float skip = A.skip ? A.skip[h] : 0.f;
  const __nv_bfloat16 zero = __float2bfloat16_rn(0.f);

  // rows t0 .. t0 + 63 of one operand into shared memory; columns past `width` and rows past the portion become zero
  auto load_rows = [&](__nv_bfloat16* dst, int ldd, int cols, const __nv_bfloat16* src, int64_t stride, int width, int t0) {
    if (A.vec) {
      const int pieces = cols / 8;
      for (int e = tid; e < kChunk * pieces; e += NT) {
        const int t = e / pieces, c = (e - t * pieces) * 8;
        const bool ok = t0 + t < sq.count && c < width;
        copy16(dst + t * ldd + c, ok ? src + static_cast<int64_t>(t0 + t) * stride + c : src, ok);
      }
    } else {
      for (int e = tid; e < kChunk * cols; e += NT) {
        const int t = e / cols, c = e - t * cols;
        dst[t * ldd + c] = (t0 + t < sq.count && c < width) ? src[static_cast<int64_t>(t0 + t) * stride + c] : zero;
      }
    }
  };
  // the chunk's running log decays and what follows from them; one warp, two tokens per lane
  float nl0 = 0.f, nl1 = 0.f, nc0 = 0.f, nc1 = 0.f;
  auto fetch_decay = [&](int t0) {
    const int a = t0 + 2 * lane;
    nl0 = a < sq.count ? fmaxf(ld[static_cast<int64_t>(a) * A.H], kLogFloor) : 0.f;
    nl1 = a + 1 < sq.count ? fmaxf(ld[static_cast<int64_t>(a + 1) * A.H], kLogFloor) : 0.f;
    nc0 = a < sq.count ? cf[static_cast<int64_t>(a) * A.H] : 0.f;
    nc1 = a + 1 < sq.count ? cf[static_cast<int64_t>(a + 1) * A.H] : 0.f;
  };
  auto commit_decay = [&]() {
    double s = static_cast<double>(nl0) + static_cast<double>(nl1);
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const double p = __shfl_up_sync(0xffffffffu, s, o);
      if (lane >= o) s += p;
    }
    const double end = __shfl_sync(0xffffffffu, s, 31);
    const double l1 = s, l0 = s - static_cast<double>(nl1);
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const double l = j ? l1 : l0;
      const float hi = static_cast<float>(l), c = j ? nc1 : nc0;
      const int t = 2 * lane + j;
      lh_s[t] = hi;
      ll_s[t] = static_cast<float>(l - static_cast<double>(hi));
      c_s[t] = c;
      el_s[t] = expf(hi);
      w_s[t] = expf(static_cast<float>(end - l)) * c;
    }
    if (lane == 0) end_s[0] = expf(static_cast<float>(end));
  };

  // ---- the carried state into accumulators, its split copy into shared memory
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
  if (has_n)
    for (int i = tid; i < DKP; i += NT) n_s[i] = (!sq.fresh && i < dk) ? nst[i] : 0.f;

  load_rows(q_s, LDK, DKP, q, A.q_stride, dk, 0);
  load_rows(k_s, LDK, DKP, k, A.k_stride, dk, 0);
  load_rows(v_s, LDV, DVB, v, A.v_stride, ncol, 0);
  asm volatile("cp.async.commit_group;" ::: "memory");
  if (warp == 0) {
    fetch_decay(0);
    commit_decay();
  }

  // ldmatrix lane roles
  const int a_row = lane & 15, a_col = (lane >> 4) * 8;                                 // A [m][k], and B [k][n] transposed
  const int b_row = (lane & 7) + ((lane >> 4) << 3), b_col = ((lane >> 3) & 1) * 8;     // B [n][k], and A [k][m] transposed
  const uint32_t q_at = smem_addr(q_s + (wr * 16 + a_row) * LDK + a_col);
  const uint32_t k_at = smem_addr(k_s + b_row * LDK + b_col);
  const uint32_t sh_at = smem_addr(sh_s + a_row * LDV + wc * ON * 8 + a_col);
  const uint32_t sl_at = smem_addr(sl_s + a_row * LDV + wc * ON * 8 + a_col);
  const uint32_t v_at = smem_addr(v_s + a_row * LDV + wc * ON * 8 + a_col);
  const uint32_t vall_at = smem_addr(v_s + a_row * LDV + a_col);
  const uint32_t kt_at = smem_addr(k_s + b_row * LDK + srow + b_col);

  for (int t0 = 0; t0 < sq.count; t0 += kChunk) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    const bool more = t0 + kChunk < sq.count;
    if (warp == 0 && more) fetch_decay(t0 + kChunk);
    // ---- read-outs of the warp's 16 tokens
    float O[ON][4], P[8][4];
#pragma unroll
    for (int n = 0; n < ON; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) O[n][e] = 0.f;
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) P[n][e] = 0.f;
#pragma unroll 4
    for (int ks = 0; ks < DKP / 16; ++ks) {
      uint32_t a[4];
      ldsm4(a, q_at + ks * 32);
#pragma unroll
      for (int j = 0; j < 4; ++j)               // q k^T, key blocks up to the warp's own
        if (j <= wr) {
          uint32_t b[4];
          ldsm4(b, k_at + j * 16 * LDK * 2 + ks * 32);
          mma(P[2 * j], a, b[0], b[1]);
          mma(P[2 * j + 1], a, b[2], b[3]);
        }
#pragma unroll
      for (int j = 0; j < ON / 2; ++j) {        // q S
        uint32_t b[4];
        ldsm4t(b, sh_at + ks * 16 * LDV * 2 + j * 32);
        mma(O[2 * j], a, b[0], b[1]);
        mma(O[2 * j + 1], a, b[2], b[3]);
        ldsm4t(b, sl_at + ks * 16 * LDV * 2 + j * 32);
        mma(O[2 * j], a, b[0], b[1]);
        mma(O[2 * j + 1], a, b[2], b[3]);
      }
    }
    const int ra = wr * 16 + gr, rb = ra + 8;   // the thread's two tokens
    const float ela = el_s[ra], elb = el_s[rb];
#pragma unroll
    for (int n = 0; n < ON; ++n) {
      O[n][0] *= ela;
      O[n][1] *= ela;
      O[n][2] *= elb;
      O[n][3] *= elb;
    }
    const float lha = lh_s[ra], lla = ll_s[ra], lhb = lh_s[rb], llb = ll_s[rb];
    float suma = 0.f, sumb = 0.f;
#pragma unroll
    for (int n = 0; n < 8; ++n)
      if (n / 2 <= wr) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int s = n * 8 + 2 * tq + e;
          const float lh = lh_s[s], ll = ll_s[s], c = c_s[s];
          P[n][e] = s <= ra ? P[n][e] * (__expf((lha - lh) + (lla - ll)) * c) : 0.f;
          P[n][2 + e] = s <= rb ? P[n][2 + e] * (__expf((lhb - lh) + (llb - ll)) * c) : 0.f;
          suma += P[n][e];
          sumb += P[n][2 + e];
        }
      }
#pragma unroll
    for (int ks = 0; ks < 4; ++ks)              // weights times v, in two parts
      if (ks <= wr) {
        uint32_t hi[4], lo[4];
        split2(P[2 * ks][0], P[2 * ks][1], hi[0], lo[0]);
        split2(P[2 * ks][2], P[2 * ks][3], hi[1], lo[1]);
        split2(P[2 * ks + 1][0], P[2 * ks + 1][1], hi[2], lo[2]);
        split2(P[2 * ks + 1][2], P[2 * ks + 1][3], hi[3], lo[3]);
#pragma unroll
        for (int j = 0; j < ON / 2; ++j) {
          uint32_t b[4];
          ldsm4t(b, v_at + ks * 16 * LDV * 2 + j * 32);
          mma(O[2 * j], hi, b[0], b[1]);
          mma(O[2 * j + 1], hi, b[2], b[3]);
          mma(O[2 * j], lo, b[0], b[1]);
          mma(O[2 * j + 1], lo, b[2], b[3]);
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
        float x = O[n][2 * half] * A.q_scale, y = O[n][2 * half + 1] * A.q_scale;
        if (A.skip) {
          const __nv_bfloat162 vv = *reinterpret_cast<const __nv_bfloat162*>(v_s + r * LDV + c);
          x = fmaf(skip, __low2float(vv), x);
          y = fmaf(skip, __high2float(vv), y);
        }
        if (pair && c + 1 < ncol) *reinterpret_cast<float2*>(orow + c) = make_float2(x, y);
        else {
          if (c < ncol) orow[c] = x;
          if (c + 1 < ncol) orow[c + 1] = y;
        }
      }
    }
    if (has_n && wc == 0) {                     // n . q: the weights' row sums, and e^(l_t) q_t . n
      float na = 0.f, nb = 0.f;
      for (int i = 2 * tq; i < DKP; i += 8) {
        const float2 nn = *reinterpret_cast<const float2*>(n_s + i);
        const float2 qa = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(q_s + ra * LDK + i));
        const float2 qb = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(q_s + rb * LDK + i));
        na = fmaf(qa.x, nn.x, fmaf(qa.y, nn.y, na));
        nb = fmaf(qb.x, nn.x, fmaf(qb.y, nn.y, nb));
      }
      suma = fmaf(ela, na, suma);
      sumb = fmaf(elb, nb, sumb);
#pragma unroll
      for (int o = 1; o < 4; o <<= 1) {
        suma += __shfl_xor_sync(0xffffffffu, suma, o);
        sumb += __shfl_xor_sync(0xffffffffu, sumb, o);
      }
      if (tq == 0) {
        if (t0 + ra < sq.count) A.nq[static_cast<int64_t>(sq.tok0 + t0 + ra) * A.H + h] = suma * A.q_scale;
        if (t0 + rb < sq.count) A.nq[static_cast<int64_t>(sq.tok0 + t0 + rb) * A.H + h] = sumb * A.q_scale;
      }
    }
    __syncthreads();                            // q and the split state have been read by everyone
    if (more) {
      load_rows(q_s, LDK, DKP, q, A.q_stride, dk, t0 + kChunk);
      asm volatile("cp.async.commit_group;" ::: "memory");
    }
    // ---- the state past this chunk
    const float end = end_s[0];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < SN; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[m][n][e] *= end;
    float nsum[MT][2];
#pragma unroll
    for (int m = 0; m < MT; ++m) nsum[m][0] = nsum[m][1] = 0.f;
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      uint32_t hi[MT][4], lo[MT][4];
      const float2 w0 = *reinterpret_cast<const float2*>(w_s + ks * 16 + 2 * tq);
      const float2 w1 = *reinterpret_cast<const float2*>(w_s + ks * 16 + 8 + 2 * tq);
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        uint32_t a[4];
        ldsm4t(a, kt_at + ks * 16 * LDK * 2 + m * 32);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&a[e]));
          const float x = f.x * (e < 2 ? w0.x : w1.x), y = f.y * (e < 2 ? w0.y : w1.y);
          nsum[m][e & 1] += x + y;
          split2(x, y, hi[m][e], lo[m][e]);
        }
      }
#pragma unroll
      for (int j = 0; j < SN / 2; ++j) {
        uint32_t b[4];
        ldsm4t(b, vall_at + ks * 16 * LDV * 2 + j * 32);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          mma(S[m][2 * j], hi[m], b[0], b[1]);
          mma(S[m][2 * j + 1], hi[m], b[2], b[3]);
          mma(S[m][2 * j], lo[m], b[0], b[1]);
          mma(S[m][2 * j + 1], lo[m], b[2], b[3]);
        }
      }
    }
    if (more) publish_state();
    if (has_n) {
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          float x = nsum[m][half];
          x += __shfl_xor_sync(0xffffffffu, x, 1);
          x += __shfl_xor_sync(0xffffffffu, x, 2);
          const int r = srow + m * 16 + gr + half * 8;
          if (tq == 0) n_s[r] = fmaf(end, n_s[r], x);
        }
    }
    __syncthreads();                            // k, v and the decays have been read by everyone
    if (more) {
      load_rows(k_s, LDK, DKP, k, A.k_stride, dk, t0 + kChunk);
      load_rows(v_s, LDV, DVB, v, A.v_stride, ncol, t0 + kChunk);
      asm volatile("cp.async.commit_group;" ::: "memory");
      if (warp == 0) commit_decay();
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
  if (has_n)
    for (int i = tid; i < dk; i += NT) nst[i] = n_s[i];
}

}  // namespace
}  // namespace b200

using namespace b200;

extern "C" {

int b200_decay_chunk_scan_supported(int dk, int dv, int dtype) {
  return dtype == B200_DTYPE_BF16 && dk >= 1 && dk <= 256 && dv >= 1;
}

int b200_decay_chunk_scan(float* o, float* nq, const void* q, int64_t q_stride, const void* k, int64_t k_stride,
                          const void* v, int64_t v_stride, const float* log_decay, const float* coef, const float* skip,
                          float q_scale, float* state, float* nstate, const int32_t* seqs, int n_seqs, int H, int G, int dk,
                          int dv, int dtype, void* stream) {
  if (n_seqs < 0 || H <= 0 || G <= 0 || H % G || dk <= 0 || dv <= 0) return fail(B200_EINVAL, "b200_decay_chunk_scan: bad sizes");
  if (!b200_decay_chunk_scan_supported(dk, dv, dtype))
    return fail(B200_ESHAPE, "b200_decay_chunk_scan: dtype %d, key size %d not supported", dtype, dk);
  if (n_seqs == 0) return 0;
  if (!o || !q || !k || !v || !log_decay || !coef || !state || !seqs || (nstate && !nq))
    return fail(B200_EINVAL, "b200_decay_chunk_scan: null pointer");
  const int vec = dk % 8 == 0 && dv % 8 == 0 && q_stride % 8 == 0 && k_stride % 8 == 0 && v_stride % 8 == 0 && aligned16(q) &&
                  aligned16(k) && aligned16(v);
  const ChunkArgs A{o, nq, static_cast<const __nv_bfloat16*>(q), static_cast<const __nv_bfloat16*>(k),
                    static_cast<const __nv_bfloat16*>(v), q_stride, k_stride, v_stride, log_decay, coef, skip, q_scale, state,
                    nstate, reinterpret_cast<const ChunkSeq*>(seqs), H, G, dk, dv, vec};
  auto launch = [&](auto kern, size_t smem, int dvb, int nt) {
    cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    kern<<<dim3(n_seqs, H, (dv + dvb - 1) / dvb), nt, smem, static_cast<cudaStream_t>(stream)>>>(A);
  };
  const bool narrow = dv <= 32;
  if (dk <= 64) {
    if (narrow) launch(decay_chunk_scan_kernel<64, 32, 1>, ChunkShape<64, 32, 1>::kBytes, 32, 128);
    else launch(decay_chunk_scan_kernel<64, 64, 1>, ChunkShape<64, 64, 1>::kBytes, 64, 128);
  } else if (dk <= 128) {
    if (narrow) launch(decay_chunk_scan_kernel<128, 32, 1>, ChunkShape<128, 32, 1>::kBytes, 32, 128);
    else launch(decay_chunk_scan_kernel<128, 64, 1>, ChunkShape<128, 64, 1>::kBytes, 64, 128);
  } else {
    if (narrow) launch(decay_chunk_scan_kernel<256, 32, 2>, ChunkShape<256, 32, 2>::kBytes, 32, 256);
    else launch(decay_chunk_scan_kernel<256, 64, 2>, ChunkShape<256, 64, 2>::kBytes, 64, 256);
  }
  return check_launch("b200_decay_chunk_scan");
}

}  // extern "C"
