// Pieces for decoder designs whose recurrences keep a matrix per head and decay it by ONE number per token and head, and
// whose sublayers are pre-normed by a bounded elementwise function instead of a statistic:
//
//   dynamic tanh residual        x += y;  out = tanh(alpha x) * w + b, elementwise, so any residual update can emit the next
//                                sublayer's input (the routed feed-forward's weighted combine does too)
//   decayed outer-product state  S_t = d_t S_(t-1) + c_t k_t v_t^T,  o_t = S_t^T (q_scale q_t) [+ skip_h v_t], d and c one number
//                                per token and head; optionally the same recurrence without v (n_t = d_t n_(t-1) + c_t k_t) and
//                                its product n_t . q_t.  Two sources of (d, c):
//                                  capped exponential gates  log gates i, f behind a soft cap, a running maximum m:
//                                      m_t = max(f + m_(t-1), i), d = exp(f + m_(t-1) - m_t), c = exp(i - m_t)
//                                  step sizes                dt = softplus(z + bias), d = exp(-exp(A_log) dt), c = dt
//   read-out norms               o / max(|n.q|, exp(-m)) made unit-RMS per head, weighted, times sigmoid(gate); and
//                                y * silu(z) made unit-RMS in equal parts of the row, weighted
//   SiLU gated linear unit       silu(g) * u
//
// Every size and constant of a design is a parameter.  Gates, decays, maxima, state, norms and the residual are fp32
// whatever the storage dtype T is.
#include <algorithm>
#include <type_traits>

#include "../../include/b200_mixers.h"
#include "b200_common.cuh"

namespace b200 {
namespace {

template <typename F>
int recurrent_by_dtype(int dtype, const char* name, F&& f) {
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

__device__ __forceinline__ float sigmoid1(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus1(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

__device__ __forceinline__ float sum_over_block(float v, float* red) {   // every thread returns the total; red: 32 floats
  v = warp_sum(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  __syncthreads();
  if (lane == 0) red[warp] = v;
  __syncthreads();
  return warp_sum(lane < nw ? red[lane] : 0.f);
}

// four consecutive elements as fp32, and back
template <typename T>
__device__ __forceinline__ float4 load4(const T* p) {
  if constexpr (sizeof(T) == 4) {
    return *reinterpret_cast<const float4*>(p);
  } else {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const T* e = reinterpret_cast<const T*>(&raw);
    return make_float4(Cvt<T>::to_f32(e[0]), Cvt<T>::to_f32(e[1]), Cvt<T>::to_f32(e[2]), Cvt<T>::to_f32(e[3]));
  }
}
template <typename T>
__device__ __forceinline__ void store4(T* p, const float4& v) {
  if constexpr (sizeof(T) == 4) {
    *reinterpret_cast<float4*>(p) = v;
  } else {
    uint2 raw;
    T* e = reinterpret_cast<T*>(&raw);
    e[0] = Cvt<T>::from_f32(v.x);
    e[1] = Cvt<T>::from_f32(v.y);
    e[2] = Cvt<T>::from_f32(v.z);
    e[3] = Cvt<T>::from_f32(v.w);
    *reinterpret_cast<uint2*>(p) = raw;
  }
}

struct SeqSpan {
  int tok0;   // first packed row
  int count;  // tokens in this step
  int slot;   // state slot
  int fresh;  // 1: the sequence starts here (the carried state counts as zero)
};

// ---- dynamic tanh residual -------------------------------------------------------------------------------------------
struct DynTanh {
  const void* w;
  const void* b;
  float alpha;
};

template <typename T, typename Y, int V>
__global__ void __launch_bounds__(256)
residual_dyn_tanh_kernel(float* __restrict__ x, const Y* __restrict__ y, int64_t y_stride, const T* __restrict__ w,
                         const T* __restrict__ b, float alpha, T* __restrict__ out, int64_t rows, int width) {
  const int per_row = width / V;
  const int64_t total = rows * per_row;
  for (int64_t e = static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x; e < total;
       e += static_cast<int64_t>(gridDim.x) * blockDim.x) {
    const int64_t r = e / per_row;
    const int c = static_cast<int>(e - r * per_row) * V;
    if constexpr (V == 4) {
      float4 s = *reinterpret_cast<const float4*>(x + r * width + c);
      if (y) {
        const float4 a = load4(y + r * y_stride + c);
        s.x += a.x;
        s.y += a.y;
        s.z += a.z;
        s.w += a.w;
        *reinterpret_cast<float4*>(x + r * width + c) = s;
      }
      if (out) {
        const float4 g = load4(w + c), o = load4(b + c);
        store4(out + r * width + c, make_float4(fmaf(tanhf(alpha * s.x), g.x, o.x), fmaf(tanhf(alpha * s.y), g.y, o.y),
                                                fmaf(tanhf(alpha * s.z), g.z, o.z), fmaf(tanhf(alpha * s.w), g.w, o.w)));
      }
    } else {
      float s = x[r * width + c];
      if (y) {
        s += Cvt<Y>::to_f32(y[r * y_stride + c]);
        x[r * width + c] = s;
      }
      if (out) out[r * width + c] = Cvt<T>::from_f32(fmaf(tanhf(alpha * s), Cvt<T>::to_f32(w[c]), Cvt<T>::to_f32(b[c])));
    }
  }
}

// x += sum_k weights[k] * ys[where[k]] (k ascending) + sigmoid(gate) * shared;  out as above.  One CTA per token.
template <typename T, int V>
__global__ void __launch_bounds__(256)
expert_combine_dyn_tanh_kernel(float* __restrict__ x, const T* __restrict__ ys, const int64_t* __restrict__ where,
                               const float* __restrict__ weights, int top, const T* __restrict__ shared_rows,
                               const float* __restrict__ gate, int64_t gate_stride, const T* __restrict__ w,
                               const T* __restrict__ b, float alpha, T* __restrict__ out, int width) {
  const int64_t n = blockIdx.x;
  const float g = (shared_rows && gate) ? sigmoid1(gate[n * gate_stride]) : 1.0f;
  for (int c = threadIdx.x * V; c < width; c += blockDim.x * V) {
    if constexpr (V == 4) {
      float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int j = 0; j < top; ++j) {
        const float wt = weights[n * top + j];
        const float4 y = load4(ys + where[n * top + j] * width + c);
        a.x = fmaf(wt, y.x, a.x);
        a.y = fmaf(wt, y.y, a.y);
        a.z = fmaf(wt, y.z, a.z);
        a.w = fmaf(wt, y.w, a.w);
      }
      if (shared_rows) {
        const float4 y = load4(shared_rows + n * width + c);
        a.x = fmaf(g, y.x, a.x);
        a.y = fmaf(g, y.y, a.y);
        a.z = fmaf(g, y.z, a.z);
        a.w = fmaf(g, y.w, a.w);
      }
      float4 s = *reinterpret_cast<const float4*>(x + n * width + c);
      s.x += a.x;
      s.y += a.y;
      s.z += a.z;
      s.w += a.w;
      *reinterpret_cast<float4*>(x + n * width + c) = s;
      if (out) {
        const float4 q = load4(w + c), o = load4(b + c);
        store4(out + n * width + c, make_float4(fmaf(tanhf(alpha * s.x), q.x, o.x), fmaf(tanhf(alpha * s.y), q.y, o.y),
                                                fmaf(tanhf(alpha * s.z), q.z, o.z), fmaf(tanhf(alpha * s.w), q.w, o.w)));
      }
    } else {
      float a = 0.f;
      for (int j = 0; j < top; ++j) a = fmaf(weights[n * top + j], Cvt<T>::to_f32(ys[where[n * top + j] * width + c]), a);
      if (shared_rows) a = fmaf(g, Cvt<T>::to_f32(shared_rows[n * width + c]), a);
      const float s = x[n * width + c] + a;
      x[n * width + c] = s;
      if (out) out[n * width + c] = Cvt<T>::from_f32(fmaf(tanhf(alpha * s), Cvt<T>::to_f32(w[c]), Cvt<T>::to_f32(b[c])));
    }
  }
}

// ---- SiLU gated linear unit --------------------------------------------------------------------------------------------
template <typename T, int V>
__global__ void __launch_bounds__(256)
silu_glu_kernel(T* __restrict__ y, const T* __restrict__ gu, int64_t rows, int ff) {
  const int per_row = ff / V;
  const int64_t total = rows * per_row;
  for (int64_t e = static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x; e < total;
       e += static_cast<int64_t>(gridDim.x) * blockDim.x) {
    const int64_t r = e / per_row;
    const int c = static_cast<int>(e - r * per_row) * V;
    const T* row = gu + r * 2 * ff;
    if constexpr (V * sizeof(T) == 16) {
      int4 gr = *reinterpret_cast<const int4*>(row + c);
      const int4 ur = *reinterpret_cast<const int4*>(row + ff + c);
      T* g = reinterpret_cast<T*>(&gr);
      const T* u = reinterpret_cast<const T*>(&ur);
#pragma unroll
      for (int i = 0; i < V; ++i) {
        const float z = Cvt<T>::to_f32(g[i]);
        g[i] = Cvt<T>::from_f32(z * sigmoid1(z) * Cvt<T>::to_f32(u[i]));
      }
      *reinterpret_cast<int4*>(y + r * ff + c) = gr;
    } else {
      const float z = Cvt<T>::to_f32(row[c]);
      y[r * ff + c] = Cvt<T>::from_f32(z * sigmoid1(z) * Cvt<T>::to_f32(row[ff + c]));
    }
  }
}

// ---- where (d, c) come from --------------------------------------------------------------------------------------------
// kind 0: capped exponential gates.  a = input gate logits, b = forget gate logits (T, [n, H] with row stride z_stride), p0 /
// p1 their biases; kind 1: step sizes.  a = step logits, p0 = bias, p1 = A_log.  p0, p1 fp32 [H].
struct DecayGates {
  const void* a;
  const void* b;
  int64_t z_stride;
  const float* p0;
  const float* p1;
  float cap;
  int kind;
};

__device__ __forceinline__ float soft_cap(float z, float cap) { return cap * tanhf(z / cap); }

template <typename T>
__device__ __forceinline__ void gate_logs(const DecayGates& G, int64_t n, int h, float& i_log, float& f_log) {
  const float zi = Cvt<T>::to_f32(static_cast<const T*>(G.a)[n * G.z_stride + h]) + G.p0[h];
  const float zf = Cvt<T>::to_f32(static_cast<const T*>(G.b)[n * G.z_stride + h]) + G.p1[h];
  i_log = soft_cap(zi, G.cap);
  f_log = -softplus1(-soft_cap(zf, G.cap));
}

template <typename T>
__device__ __forceinline__ void step_size(const DecayGates& G, int64_t n, int h, float& log_d, float& c) {
  c = softplus1(Cvt<T>::to_f32(static_cast<const T*>(G.a)[n * G.z_stride + h]) + G.p0[h]);
  log_d = -expf(G.p1[h]) * c;
}

// (f, i) stands for m -> max(f + m, i); `first` is applied before `then`
__device__ __forceinline__ float2 max_plus(const float2& first, const float2& then) {
  return make_float2(first.x + then.x, fmaxf(then.x + first.y, then.y));
}

// Capped gates of a whole portion: one CTA per (sequence, head); 256 tokens at a time an inclusive scan of the max-plus
// maps gives every token's running maximum.  m_state [slots, H] is read (unless fresh: 0) and written back.
template <typename T>
__global__ void __launch_bounds__(256)
capped_gates_kernel(float* __restrict__ log_decay, float* __restrict__ coef, float* __restrict__ m_seq, DecayGates G,
                    float* __restrict__ m_state, const SeqSpan* __restrict__ seqs, int H) {
  __shared__ float2 part[8];
  __shared__ float last[8];
  __shared__ float carry;
  const SeqSpan sq = seqs[blockIdx.x];
  const int h = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  float* ms = m_state + static_cast<int64_t>(sq.slot) * H + h;
  float m0 = sq.fresh ? 0.f : *ms;
  for (int t0 = 0; t0 < sq.count; t0 += 256) {
    const int t = t0 + threadIdx.x;
    const bool in = t < sq.count;
    float i_log = -INFINITY, f_log = 0.f;
    if (in) gate_logs<T>(G, sq.tok0 + t, h, i_log, f_log);
    float2 s = make_float2(f_log, i_log);           // a token past the end is the identity map (0, -inf)
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float2 p = make_float2(__shfl_up_sync(0xffffffffu, s.x, o), __shfl_up_sync(0xffffffffu, s.y, o));
      if (lane >= o) s = max_plus(p, s);
    }
    if (lane == 31) part[warp] = s;
    __syncthreads();
    float start = m0;                               // the maximum before this warp's first token
    for (int w = 0; w < warp; ++w) start = fmaxf(part[w].x + start, part[w].y);
    const float m = fmaxf(s.x + start, s.y);
    if (lane == 31) last[warp] = m;
    float before = __shfl_up_sync(0xffffffffu, m, 1);
    if (threadIdx.x == 255) carry = m;
    __syncthreads();
    if (lane == 0) before = warp == 0 ? m0 : last[warp - 1];   // exactly the value the token before was given
    if (in) {
      const int64_t at = static_cast<int64_t>(sq.tok0 + t) * H + h;
      log_decay[at] = f_log + before - m;
      coef[at] = expf(i_log - m);
      m_seq[at] = m;
    }
    m0 = carry;
    __syncthreads();
  }
  if (threadIdx.x == 0) *ms = m0;
}

template <typename T>
__global__ void __launch_bounds__(256)
step_sizes_kernel(float* __restrict__ log_decay, float* __restrict__ coef, DecayGates G, int64_t n_tok, int H) {
  const int64_t total = n_tok * H;
  for (int64_t e = static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x; e < total;
       e += static_cast<int64_t>(gridDim.x) * blockDim.x) {
    const int64_t n = e / H;
    float d, c;
    step_size<T>(G, n, static_cast<int>(e - n * H), d, c);
    log_decay[e] = d;
    coef[e] = c;
  }
}

// ---- the scan: any portions, token by token ---------------------------------------------------------------------------
// One CTA per (sequence, head, 32 value columns).  Four adjacent lanes share a value column; lane r of the four keeps the
// state rows i = r, r + 4, ... of that column in registers for the whole portion.  kScanChunk tokens' inputs are staged in
// shared memory at a time, double buffered (q and c * k grouped by r so that a thread's rows are contiguous).  A fifth warp
// of the CTAs of the first columns runs the vector recurrence n when the design has one.
constexpr int kScanChunk = 8;
constexpr int kScanNT = 128;
constexpr int kScanCols = kScanNT / 4;

struct ScanArgs {
  float* o;            // [n, H, dv]
  float* nq;           // [n, H] or NULL
  const void* q;
  const void* k;
  const void* v;
  int64_t q_stride, k_stride, v_stride;
  const float* log_decay;  // [n, H]
  const float* coef;   // [n, H]
  const float* skip;   // [H] or NULL
  float q_scale;
  float* state;        // [slots, H, dk, dv]
  float* nstate;       // [slots, H, dk] or NULL
  const SeqSpan* seqs;
  int H, G, dk, dv;
};

template <typename T, int DK>
__global__ void __launch_bounds__(kScanNT + 32)
decay_scan_kernel(const ScanArgs A) {
  extern __shared__ __align__(16) float sc_sm[];
  constexpr int RW4 = DK / 4;
  constexpr int ROW = 2 * DK + kScanCols + 4;       // q | c k | v | d, padded to 16 bytes
  const SeqSpan sq = A.seqs[blockIdx.x];
  const int h = blockIdx.y, g = h / (A.H / A.G), dk = A.dk, dv = A.dv;
  const int tid = threadIdx.x;
  const bool main = tid < kScanNT;
  const bool side = !main && A.nstate != nullptr && blockIdx.z == 0;
  const int r = tid & 3, cl = (tid & (kScanNT - 1)) >> 2, lane = tid & 31;
  const int col0 = blockIdx.z * kScanCols, col = col0 + cl;
  const int ncol = min(kScanCols, dv - col0);
  float* st = A.state + (static_cast<int64_t>(sq.slot) * A.H + h) * dk * dv;
  float* nst = A.nstate ? A.nstate + (static_cast<int64_t>(sq.slot) * A.H + h) * dk : nullptr;
  const T* q = static_cast<const T*>(A.q) + static_cast<int64_t>(sq.tok0) * A.q_stride + static_cast<int64_t>(g) * dk;
  const T* k = static_cast<const T*>(A.k) + static_cast<int64_t>(sq.tok0) * A.k_stride + static_cast<int64_t>(g) * dk;
  const T* v = static_cast<const T*>(A.v) + static_cast<int64_t>(sq.tok0) * A.v_stride + static_cast<int64_t>(h) * dv + col0;
  const float* dec = A.log_decay + static_cast<int64_t>(sq.tok0) * A.H + h;
  const float* cof = A.coef + static_cast<int64_t>(sq.tok0) * A.H + h;
  const float skip = A.skip ? A.skip[h] : 0.f;
  float S[RW4];
  constexpr int NL = DK / 32;
  float N[NL];
#pragma unroll
  for (int j = 0; j < RW4; ++j) {
    const int i = 4 * j + r;
    S[j] = (main && !sq.fresh && i < dk && cl < ncol) ? st[static_cast<int64_t>(i) * dv + col] : 0.f;
  }
#pragma unroll
  for (int j = 0; j < NL; ++j) N[j] = (side && !sq.fresh && lane + 32 * j < dk) ? nst[lane + 32 * j] : 0.f;

  auto stage = [&](float* dst, int t0) {
    const int n_here = min(kScanChunk, sq.count - t0);
#pragma unroll 4
    for (int e = tid; e < n_here * DK; e += kScanNT + 32) {
      const int tt = e / DK, i = e % DK, at = (i & 3) * RW4 + (i >> 2);
      const int64_t t = t0 + tt;
      float* row = dst + tt * ROW;
      row[at] = i < dk ? Cvt<T>::to_f32(q[t * A.q_stride + i]) * A.q_scale : 0.f;
      row[DK + at] = i < dk ? Cvt<T>::to_f32(k[t * A.k_stride + i]) * cof[t * A.H] : 0.f;
    }
    for (int e = tid; e < n_here * kScanCols; e += kScanNT + 32) {
      const int tt = e / kScanCols, i = e % kScanCols;
      dst[tt * ROW + 2 * DK + i] = i < ncol ? Cvt<T>::to_f32(v[static_cast<int64_t>(t0 + tt) * A.v_stride + i]) : 0.f;
    }
    if (tid < n_here) dst[tid * ROW + 2 * DK + kScanCols] = expf(dec[static_cast<int64_t>(t0 + tid) * A.H]);
  };
  float* buf0 = sc_sm;
  float* buf1 = sc_sm + kScanChunk * ROW;
  stage(buf0, 0);
  __syncthreads();
  for (int t0 = 0; t0 < sq.count; t0 += kScanChunk) {
    const bool odd = (t0 / kScanChunk) & 1;
    const float* cur = odd ? buf1 : buf0;
    if (t0 + kScanChunk < sq.count) stage(odd ? buf0 : buf1, t0 + kScanChunk);
    const int n_here = min(kScanChunk, sq.count - t0);
    if (main) {
      for (int tt = 0; tt < n_here; ++tt) {
        const float* row = cur + tt * ROW;
        const float d = row[2 * DK + kScanCols], vc = row[2 * DK + cl];
        const float* qr = row + r * RW4;
        const float* kr = row + DK + r * RW4;
        float o0 = 0.f, o1 = 0.f;
#pragma unroll
        for (int j = 0; j < RW4; j += 4) {
          const float4 q4 = *reinterpret_cast<const float4*>(qr + j);
          const float4 k4 = *reinterpret_cast<const float4*>(kr + j);
          S[j] = fmaf(d, S[j], k4.x * vc);
          o0 = fmaf(S[j], q4.x, o0);
          S[j + 1] = fmaf(d, S[j + 1], k4.y * vc);
          o1 = fmaf(S[j + 1], q4.y, o1);
          S[j + 2] = fmaf(d, S[j + 2], k4.z * vc);
          o0 = fmaf(S[j + 2], q4.z, o0);
          S[j + 3] = fmaf(d, S[j + 3], k4.w * vc);
          o1 = fmaf(S[j + 3], q4.w, o1);
        }
        float o = o0 + o1;
        o += __shfl_xor_sync(0xffffffffu, o, 1);
        o += __shfl_xor_sync(0xffffffffu, o, 2);
        if (r == 0 && cl < ncol) A.o[(static_cast<int64_t>(sq.tok0 + t0 + tt) * A.H + h) * dv + col] = fmaf(skip, vc, o);
      }
    } else if (side) {
      for (int tt = 0; tt < n_here; ++tt) {
        const float* row = cur + tt * ROW;
        const float d = row[2 * DK + kScanCols];
        float a = 0.f;
#pragma unroll
        for (int j = 0; j < NL; ++j) {
          const int i = lane + 32 * j, at = (i & 3) * RW4 + (i >> 2);
          N[j] = fmaf(d, N[j], row[DK + at]);
          a = fmaf(N[j], row[at], a);
        }
        a = warp_sum(a);
        if (lane == 0) A.nq[static_cast<int64_t>(sq.tok0 + t0 + tt) * A.H + h] = a;
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int j = 0; j < RW4; ++j) {
    const int i = 4 * j + r;
    if (main && i < dk && cl < ncol) st[static_cast<int64_t>(i) * dv + col] = S[j];
  }
#pragma unroll
  for (int j = 0; j < NL; ++j)
    if (side && lane + 32 * j < dk) nst[lane + 32 * j] = N[j];
}

// ---- one token per sequence --------------------------------------------------------------------------------------------
// Bound by the state's bytes: every element is read and written once, as 16-byte accesses along the value columns.  One CTA
// per (sequence, head, LPR * V value columns): LPR lanes cover a row's columns, the CTA's 256 threads 256 / LPR rows at a
// time; partial read-outs meet in shared memory.  (d, c) are formed here from the gate logits; the running maximum is only
// READ from the state (every CTA of a head needs the old one) and handed on in m_seq: the read-out norm stores it.
struct StepArgs {
  float* o;
  float* nq;
  float* m_seq;
  const void* q;
  const void* k;
  const void* v;
  int64_t q_stride, k_stride, v_stride;
  DecayGates gates;
  const float* skip;
  float q_scale;
  float* state;
  float* nstate;
  const float* m_state;
  const SeqSpan* seqs;
  int H, G, dk, dv;
};

template <typename T, int V, int LPR>
__global__ void __launch_bounds__(256)
decay_step_kernel(const StepArgs A) {
  extern __shared__ __align__(16) float sp_sm[];     // q[dk] | c k[dk] | partial read-outs [256][V]
  __shared__ float red[32];
  constexpr int RPI = 256 / LPR;                     // rows per iteration
  const SeqSpan sq = A.seqs[blockIdx.x];
  const int h = blockIdx.y, g = h / (A.H / A.G), dk = A.dk, dv = A.dv, tid = threadIdx.x;
  const int64_t n = sq.tok0;
  float* qs = sp_sm;
  float* ks = sp_sm + dk;
  float* ps = sp_sm + ((2 * dk + 3) & ~3);
  float d, c;
  if (A.gates.kind == 0) {
    float i_log, f_log;
    gate_logs<T>(A.gates, n, h, i_log, f_log);
    const float m0 = sq.fresh ? 0.f : A.m_state[static_cast<int64_t>(sq.slot) * A.H + h];
    const float m = fmaxf(f_log + m0, i_log);
    d = expf(f_log + m0 - m);
    c = expf(i_log - m);
    if (blockIdx.z == 0 && tid == 0) A.m_seq[n * A.H + h] = m;
  } else {
    step_size<T>(A.gates, n, h, d, c);
    d = expf(d);
  }
  const T* q = static_cast<const T*>(A.q) + n * A.q_stride + static_cast<int64_t>(g) * dk;
  const T* k = static_cast<const T*>(A.k) + n * A.k_stride + static_cast<int64_t>(g) * dk;
  for (int i = tid; i < dk; i += 256) {
    qs[i] = Cvt<T>::to_f32(q[i]) * A.q_scale;
    ks[i] = Cvt<T>::to_f32(k[i]) * c;
  }
  const int lr = tid % LPR, row0 = tid / LPR;
  const int col = (blockIdx.z * LPR + lr) * V;
  const bool has = col < dv;
  const T* vp = static_cast<const T*>(A.v) + n * A.v_stride + static_cast<int64_t>(h) * dv + col;
  float vv[V], acc[V];
#pragma unroll
  for (int u = 0; u < V; ++u) {
    vv[u] = has ? Cvt<T>::to_f32(vp[u]) : 0.f;
    acc[u] = 0.f;
  }
  __syncthreads();
  float* st = A.state + (static_cast<int64_t>(sq.slot) * A.H + h) * dk * dv + col;
  if (has) {
    constexpr int U = 4;                             // rows in flight per thread
    for (int i0 = row0; i0 < dk; i0 += U * RPI) {
      float s[U][V];
#pragma unroll
      for (int j = 0; j < U; ++j) {
        const int i = i0 + j * RPI;
#pragma unroll
        for (int u = 0; u < V; ++u) s[j][u] = 0.f;
        if (i < dk && !sq.fresh) {
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
#pragma unroll
      for (int j = 0; j < U; ++j) {
        const int i = i0 + j * RPI;
        if (i < dk) {
          const float ki = ks[i], qi = qs[i];
#pragma unroll
          for (int u = 0; u < V; ++u) {
            s[j][u] = fmaf(d, s[j][u], ki * vv[u]);
            acc[u] = fmaf(s[j][u], qi, acc[u]);
          }
          if constexpr (V == 4)
            *reinterpret_cast<float4*>(st + static_cast<int64_t>(i) * dv) = make_float4(s[j][0], s[j][1], s[j][2], s[j][3]);
          else
            st[static_cast<int64_t>(i) * dv] = s[j][0];
        }
      }
    }
  }
#pragma unroll
  for (int u = 0; u < V; ++u) ps[tid * V + u] = acc[u];
  __syncthreads();
  const float skip = A.skip ? A.skip[h] : 0.f;
  const int c0 = blockIdx.z * LPR * V;
  for (int e = tid; e < LPR * V; e += 256) {
    if (c0 + e >= dv) continue;
    float o = 0.f;
    for (int rr = 0; rr < RPI; ++rr) o += ps[rr * LPR * V + e];
    A.o[(n * A.H + h) * dv + c0 + e] =
        fmaf(skip, Cvt<T>::to_f32(static_cast<const T*>(A.v)[n * A.v_stride + static_cast<int64_t>(h) * dv + c0 + e]), o);
  }
  if (A.nstate != nullptr && blockIdx.z == 0) {
    float* nst = A.nstate + (static_cast<int64_t>(sq.slot) * A.H + h) * dk;
    float a = 0.f;
    for (int i = tid; i < dk; i += 256) {
      const float x = fmaf(d, sq.fresh ? 0.f : nst[i], ks[i]);
      nst[i] = x;
      a = fmaf(x, qs[i], a);
    }
    a = sum_over_block(a, red);
    if (tid == 0) A.nq[n * A.H + h] = a;
  }
}

// ---- read-out norms ----------------------------------------------------------------------------------------------------
// One warp per (token, head): o / (max(|nq|, exp(-m)) + floor), unit RMS, times w[h * dv + i], times sigmoid(gate).  When
// m_state is given (steps of one token per sequence, row n = sequence n), the token's running maximum becomes the carried
// one.
template <typename T, bool VEC>
__global__ void __launch_bounds__(256)
normalized_head_out_kernel(T* __restrict__ out, int64_t out_stride, const float* __restrict__ o, const float* __restrict__ nq,
                           const float* __restrict__ m_seq, float floor_, const T* __restrict__ w, const T* __restrict__ gate,
                           int64_t gate_stride, float eps, float* __restrict__ m_state, const SeqSpan* __restrict__ seqs,
                           int64_t rows, int H, int dv) {
  const int64_t row = static_cast<int64_t>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  if (row >= rows) return;
  const int lane = threadIdx.x & 31;
  const int64_t n = row / H;
  const int h = static_cast<int>(row - n * H);
  const float* x = o + row * dv;
  const T* gr = gate + n * gate_stride + static_cast<int64_t>(h) * dv;
  const T* wr = w + static_cast<int64_t>(h) * dv;
  T* dst = out + n * out_stride + static_cast<int64_t>(h) * dv;
  const float m = m_seq[row];
  const float r = 1.0f / (fmaxf(fabsf(nq[row]), expf(-m)) + floor_);
  float ss = 0.f;
  if constexpr (VEC) {            // dv a multiple of 4, at most 512: the row stays in registers
    float4 y[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int i = 4 * (lane + 32 * j);
      y[j] = i < dv ? *reinterpret_cast<const float4*>(x + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      y[j].x *= r;
      y[j].y *= r;
      y[j].z *= r;
      y[j].w *= r;
      ss = fmaf(y[j].x, y[j].x, fmaf(y[j].y, y[j].y, fmaf(y[j].z, y[j].z, fmaf(y[j].w, y[j].w, ss))));
    }
    const float inv = rsqrtf(warp_sum(ss) / static_cast<float>(dv) + eps);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int i = 4 * (lane + 32 * j);
      if (i >= dv) break;
      const float4 g = load4(gr + i), ww = load4(wr + i);
      store4(dst + i, make_float4(y[j].x * inv * ww.x * sigmoid1(g.x), y[j].y * inv * ww.y * sigmoid1(g.y),
                                  y[j].z * inv * ww.z * sigmoid1(g.z), y[j].w * inv * ww.w * sigmoid1(g.w)));
    }
  } else {
    for (int i = lane; i < dv; i += 32) {
      const float y = x[i] * r;
      ss = fmaf(y, y, ss);
    }
    const float inv = rsqrtf(warp_sum(ss) / static_cast<float>(dv) + eps);
    for (int i = lane; i < dv; i += 32)
      dst[i] = Cvt<T>::from_f32(x[i] * r * inv * Cvt<T>::to_f32(wr[i]) * sigmoid1(Cvt<T>::to_f32(gr[i])));
  }
  if (m_state != nullptr && lane == 0) m_state[static_cast<int64_t>(seqs[n].slot) * H + h] = m;
}

// One CTA per (token, part): y * silu(z) over the part's columns, unit RMS, times w.  V columns per access.
template <typename T, int V>
__global__ void __launch_bounds__(256)
gated_part_norm_kernel(T* __restrict__ out, const float* __restrict__ y, const T* __restrict__ z, int64_t z_stride,
                       const T* __restrict__ w, float eps, int inner, int part) {
  extern __shared__ __align__(16) float gn_row[];
  __shared__ float red[32];
  const int64_t n = blockIdx.x;
  const int c0 = blockIdx.y * part;
  const float* yr = y + n * inner + c0;
  const T* zr = z + n * z_stride + c0;
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < part; i += blockDim.x * V) {
    if constexpr (V == 4) {
      const float4 g = load4(zr + i);
      float4 v = *reinterpret_cast<const float4*>(yr + i);
      v.x *= g.x * sigmoid1(g.x);
      v.y *= g.y * sigmoid1(g.y);
      v.z *= g.z * sigmoid1(g.z);
      v.w *= g.w * sigmoid1(g.w);
      *reinterpret_cast<float4*>(gn_row + i) = v;
      ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
    } else {
      const float g = Cvt<T>::to_f32(zr[i]);
      const float v = yr[i] * (g * sigmoid1(g));
      gn_row[i] = v;
      ss = fmaf(v, v, ss);
    }
  }
  const float inv = rsqrtf(sum_over_block(ss, red) / static_cast<float>(part) + eps);
  for (int i = threadIdx.x * V; i < part; i += blockDim.x * V) {     // every thread reads back what it wrote
    if constexpr (V == 4) {
      const float4 v = *reinterpret_cast<const float4*>(gn_row + i), ww = load4(w + c0 + i);
      store4(out + n * inner + c0 + i, make_float4(v.x * inv * ww.x, v.y * inv * ww.y, v.z * inv * ww.z, v.w * inv * ww.w));
    } else {
      out[n * inner + c0 + i] = Cvt<T>::from_f32(gn_row[i] * inv * Cvt<T>::to_f32(w[c0 + i]));
    }
  }
}

}  // namespace
}  // namespace b200

using namespace b200;

extern "C" {

int b200_residual_dyn_tanh(float* x, const void* y, int64_t y_stride, int y_is_f32, const void* w, const void* b, float alpha,
                           void* out, int64_t rows, int width, int dtype, void* stream) {
  if (rows < 0 || width <= 0 || (y && y_stride < width)) return fail(B200_EINVAL, "b200_residual_dyn_tanh: bad sizes");
  if (rows == 0 || (!y && !out)) return 0;
  if (!x || (out && (!w || !b))) return fail(B200_EINVAL, "b200_residual_dyn_tanh: null pointer");
  const bool vec = width % 4 == 0 && (!y || y_stride % 4 == 0) && aligned16(x) && aligned16(y) && aligned16(w) &&
                   aligned16(b) && aligned16(out);
  const int64_t items = rows * (vec ? width / 4 : width);
  const unsigned grid = static_cast<unsigned>(std::min<int64_t>((items + 255) / 256, kNumSMs * 16));
  return recurrent_by_dtype(dtype, "b200_residual_dyn_tanh", [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    auto launch = [&](auto kern, auto* yp) {
      kern<<<grid, 256, 0, static_cast<cudaStream_t>(stream)>>>(x, yp, y_stride, static_cast<const T*>(w),
                                                                static_cast<const T*>(b), alpha, static_cast<T*>(out), rows,
                                                                width);
    };
    if (y_is_f32) {
      const float* yp = static_cast<const float*>(y);
      if (vec) launch(residual_dyn_tanh_kernel<T, float, 4>, yp);
      else launch(residual_dyn_tanh_kernel<T, float, 1>, yp);
    } else {
      const T* yp = static_cast<const T*>(y);
      if (vec) launch(residual_dyn_tanh_kernel<T, T, 4>, yp);
      else launch(residual_dyn_tanh_kernel<T, T, 1>, yp);
    }
    return check_launch("b200_residual_dyn_tanh");
  });
}

int b200_expert_combine_dyn_tanh(float* x, const void* ys, const int64_t* where, const float* weights, int top,
                                 const void* shared_rows, const float* shared_gate, int64_t gate_stride, const void* w,
                                 const void* b, float alpha, void* out, int64_t n_tok, int width, int dtype, void* stream) {
  if (n_tok < 0 || top < 0 || width <= 0) return fail(B200_EINVAL, "b200_expert_combine_dyn_tanh: bad sizes");
  if (n_tok == 0) return 0;
  if (!x || (top > 0 && (!ys || !where || !weights)) || (out && (!w || !b)))
    return fail(B200_EINVAL, "b200_expert_combine_dyn_tanh: null pointer");
  const bool vec = width % 4 == 0 && aligned16(x) && aligned16(ys) && aligned16(shared_rows) && aligned16(w) &&
                   aligned16(b) && aligned16(out);
  const int per = vec ? width / 4 : width;
  const int nt = per <= 64 ? 64 : (per <= 128 ? 128 : 256);
  return recurrent_by_dtype(dtype, "b200_expert_combine_dyn_tanh", [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    auto launch = [&](auto kern) {
      kern<<<static_cast<unsigned>(n_tok), nt, 0, static_cast<cudaStream_t>(stream)>>>(
          x, static_cast<const T*>(ys), where, weights, top, static_cast<const T*>(shared_rows), shared_gate, gate_stride,
          static_cast<const T*>(w), static_cast<const T*>(b), alpha, static_cast<T*>(out), width);
    };
    if (vec) launch(expert_combine_dyn_tanh_kernel<T, 4>);
    else launch(expert_combine_dyn_tanh_kernel<T, 1>);
    return check_launch("b200_expert_combine_dyn_tanh");
  });
}

int b200_silu_glu(void* y, const void* gu, int64_t rows, int ff, int dtype, void* stream) {
  if (rows < 0 || ff <= 0) return fail(B200_EINVAL, "b200_silu_glu: bad sizes");
  if (rows == 0) return 0;
  if (!y || !gu) return fail(B200_EINVAL, "b200_silu_glu: null pointer");
  return recurrent_by_dtype(dtype, "b200_silu_glu", [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    constexpr int V = 16 / sizeof(T);
    const bool vec = ff % V == 0 && aligned16(y) && aligned16(gu);
    const int64_t items = rows * (vec ? ff / V : ff);
    const unsigned grid = static_cast<unsigned>(std::min<int64_t>((items + 255) / 256, kNumSMs * 16));
    auto s = static_cast<cudaStream_t>(stream);
    if (vec) silu_glu_kernel<T, V><<<grid, 256, 0, s>>>(static_cast<T*>(y), static_cast<const T*>(gu), rows, ff);
    else silu_glu_kernel<T, 1><<<grid, 256, 0, s>>>(static_cast<T*>(y), static_cast<const T*>(gu), rows, ff);
    return check_launch("b200_silu_glu");
  });
}

int b200_capped_gates(float* log_decay, float* coef, float* m_seq, const void* zi, const void* zf, int64_t z_stride,
                      const float* bias_i, const float* bias_f, float cap, float* m_state, const int32_t* seqs, int n_seqs,
                      int H, int dtype, void* stream) {
  if (n_seqs < 0 || H <= 0 || !(cap > 0.f)) return fail(B200_EINVAL, "b200_capped_gates: bad sizes");
  if (n_seqs == 0) return 0;
  if (!log_decay || !coef || !m_seq || !zi || !zf || !bias_i || !bias_f || !m_state || !seqs)
    return fail(B200_EINVAL, "b200_capped_gates: null pointer");
  const DecayGates G{zi, zf, z_stride, bias_i, bias_f, cap, 0};
  return recurrent_by_dtype(dtype, "b200_capped_gates", [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    capped_gates_kernel<T><<<dim3(n_seqs, H), 256, 0, static_cast<cudaStream_t>(stream)>>>(
        log_decay, coef, m_seq, G, m_state, reinterpret_cast<const SeqSpan*>(seqs), H);
    return check_launch("b200_capped_gates");
  });
}

int b200_step_sizes(float* log_decay, float* coef, const void* z, int64_t z_stride, const float* bias, const float* a_log,
                    int64_t n_tok, int H, int dtype, void* stream) {
  if (n_tok < 0 || H <= 0) return fail(B200_EINVAL, "b200_step_sizes: bad sizes");
  if (n_tok == 0) return 0;
  if (!log_decay || !coef || !z || !bias || !a_log) return fail(B200_EINVAL, "b200_step_sizes: null pointer");
  const DecayGates G{z, nullptr, z_stride, bias, a_log, 1.f, 1};
  const unsigned grid = static_cast<unsigned>(std::min<int64_t>((n_tok * H + 255) / 256, kNumSMs * 16));
  return recurrent_by_dtype(dtype, "b200_step_sizes", [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    step_sizes_kernel<T><<<grid, 256, 0, static_cast<cudaStream_t>(stream)>>>(log_decay, coef, G, n_tok, H);
    return check_launch("b200_step_sizes");
  });
}

int b200_decay_scan(float* o, float* nq, const void* q, int64_t q_stride, const void* k, int64_t k_stride, const void* v,
                    int64_t v_stride, const float* log_decay, const float* coef, const float* skip, float q_scale, float* state,
                    float* nstate, const int32_t* seqs, int n_seqs, int H, int G, int dk, int dv, int dtype, void* stream) {
  if (n_seqs < 0 || H <= 0 || G <= 0 || H % G || dk <= 0 || dv <= 0) return fail(B200_EINVAL, "b200_decay_scan: bad sizes");
  if (dk > 512) return fail(B200_ESHAPE, "b200_decay_scan: key size %d beyond 512", dk);
  if (n_seqs == 0) return 0;
  if (!o || !q || !k || !v || !log_decay || !coef || !state || !seqs || (nstate && !nq))
    return fail(B200_EINVAL, "b200_decay_scan: null pointer");
  const int dkt = dk <= 32 ? 32 : (dk <= 64 ? 64 : (dk <= 128 ? 128 : (dk <= 256 ? 256 : 512)));
  const size_t smem = sizeof(float) * 2 * kScanChunk * (2 * static_cast<size_t>(dkt) + kScanCols + 4);
  const dim3 grid(n_seqs, H, (dv + kScanCols - 1) / kScanCols);
  const ScanArgs A{o, nq, q, k, v, q_stride, k_stride, v_stride, log_decay, coef, skip, q_scale, state, nstate,
                   reinterpret_cast<const SeqSpan*>(seqs), H, G, dk, dv};
  return recurrent_by_dtype(dtype, "b200_decay_scan", [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    auto launch = [&](auto kern) {
      if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
      kern<<<grid, kScanNT + 32, smem, static_cast<cudaStream_t>(stream)>>>(A);
    };
    if (dkt == 32) launch(decay_scan_kernel<T, 32>);
    else if (dkt == 64) launch(decay_scan_kernel<T, 64>);
    else if (dkt == 128) launch(decay_scan_kernel<T, 128>);
    else if (dkt == 256) launch(decay_scan_kernel<T, 256>);
    else launch(decay_scan_kernel<T, 512>);
    return check_launch("b200_decay_scan");
  });
}

int b200_decay_step(float* o, float* nq, float* m_seq, const void* q, int64_t q_stride, const void* k, int64_t k_stride,
                    const void* v, int64_t v_stride, int gate_kind, const void* za, const void* zb, int64_t z_stride,
                    const float* p0, const float* p1, float cap, const float* skip, float q_scale, float* state,
                    float* nstate, const float* m_state, const int32_t* seqs, int n_seqs, int H, int G, int dk, int dv,
                    int dtype, void* stream) {
  if (n_seqs < 0 || H <= 0 || G <= 0 || H % G || dk <= 0 || dv <= 0 || gate_kind < 0 || gate_kind > 1)
    return fail(B200_EINVAL, "b200_decay_step: bad sizes");
  if (n_seqs == 0) return 0;
  if (!o || !q || !k || !v || !za || !p0 || !p1 || !state || !seqs || (nstate && !nq) ||
      (gate_kind == 0 && (!zb || !m_state || !m_seq || !(cap > 0.f))))
    return fail(B200_EINVAL, "b200_decay_step: null pointer");
  const size_t smem = sizeof(float) * ((2 * static_cast<size_t>(dk) + 3) / 4 * 4 + 256 * 4);
  if (smem > 200 * 1024) return fail(B200_ESHAPE, "b200_decay_step: key size %d too large", dk);
  const StepArgs A{o, nq, m_seq, q, k, v, q_stride, k_stride, v_stride,
                   DecayGates{za, zb, z_stride, p0, p1, cap, gate_kind}, skip, q_scale, state, nstate, m_state,
                   reinterpret_cast<const SeqSpan*>(seqs), H, G, dk, dv};
  return recurrent_by_dtype(dtype, "b200_decay_step", [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    auto launch = [&](auto kern, int cols) {
      if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
      kern<<<dim3(n_seqs, H, (dv + cols - 1) / cols), 256, smem, static_cast<cudaStream_t>(stream)>>>(A);
    };
    if (dv % 4 == 0 && aligned16(state)) {
      if (dv <= 32) launch(decay_step_kernel<T, 4, 8>, 32);
      else if (dv <= 64) launch(decay_step_kernel<T, 4, 16>, 64);
      else launch(decay_step_kernel<T, 4, 32>, 128);
    } else {
      launch(decay_step_kernel<T, 1, 32>, 32);
    }
    return check_launch("b200_decay_step");
  });
}

int b200_normalized_head_out(void* out, int64_t out_stride, const float* o, const float* nq, const float* m_seq, float floor_,
                             const void* w, const void* gate, int64_t gate_stride, float eps, float* m_state,
                             const int32_t* seqs, int64_t n_tok, int H, int dv, int dtype, void* stream) {
  if (n_tok < 0 || H <= 0 || dv <= 0) return fail(B200_EINVAL, "b200_normalized_head_out: bad sizes");
  if (n_tok == 0) return 0;
  if (!out || !o || !nq || !m_seq || !w || !gate || (m_state && !seqs))
    return fail(B200_EINVAL, "b200_normalized_head_out: null pointer");
  const int64_t rows = n_tok * H;
  return recurrent_by_dtype(dtype, "b200_normalized_head_out", [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    const bool vec = dv % 4 == 0 && dv <= 512 && gate_stride % 4 == 0 && out_stride % 4 == 0 && aligned16(o) && aligned16(w) &&
                     aligned16(gate) && aligned16(out);
    auto launch = [&](auto kern) {
      kern<<<static_cast<unsigned>((rows + 7) / 8), 256, 0, static_cast<cudaStream_t>(stream)>>>(
          static_cast<T*>(out), out_stride, o, nq, m_seq, floor_, static_cast<const T*>(w), static_cast<const T*>(gate),
          gate_stride, eps, m_state, reinterpret_cast<const SeqSpan*>(seqs), rows, H, dv);
    };
    if (vec) launch(normalized_head_out_kernel<T, true>);
    else launch(normalized_head_out_kernel<T, false>);
    return check_launch("b200_normalized_head_out");
  });
}

int b200_gated_part_norm(void* out, const float* y, const void* z, int64_t z_stride, const void* w, float eps, int64_t n_tok,
                         int inner, int parts, int dtype, void* stream) {
  if (n_tok < 0 || inner <= 0 || parts <= 0 || inner % parts) return fail(B200_EINVAL, "b200_gated_part_norm: bad sizes");
  if (n_tok == 0) return 0;
  if (!out || !y || !z || !w) return fail(B200_EINVAL, "b200_gated_part_norm: null pointer");
  const int part = inner / parts;
  const size_t smem = sizeof(float) * static_cast<size_t>(part);
  if (smem > 200 * 1024 || parts > 65535) return fail(B200_ESHAPE, "b200_gated_part_norm: %d parts of %d", parts, part);
  return recurrent_by_dtype(dtype, "b200_gated_part_norm", [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    const bool vec = part % 4 == 0 && z_stride % 4 == 0 && aligned16(y) && aligned16(z) && aligned16(w) && aligned16(out);
    const int per = vec ? part / 4 : part;
    const int nt = per <= 32 ? 32 : (per <= 64 ? 64 : (per <= 128 ? 128 : 256));
    auto launch = [&](auto kern) {
      if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
      kern<<<dim3(static_cast<unsigned>(n_tok), parts), nt, smem, static_cast<cudaStream_t>(stream)>>>(
          static_cast<T*>(out), y, static_cast<const T*>(z), z_stride, static_cast<const T*>(w), eps, inner, part);
    };
    if (vec) launch(gated_part_norm_kernel<T, 4>);
    else launch(gated_part_norm_kernel<T, 1>);
    return check_launch("b200_gated_part_norm");
  });
}

}  // extern "C"
