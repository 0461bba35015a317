// Pieces for decoder designs with a per-channel selective state space and sublayers normed on both sides:
//
//   sandwich residual        x += s * ls * w * y * rsqrt(mean(y^2) + eps);  out = w_next * x * rsqrt(mean(x^2) + eps_next): the
//                            post-norm of one sublayer and the pre-norm of the next in one pass over the row
//   gated linear unit        gelu_tanh(g) * u
//   selective scan           per channel c and state n, with dt = softplus(z + bias) and rates A < 0:
//                              S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n;   y_c = sum_n S[c, n] C_n + D_c x_c
//                            and out = gain * y * silu(gate), for portions of any length or one token per sequence
//
// Every size and constant is a parameter.  Step sizes, exponentials, state, read-outs, norms and the residual are fp32 whatever
// the storage dtype T is.
#include <algorithm>
#include <type_traits>

#include "../../include/b200_mixers.h"
#include "b200_common.cuh"

namespace b200 {
namespace {

template <typename F>
int selective_by_dtype(int dtype, const char* name, F&& f) {
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

__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

template <typename T, int V>
__device__ __forceinline__ void load_vec(float (&d)[V], const T* p) {
  if constexpr (V == 1) {
    d[0] = Cvt<T>::to_f32(p[0]);
  } else {
    constexpr int E = 16 / sizeof(T);
#pragma unroll
    for (int j = 0; j < V / E; ++j) {
      const int4 raw = *reinterpret_cast<const int4*>(p + j * E);
      const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
      for (int i = 0; i < E; ++i) d[j * E + i] = Cvt<T>::to_f32(e[i]);
    }
  }
}
template <typename T, int V>
__device__ __forceinline__ void store_vec(T* p, const float (&d)[V]) {
  if constexpr (V == 1) {
    p[0] = Cvt<T>::from_f32(d[0]);
  } else {
    constexpr int E = 16 / sizeof(T);
#pragma unroll
    for (int j = 0; j < V / E; ++j) {
      int4 raw;
      T* e = reinterpret_cast<T*>(&raw);
#pragma unroll
      for (int i = 0; i < E; ++i) e[i] = Cvt<T>::from_f32(d[j * E + i]);
      *reinterpret_cast<int4*>(p + j * E) = raw;
    }
  }
}

// ---- post-norm, residual, pre-norm -------------------------------------------------------------------------------------
constexpr int kSandNT = 128;

__device__ __forceinline__ float sand_sum(float v, float* red) {   // red: 4 floats of its own per call
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  return (red[0] + red[1]) + (red[2] + red[3]);
}

struct SandArgs {
  float* x;
  const void* y;
  int64_t y_stride;
  float sign;
  const void* w;
  const void* ls;
  float eps;
  const void* w_next;
  void* out;
  float eps_next;
  int width;
};

// A row's numbers stay in registers: NV runs of V consecutive elements per thread (V = 8, or 1 for widths off the 16-byte grid).
template <typename T, typename Y, int V, int NV>
__global__ void __launch_bounds__(kSandNT)
sandwich_residual_kernel(const SandArgs A) {
  __shared__ float red[8];
  const int64_t n = blockIdx.x;
  const int width = A.width;
  const Y* yr = static_cast<const Y*>(A.y) + n * A.y_stride;
  float* xr = A.x + n * width;
  const T* w = static_cast<const T*>(A.w);
  const T* ls = static_cast<const T*>(A.ls);
  float y[NV][V], x[NV][V];
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const int c = (j * kSandNT + threadIdx.x) * V;
    if (c < width) {
      load_vec<Y, V>(y[j], yr + c);
      load_vec<float, V>(x[j], xr + c);
#pragma unroll
      for (int i = 0; i < V; ++i) ss = fmaf(y[j][i], y[j][i], ss);
    }
  }
  const float inv = A.sign * rsqrtf(sand_sum(ss, red) / static_cast<float>(width) + A.eps);
  float sx = 0.f;
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const int c = (j * kSandNT + threadIdx.x) * V;
    if (c < width) {
      float g[V], s[V];
      load_vec<T, V>(g, w + c);
      if (ls) load_vec<T, V>(s, ls + c);
#pragma unroll
      for (int i = 0; i < V; ++i) {
        float f = y[j][i] * inv * g[i];
        if (ls) f *= s[i];
        x[j][i] += f;
        sx = fmaf(x[j][i], x[j][i], sx);
      }
      store_vec<float, V>(xr + c, x[j]);
    }
  }
  if (A.out == nullptr) return;
  const float inx = rsqrtf(sand_sum(sx, red + 4) / static_cast<float>(width) + A.eps_next);
  const T* wn = static_cast<const T*>(A.w_next);
  T* out = static_cast<T*>(A.out) + n * width;
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const int c = (j * kSandNT + threadIdx.x) * V;
    if (c < width) {
      float g[V];
      load_vec<T, V>(g, wn + c);
#pragma unroll
      for (int i = 0; i < V; ++i) g[i] *= x[j][i] * inx;
      store_vec<T, V>(out + c, g);
    }
  }
}

// Any width: the row of y, then of x, in shared memory.
template <typename T, typename Y>
__global__ void __launch_bounds__(kSandNT)
sandwich_residual_any_kernel(const SandArgs A) {
  extern __shared__ float sand_row[];
  __shared__ float red[8];
  const int64_t n = blockIdx.x;
  const int width = A.width;
  const Y* yr = static_cast<const Y*>(A.y) + n * A.y_stride;
  float* xr = A.x + n * width;
  const T* w = static_cast<const T*>(A.w);
  const T* ls = static_cast<const T*>(A.ls);
  float ss = 0.f;
  for (int i = threadIdx.x; i < width; i += kSandNT) {
    const float v = Cvt<Y>::to_f32(yr[i]);
    sand_row[i] = v;
    ss = fmaf(v, v, ss);
  }
  const float inv = A.sign * rsqrtf(sand_sum(ss, red) / static_cast<float>(width) + A.eps);
  float sx = 0.f;
  for (int i = threadIdx.x; i < width; i += kSandNT) {
    float f = sand_row[i] * inv * Cvt<T>::to_f32(w[i]);
    if (ls) f *= Cvt<T>::to_f32(ls[i]);
    const float v = xr[i] + f;
    xr[i] = v;
    sand_row[i] = v;
    sx = fmaf(v, v, sx);
  }
  if (A.out == nullptr) return;
  const float inx = rsqrtf(sand_sum(sx, red + 4) / static_cast<float>(width) + A.eps_next);
  const T* wn = static_cast<const T*>(A.w_next);
  T* out = static_cast<T*>(A.out) + n * width;
  for (int i = threadIdx.x; i < width; i += kSandNT) out[i] = Cvt<T>::from_f32(sand_row[i] * inx * Cvt<T>::to_f32(wn[i]));
}

// ---- gelu_tanh(g) * u ----------------------------------------------------------------------------------------------------
__device__ __forceinline__ float gelu_tanh_f(float z) {
  // z/2 (1 + tanh(a)) = z / (1 + exp(-2a)), a = sqrt(2/pi) (z + 0.044715 z^3)
  const float a = 0.7978845608028654f * fmaf(0.044715f * z * z, z, z);
  return z / (1.0f + expf(-2.0f * a));
}

template <typename T, int V>
__global__ void __launch_bounds__(256)
gelu_glu_kernel(T* __restrict__ y, const T* __restrict__ gu, int64_t rows, int ff) {
  const int per_row = ff / V;
  const int64_t total = rows * per_row;
  for (int64_t e = static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x; e < total;
       e += static_cast<int64_t>(gridDim.x) * blockDim.x) {
    const int64_t r = e / per_row;
    const int c = static_cast<int>(e - r * per_row) * V;
    float g[V], u[V];
    load_vec<T, V>(g, gu + r * 2 * ff + c);
    load_vec<T, V>(u, gu + r * 2 * ff + ff + c);
#pragma unroll
    for (int i = 0; i < V; ++i) g[i] = gelu_tanh_f(g[i]) * u[i];
    store_vec<T, V>(y + r * ff + c, g);
  }
}

// ---- selective scan ------------------------------------------------------------------------------------------------------
struct SelSeq {
  int tok0;   // first packed row
  int count;  // tokens in this step
  int slot;   // state slot
  int fresh;  // 1: the sequence starts here (the carried state counts as zero)
};

struct SelArgs {
  void* out; int64_t out_stride;
  const void* x; int64_t x_stride;
  const void* dt; int64_t dt_stride;
  const float* dt_bias;
  const float* a;                     // [I][N], the rates
  const void* b; const void* c; int64_t bc_stride;
  const float* skip;                  // [I]
  const void* z; int64_t z_stride;
  float gain;
  float* state;                       // [slots][I][N]
  const SelSeq* seqs;
  int I, N, lg;                       // lg: log2 of the lanes that share a channel
  int vec;                            // rows of x, dt and z may be copied in 16-byte pieces and out written in pairs
  int vec_bc;                         // rows of B and C may be copied in 16-byte pieces
};

// Step sizes and gates of 16-bit models use the hardware's exponential and reciprocal (relative errors of a few 1e-7).
// softplus(z) = max(z, 0) + log(1 + u), u = exp(-|z|), with log(1 + u) = 2 artanh(r), r = u / (2 + u) <= 1/3, and the Taylor
// series artanh(r) = r (1 + r^2/3 + r^4/5 + ...), cut after r^12 / 13 (relative remainder below 2e-8): accurate for small u too.
template <typename T>
__device__ __forceinline__ float step_of(float z) {
  if constexpr (sizeof(T) == 4) {
    return softplus_f(z);
  } else {
    const float u = __expf(-fabsf(z)), r = __fdividef(u, 2.0f + u), q = r * r;
    float p = fmaf(q, 1.0f / 13.0f, 1.0f / 11.0f);
    p = fmaf(p, q, 1.0f / 9.0f);
    p = fmaf(p, q, 1.0f / 7.0f);
    p = fmaf(p, q, 1.0f / 5.0f);
    p = fmaf(p, q, 1.0f / 3.0f);
    p = fmaf(p, q, 1.0f);
    return fmaxf(z, 0.f) + 2.0f * r * p;
  }
}
template <typename T>
__device__ __forceinline__ float gate_of(float z) {
  if constexpr (sizeof(T) == 4) return silu_f(z);
  else return __fdividef(z, 1.0f + __expf(-z));
}

// Two fp32 numbers in one 64-bit register: sm_100 multiplies and adds both with one instruction.
using f32x2 = unsigned long long;
__device__ __forceinline__ f32x2 pack2(float lo, float hi) {
  f32x2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
  return r;
}
__device__ __forceinline__ void unpack2(f32x2 v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
  f32x2 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ float exp2_hw(float x) {
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
  return r;
}

// S <- exp(dt A) S + w for two states.  16-bit models: A2 = A log2(e) and the hardware's exp2 instruction.  fp32: A2 = A and
// S + (exp(dt A) - 1) S: a factor just below one would be rounded the same way for thousands of tokens, its distance to one is not.
template <typename T>
__device__ __forceinline__ f32x2 decayed(f32x2 S, f32x2 dt, f32x2 a2, f32x2 w) {
  float x, y;
  unpack2(mul2(dt, a2), x, y);
  if constexpr (sizeof(T) == 4) {
    float s, t;
    unpack2(fma2(pack2(expm1f(x), expm1f(y)), S, w), x, y);
    unpack2(S, s, t);
    return pack2(s + x, t + y);
  } else {
    return fma2(pack2(exp2_hw(x), exp2_hw(y)), S, w);
  }
}

__device__ __forceinline__ void sel_copy16(void* dst, const void* src, bool valid) {
  const uint32_t d = static_cast<uint32_t>(__cvta_generic_to_shared(dst));
  const int bytes = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(bytes) : "memory");
}

// One CTA (128 threads) per (sequence, 128 / L channels), L = 2^lg adjacent lanes per channel, NPT states each in registers for
// the whole portion.  32 tokens are staged at a time: their rows arrive by cp.async one stage ahead; step sizes (one softplus per
// token and channel) and B, C in fp32 are formed once per stage; the read-outs leave gated.  Four tokens are computed together:
// only the four multiply-adds of a state depend on each other, and the lanes of a channel sum four read-outs in one butterfly.
constexpr int kSelNT = 128;
constexpr int kSelTok = 32;

template <typename T>
inline size_t sel_smem(int ch, int np, int n) {
  return sizeof(float) * kSelTok * (2 * static_cast<size_t>(ch) + 2 * static_cast<size_t>(np)) +
         2 * kSelTok * (3 * static_cast<size_t>(ch) + 2 * static_cast<size_t>(n)) * sizeof(T);
}

template <typename T, int NPT>
__global__ void __launch_bounds__(kSelNT)
selective_scan_kernel(const SelArgs A) {
  extern __shared__ __align__(16) unsigned char sel_raw[];
  const SelSeq sq = A.seqs[blockIdx.y];
  if (sq.count <= 0) return;
  const int tid = threadIdx.x, lg = A.lg, L = 1 << lg, lgc = 7 - lg, CH = 1 << lgc, NP = NPT << lg;
  const int I = A.I, N = A.N, c0 = blockIdx.x * CH, nch = min(CH, I - c0);
  float2* ds = reinterpret_cast<float2*>(sel_raw);                       // (dt, dt x) [tok][CH]; later (read-out, -)
  float* bc = reinterpret_cast<float*>(ds + kSelTok * CH);               // B | C, [tok][2 NP]
  T* raw = reinterpret_cast<T*>(bc + kSelTok * 2 * NP);                  // [2 stages]: [x, dt, z][tok][CH], [B, C][tok][N]
  const int stage_elems = kSelTok * (3 * CH + 2 * N);
  const int cl = tid >> lg, sub = tid & (L - 1), ch = c0 + cl;
  const bool has = cl < nch;
  const T* xp = static_cast<const T*>(A.x) + static_cast<int64_t>(sq.tok0) * A.x_stride + c0;
  const T* dp = static_cast<const T*>(A.dt) + static_cast<int64_t>(sq.tok0) * A.dt_stride + c0;
  const T* zp = static_cast<const T*>(A.z) + static_cast<int64_t>(sq.tok0) * A.z_stride + c0;
  const T* bp = static_cast<const T*>(A.b) + static_cast<int64_t>(sq.tok0) * A.bc_stride;
  const T* cp = static_cast<const T*>(A.c) + static_cast<int64_t>(sq.tok0) * A.bc_stride;
  T* op = static_cast<T*>(A.out) + static_cast<int64_t>(sq.tok0) * A.out_stride + c0;
  float* st = A.state + (static_cast<int64_t>(sq.slot) * I + ch) * N;
  // the channels a thread converts and stores never change from stage to stage: two neighbours (vec) or one
  const int cv = A.vec ? (tid & (CH / 2 - 1)) * 2 : tid & (CH - 1);
  const int tv = A.vec ? tid >> (lgc - 1) : tid >> lgc, tstep = A.vec ? kSelNT >> (lgc - 1) : kSelNT >> lgc;
  const bool cok = cv < nch;
  const float bias0 = cok ? A.dt_bias[c0 + cv] : 0.f, bias1 = cok && A.vec ? A.dt_bias[c0 + cv + 1] : 0.f;
  const float skip0 = cok ? A.skip[c0 + cv] : 0.f, skip1 = cok && A.vec ? A.skip[c0 + cv + 1] : 0.f;

  auto load_stage = [&](int t0, int buf) {
    T* dst = raw + buf * stage_elems;
    const int nt = min(kSelTok, sq.count - t0);
    constexpr int E = 16 / sizeof(T), LE = sizeof(T) == 4 ? 2 : 3;
    if (A.vec) {
      const int lp = lgc - LE;                                           // log2 of the pieces of a row
      for (int e = tid; e < (3 * kSelTok) << lp; e += kSelNT) {
        const int row = e >> lp, which = row / kSelTok, t = row & (kSelTok - 1), c = (e & ((1 << lp) - 1)) * E;
        const bool ok = t < nt && c < nch;
        const T* src = which == 0 ? xp : (which == 1 ? dp : zp);
        const int64_t stride = which == 0 ? A.x_stride : (which == 1 ? A.dt_stride : A.z_stride);
        sel_copy16(dst + row * CH + c, ok ? src + static_cast<int64_t>(t0 + t) * stride + c : src, ok);
      }
    } else {
      for (int e = tid; e < kSelTok * CH; e += kSelNT) {
        const int t = e >> lgc, c = e & (CH - 1);
        if (t < nt && c < nch) {
          dst[t * CH + c] = xp[static_cast<int64_t>(t0 + t) * A.x_stride + c];
          dst[(kSelTok + t) * CH + c] = dp[static_cast<int64_t>(t0 + t) * A.dt_stride + c];
          dst[(2 * kSelTok + t) * CH + c] = zp[static_cast<int64_t>(t0 + t) * A.z_stride + c];
        }
      }
    }
    dst += 3 * kSelTok * CH;
    const int t = tid >> 2;                                              // four threads per row of B and C
    if (A.vec_bc) {
      for (int n = (tid & 3) * E; n < 2 * N; n += 4 * E) {
        const T* src = n < N ? bp + n : cp + n - N;
        sel_copy16(dst + t * 2 * N + n, t < nt ? src + static_cast<int64_t>(t0 + t) * A.bc_stride : src, t < nt);
      }
    } else if (t < nt) {
      for (int n = tid & 3; n < 2 * N; n += 4) dst[t * 2 * N + n] = (n < N ? bp + n : cp + n - N)[static_cast<int64_t>(t0 + t) * A.bc_stride];
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  load_stage(0, 0);
  f32x2 S[NPT / 2], a2[NPT / 2];
#pragma unroll
  for (int j = 0; j < NPT; j += 2) {
    float s[2], a[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int n = sub * NPT + j + i;
      const bool ok = has && n < N;
      s[i] = (ok && !sq.fresh) ? st[n] : 0.f;
      a[i] = ok ? A.a[static_cast<int64_t>(ch) * N + n] * (sizeof(T) == 4 ? 1.0f : 1.4426950408889634f) : 0.f;
    }
    S[j / 2] = pack2(s[0], s[1]);
    a2[j / 2] = pack2(a[0], a[1]);
  }
  for (int t0 = 0, buf = 0; t0 < sq.count; t0 += kSelTok, buf ^= 1) {
    const int nt = min(kSelTok, sq.count - t0), nt4 = (nt + 3) & ~3;     // up to three tokens of padding: dt = 0 leaves the state
    const T* rx = raw + buf * stage_elems;
    const T* rd = rx + kSelTok * CH;
    const T* rz = rd + kSelTok * CH;
    const T* rbc = rz + kSelTok * CH;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    if (t0 + kSelTok < sq.count) load_stage(t0 + kSelTok, buf ^ 1);
#pragma unroll 4
    for (int t = tv; t < nt4; t += tstep) {
      const int e = t * CH + cv;
      const bool ok = cok && t < nt;
      const float da = ok ? step_of<T>(Cvt<T>::to_f32(rd[e]) + bias0) : 0.f;
      const float xa = ok ? Cvt<T>::to_f32(rx[e]) : 0.f;
      if (A.vec) {
        const float db = ok ? step_of<T>(Cvt<T>::to_f32(rd[e + 1]) + bias1) : 0.f;
        const float xb = ok ? Cvt<T>::to_f32(rx[e + 1]) : 0.f;
        *reinterpret_cast<float4*>(ds + e) = make_float4(da, da * xa, db, db * xb);
      } else {
        ds[e] = make_float2(da, da * xa);
      }
    }
    {
      const int t = tid >> 2;
      if (t < nt4)
        for (int n = tid & 3; n < NP; n += 4) {
          const bool ok = t < nt && n < N;
          bc[t * 2 * NP + n] = ok ? Cvt<T>::to_f32(rbc[t * 2 * N + n]) : 0.f;
          bc[t * 2 * NP + NP + n] = ok ? Cvt<T>::to_f32(rbc[t * 2 * N + N + n]) : 0.f;
        }
    }
    __syncthreads();
    const float* bt = bc + sub * NPT;
    for (int t = 0; t < nt4; t += 4) {
      float2 d[4];
      float y[4];
#pragma unroll
      for (int u = 0; u < 4; ++u) d[u] = ds[(t + u) * CH + cl];
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const float* row = bt + (t + u) * 2 * NP;
        f32x2 B[NPT / 2], C[NPT / 2];
        if constexpr (NPT % 4 == 0) {
#pragma unroll
          for (int j = 0; j < NPT; j += 4) {
            const ulonglong2 b2 = *reinterpret_cast<const ulonglong2*>(row + j), c2 = *reinterpret_cast<const ulonglong2*>(row + NP + j);
            B[j / 2] = b2.x;
            B[j / 2 + 1] = b2.y;
            C[j / 2] = c2.x;
            C[j / 2 + 1] = c2.y;
          }
        } else {
#pragma unroll
          for (int j = 0; j < NPT; j += 2) {
            B[j / 2] = *reinterpret_cast<const f32x2*>(row + j);
            C[j / 2] = *reinterpret_cast<const f32x2*>(row + NP + j);
          }
        }
        const f32x2 dt2 = pack2(d[u].x, d[u].x), dx2 = pack2(d[u].y, d[u].y);
        f32x2 acc = pack2(0.f, 0.f);
#pragma unroll
        for (int j = 0; j < NPT / 2; ++j) {
          S[j] = decayed<T>(S[j], dt2, a2[j], mul2(dx2, B[j]));
          acc = fma2(S[j], C[j], acc);
        }
        float y0, y1;
        unpack2(acc, y0, y1);
        y[u] = y0 + y1;
      }
      // the channel's lanes have read (dt, dt x) of these tokens: they are in one warp, and the shuffles come after their reads
      if (lg == 0) {
#pragma unroll
        for (int u = 0; u < 4; ++u) ds[(t + u) * CH + cl].x = y[u];
      } else {
        const bool odd = sub & 1;
        float k0 = (odd ? y[2] : y[0]) + __shfl_xor_sync(0xffffffffu, odd ? y[0] : y[2], 1);
        float k1 = (odd ? y[3] : y[1]) + __shfl_xor_sync(0xffffffffu, odd ? y[1] : y[3], 1);
        const int tk = t + (odd ? 2 : 0);
        if (lg == 1) {
          ds[tk * CH + cl].x = k0;
          ds[(tk + 1) * CH + cl].x = k1;
        } else {
          const bool hi = sub & 2;
          float k = (hi ? k1 : k0) + __shfl_xor_sync(0xffffffffu, hi ? k0 : k1, 2);
          for (int o = 4; o < L; o <<= 1) k += __shfl_xor_sync(0xffffffffu, k, o);
          if (sub < 4) ds[(tk + (hi ? 1 : 0)) * CH + cl].x = k;
        }
      }
    }
    __syncthreads();
    if (cok)
#pragma unroll 4
      for (int t = tv; t < nt; t += tstep) {
        const int e = t * CH + cv;
        T* dst = op + static_cast<int64_t>(t0 + t) * A.out_stride + cv;
        const float ya = A.gain * fmaf(skip0, Cvt<T>::to_f32(rx[e]), ds[e].x) * gate_of<T>(Cvt<T>::to_f32(rz[e]));
        if (A.vec) {
          const float yb = A.gain * fmaf(skip1, Cvt<T>::to_f32(rx[e + 1]), ds[e + 1].x) * gate_of<T>(Cvt<T>::to_f32(rz[e + 1]));
          struct alignas(2 * sizeof(T)) Pair { T a, b; };
          *reinterpret_cast<Pair*>(dst) = Pair{Cvt<T>::from_f32(ya), Cvt<T>::from_f32(yb)};
        } else {
          *dst = Cvt<T>::from_f32(ya);
        }
      }
    __syncthreads();
  }
#pragma unroll
  for (int j = 0; j < NPT; j += 2) {
    float lo, hi;
    unpack2(S[j / 2], lo, hi);
    const int n = sub * NPT + j;
    if (has && n < N) st[n] = lo;
    if (has && n + 1 < N) st[n + 1] = hi;
  }
}

// One token per sequence: bound by the state's bytes, which are read and written once, in 16-byte pieces when V = 4.  A thread
// asks memory for everything it needs - P pieces of a channel's state among it - before it computes.
template <typename T, int V, int P>
__global__ void __launch_bounds__(128)
selective_step_kernel(const SelArgs A) {
  const SelSeq sq = A.seqs[blockIdx.y];
  const int lg = A.lg, L = 1 << lg, N = A.N;
  const int ch = blockIdx.x * (128 >> lg) + (threadIdx.x >> lg), sub = threadIdx.x & (L - 1);
  const bool has = ch < A.I, writes = has && sub == 0;
  const int64_t n = sq.tok0;
  float y = 0.f, x = 0.f, z = 0.f, skip = 0.f;
  if (has) {
    float* st = A.state + (static_cast<int64_t>(sq.slot) * A.I + ch) * N;
    const float* al = A.a + static_cast<int64_t>(ch) * N;
    const T* bp = static_cast<const T*>(A.b) + n * A.bc_stride;
    const T* cp = static_cast<const T*>(A.c) + n * A.bc_stride;
    float s[P][V], a[P][V], bb[P][V], cc[P][V];
    auto fetch = [&](int p, int i) {
      if constexpr (V == 4) {
        const float4 r = *reinterpret_cast<const float4*>(al + i);
        a[p][0] = r.x; a[p][1] = r.y; a[p][2] = r.z; a[p][3] = r.w;
        const float4 q = sq.fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(st + i);
        s[p][0] = q.x; s[p][1] = q.y; s[p][2] = q.z; s[p][3] = q.w;
      } else {
        a[p][0] = al[i];
        s[p][0] = sq.fresh ? 0.f : st[i];
      }
      if (V == 4 && A.vec_bc) {
        struct alignas(V * sizeof(T)) Four { T e[V]; };
        const Four b4 = *reinterpret_cast<const Four*>(bp + i), c4 = *reinterpret_cast<const Four*>(cp + i);
#pragma unroll
        for (int u = 0; u < V; ++u) {
          bb[p][u] = Cvt<T>::to_f32(b4.e[u]);
          cc[p][u] = Cvt<T>::to_f32(c4.e[u]);
        }
      } else {
#pragma unroll
        for (int u = 0; u < V; ++u) {
          bb[p][u] = Cvt<T>::to_f32(bp[i + u]);
          cc[p][u] = Cvt<T>::to_f32(cp[i + u]);
        }
      }
    };
    int i0 = sub * V;
#pragma unroll
    for (int p = 0; p < P; ++p)
      if (i0 + p * L * V < N) fetch(p, i0 + p * L * V);
    x = Cvt<T>::to_f32(static_cast<const T*>(A.x)[n * A.x_stride + ch]);
    if (writes) {
      z = Cvt<T>::to_f32(static_cast<const T*>(A.z)[n * A.z_stride + ch]);
      skip = A.skip[ch];
    }
    const float dt = step_of<T>(Cvt<T>::to_f32(static_cast<const T*>(A.dt)[n * A.dt_stride + ch]) + A.dt_bias[ch]);
    const float dx = dt * x, dts = sizeof(T) == 4 ? dt : dt * 1.4426950408889634f;    // 16-bit models: powers of two
    while (i0 < N) {
#pragma unroll
      for (int p = 0; p < P; ++p) {
        const int i = i0 + p * L * V;
        if (i >= N) continue;
        if constexpr (V == 4) {
          const f32x2 dt2 = pack2(dts, dts), dx2 = pack2(dx, dx);
#pragma unroll
          for (int u = 0; u < V; u += 2)
            unpack2(decayed<T>(pack2(s[p][u], s[p][u + 1]), dt2, pack2(a[p][u], a[p][u + 1]),
                               mul2(dx2, pack2(bb[p][u], bb[p][u + 1]))), s[p][u], s[p][u + 1]);
          *reinterpret_cast<float4*>(st + i) = make_float4(s[p][0], s[p][1], s[p][2], s[p][3]);
        } else {
          float unused;
          unpack2(decayed<T>(pack2(s[p][0], 0.f), pack2(dts, 0.f), pack2(a[p][0], 0.f), pack2(dx * bb[p][0], 0.f)), s[p][0], unused);
          st[i] = s[p][0];
        }
#pragma unroll
        for (int u = 0; u < V; ++u) y = fmaf(s[p][u], cc[p][u], y);
      }
      i0 += P * L * V;
#pragma unroll
      for (int p = 0; p < P; ++p)
        if (i0 + p * L * V < N) fetch(p, i0 + p * L * V);
    }
  }
  for (int o = 1; o < L; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
  if (writes)
    static_cast<T*>(A.out)[n * A.out_stride + ch] = Cvt<T>::from_f32(A.gain * fmaf(skip, x, y) * gate_of<T>(z));
}

inline int sel_check(const char* what, const SelArgs& A, int n_seqs) {
  if (n_seqs < 0 || A.I <= 0 || A.N <= 0) return fail(B200_EINVAL, "%s: bad sizes", what);
  if (n_seqs > 65535) return fail(B200_ESHAPE, "%s: %d sequences", what, n_seqs);
  if (n_seqs > 0 && (!A.out || !A.x || !A.dt || !A.dt_bias || !A.a || !A.b || !A.c || !A.skip || !A.z || !A.state || !A.seqs))
    return fail(B200_EINVAL, "%s: null pointer", what);
  return 0;
}

}  // namespace
}  // namespace b200

using namespace b200;

extern "C" {

int b200_sandwich_residual(float* x, const void* y, int64_t y_stride, int y_is_f32, float sign, const void* w_norm,
                           const void* layer_scale, float eps, const void* w_next, float eps_next, void* out, int rows,
                           int width, int dtype, void* stream) {
  if (rows < 0 || width <= 0 || width > 50000) return fail(B200_EINVAL, "b200_sandwich_residual: bad sizes");
  if (rows == 0) return 0;
  if (!x || !y || !w_norm || (out && !w_next)) return fail(B200_EINVAL, "b200_sandwich_residual: null pointer");
  const SandArgs A{x, y, y_stride, sign, w_norm, layer_scale, eps, w_next, out, eps_next, width};
  auto s = static_cast<cudaStream_t>(stream);
  return selective_by_dtype(dtype, "b200_sandwich_residual", [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    auto run = [&](auto* ytag) {
      using Y = std::remove_pointer_t<decltype(ytag)>;
      const bool vec = width % 8 == 0 && (y_stride * sizeof(Y)) % 16 == 0 && aligned16(x) && aligned16(y) && aligned16(w_norm) &&
                       (!layer_scale || aligned16(layer_scale)) && (!out || (aligned16(out) && aligned16(w_next)));
      const int per = kSandNT * 8;
      if (vec && width <= per) sandwich_residual_kernel<T, Y, 8, 1><<<rows, kSandNT, 0, s>>>(A);
      else if (vec && width <= 2 * per) sandwich_residual_kernel<T, Y, 8, 2><<<rows, kSandNT, 0, s>>>(A);
      else if (vec && width <= 4 * per) sandwich_residual_kernel<T, Y, 8, 4><<<rows, kSandNT, 0, s>>>(A);
      else if (vec && width <= 8 * per) sandwich_residual_kernel<T, Y, 8, 8><<<rows, kSandNT, 0, s>>>(A);
      else {
        const size_t smem = static_cast<size_t>(width) * sizeof(float);
        auto kern = sandwich_residual_any_kernel<T, Y>;
        if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
        kern<<<rows, kSandNT, smem, s>>>(A);
      }
    };
    if (y_is_f32) run(static_cast<float*>(nullptr));
    else run(static_cast<T*>(nullptr));
    return check_launch("b200_sandwich_residual");
  });
}

int b200_gelu_glu(void* y, const void* gu, int64_t rows, int ff, int dtype, void* stream) {
  if (rows < 0 || ff <= 0) return fail(B200_EINVAL, "b200_gelu_glu: bad sizes");
  if (rows == 0) return 0;
  if (!y || !gu) return fail(B200_EINVAL, "b200_gelu_glu: null pointer");
  return selective_by_dtype(dtype, "b200_gelu_glu", [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    constexpr int V = 16 / sizeof(T);
    const bool vec = ff % V == 0 && aligned16(y) && aligned16(gu);
    const int64_t items = rows * (vec ? ff / V : ff);
    const unsigned grid = static_cast<unsigned>(std::min<int64_t>((items + 255) / 256, kNumSMs * 16));
    auto s = static_cast<cudaStream_t>(stream);
    if (vec) gelu_glu_kernel<T, V><<<grid, 256, 0, s>>>(static_cast<T*>(y), static_cast<const T*>(gu), rows, ff);
    else gelu_glu_kernel<T, 1><<<grid, 256, 0, s>>>(static_cast<T*>(y), static_cast<const T*>(gu), rows, ff);
    return check_launch("b200_gelu_glu");
  });
}

int b200_selective_scan(void* out, int64_t out_stride, const void* x, int64_t x_stride, const void* dt, int64_t dt_stride,
                        const float* dt_bias, const float* a, const void* b, const void* c, int64_t bc_stride,
                        const float* skip, const void* z, int64_t z_stride, float gain, float* state, const int32_t* seqs,
                        int n_seqs, int inner, int n_state, int dtype, void* stream) {
  SelArgs A{out, out_stride, x, x_stride, dt, dt_stride, dt_bias, a, b, c, bc_stride, skip, z, z_stride, gain, state,
            reinterpret_cast<const SelSeq*>(seqs), inner, n_state, 0, 0, 0};
  if (const int rc = sel_check("b200_selective_scan", A, n_seqs)) return rc;
  if (n_state > 256) return fail(B200_ESHAPE, "b200_selective_scan: %d states per channel beyond 256", n_state);
  if (n_seqs == 0) return 0;
  // lanes per channel: at most 8 states a lane, fewer (down to 2) while the launch has too few warps to fill the GPU
  int lg = 0;
  while ((8 << lg) < n_state) ++lg;
  auto warps = [&](int l) { return static_cast<int64_t>(n_seqs) * ((static_cast<int64_t>(inner) << l) + 127) / 128 * 4; };
  while (lg < 5 && warps(lg) < kNumSMs * 8 && ((n_state + (1 << lg) - 1) >> lg) > 2) ++lg;
  A.lg = lg;
  const int npt = (n_state + (1 << lg) - 1) >> lg;
  const int ch = kSelNT >> lg;
  return selective_by_dtype(dtype, "b200_selective_scan", [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    constexpr int E = 16 / sizeof(T);
    A.vec = ch % E == 0 && inner % E == 0 && x_stride % E == 0 && dt_stride % E == 0 && z_stride % E == 0 && aligned16(x) &&
            aligned16(dt) && aligned16(z) && out_stride % 2 == 0 && reinterpret_cast<uintptr_t>(out) % (2 * sizeof(T)) == 0;
    A.vec_bc = n_state % E == 0 && bc_stride % E == 0 && aligned16(b) && aligned16(c);
    auto launch = [&](auto kern, int per_lane) {
      const size_t smem = sel_smem<T>(ch, per_lane << lg, n_state);
      if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
      kern<<<dim3((inner + ch - 1) / ch, n_seqs), kSelNT, smem, static_cast<cudaStream_t>(stream)>>>(A);
    };
    if (npt <= 2) launch(selective_scan_kernel<T, 2>, 2);
    else if (npt <= 4) launch(selective_scan_kernel<T, 4>, 4);
    else if (npt <= 6) launch(selective_scan_kernel<T, 6>, 6);
    else launch(selective_scan_kernel<T, 8>, 8);
    return check_launch("b200_selective_scan");
  });
}

int b200_selective_step(void* out, int64_t out_stride, const void* x, int64_t x_stride, const void* dt, int64_t dt_stride,
                        const float* dt_bias, const float* a, const void* b, const void* c, int64_t bc_stride,
                        const float* skip, const void* z, int64_t z_stride, float gain, float* state, const int32_t* seqs,
                        int n_seqs, int inner, int n_state, int dtype, void* stream) {
  SelArgs A{out, out_stride, x, x_stride, dt, dt_stride, dt_bias, a, b, c, bc_stride, skip, z, z_stride, gain, state,
            reinterpret_cast<const SelSeq*>(seqs), inner, n_state, 0, 0, 0};
  if (const int rc = sel_check("b200_selective_step", A, n_seqs)) return rc;
  if (n_seqs == 0) return 0;
  const int per = n_state % 4 == 0 ? n_state / 4 : n_state;      // pieces of a channel's state
  const int pieces = per > 1 ? 2 : 1;                            // per lane at a time
  while (A.lg < 5 && (pieces << A.lg) < per) ++A.lg;
  const int ch = 128 >> A.lg;
  return selective_by_dtype(dtype, "b200_selective_step", [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    A.vec_bc = bc_stride % 4 == 0 && (reinterpret_cast<uintptr_t>(b) | reinterpret_cast<uintptr_t>(c)) % (4 * sizeof(T)) == 0;
    const dim3 grid((inner + ch - 1) / ch, n_seqs);
    auto s = static_cast<cudaStream_t>(stream);
    if (n_state % 4 == 0 && pieces == 2) selective_step_kernel<T, 4, 2><<<grid, 128, 0, s>>>(A);
    else if (n_state % 4 == 0) selective_step_kernel<T, 4, 1><<<grid, 128, 0, s>>>(A);
    else selective_step_kernel<T, 1, 2><<<grid, 128, 0, s>>>(A);
    return check_launch("b200_selective_step");
  });
}

}  // extern "C"
