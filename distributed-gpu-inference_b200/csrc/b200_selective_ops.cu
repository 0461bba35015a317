// Pieces for decoder designs with a per-channel selective state space and sublayers normed on both sides:
//
//   sandwich residual        x += s * ls * w * y * rsqrt(mean(y^2) + eps);  out = w_next * x * rsqrt(mean(x^2) + eps_next): the
//                            post-norm of one sublayer and the pre-norm of the next in one pass over the row
//   gated linear unit        gelu_tanh(g) * u
//   selective scan           per channel c and state n, with dt = softplus(z + bias) and A = -exp(A_log):
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
  const float* a_log;                 // [I][N]
  const void* b; const void* c; int64_t bc_stride;
  const float* skip;                  // [I]
  const void* z; int64_t z_stride;
  float gain;
  float* state;                       // [slots][I][N]
  const SelSeq* seqs;
  int I, N, lg;                       // lg: log2 of the lanes that share a channel
  int vec;                            // rows of x, dt and z may be copied in 16-byte pieces
};

// S <- exp(dt A) S + w.  16-bit models: A2 = A log2(e) and the hardware's exp2 instruction.  fp32: A2 = A and S + (exp(dt A) - 1) S:
// a factor just below one would be rounded the same way for thousands of tokens, its distance to one is not.
template <typename T>
__device__ __forceinline__ float decayed(float S, float dt, float a2, float w) {
  if constexpr (sizeof(T) == 4) {
    return S + fmaf(expm1f(dt * a2), S, w);
  } else {
    float r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(dt * a2));
    return fmaf(r, S, w);
  }
}

__device__ __forceinline__ void sel_copy16(void* dst, const void* src, bool valid) {
  const uint32_t d = static_cast<uint32_t>(__cvta_generic_to_shared(dst));
  const int bytes = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(bytes) : "memory");
}

// One CTA (128 threads) per (sequence, 128 / L channels), L = 2^lg adjacent lanes per channel, NPT states each in registers for
// the whole portion.  32 tokens are staged at a time: the rows of x, dt and the gate arrive by cp.async one stage ahead; step
// sizes (one softplus per token and channel) and B, C in fp32 are formed once per stage; the read-outs leave gated.
constexpr int kSelNT = 128;
constexpr int kSelTok = 32;

template <typename T>
inline size_t sel_smem(int ch, int np) {
  return sizeof(float) * kSelTok * (2 * static_cast<size_t>(ch) + 2 * static_cast<size_t>(np)) +
         2 * 3 * kSelTok * static_cast<size_t>(ch) * sizeof(T);
}

template <typename T, int NPT>
__global__ void __launch_bounds__(kSelNT)
selective_scan_kernel(const SelArgs A) {
  extern __shared__ __align__(16) unsigned char sel_raw[];
  const SelSeq sq = A.seqs[blockIdx.y];
  if (sq.count <= 0) return;
  const int tid = threadIdx.x, lg = A.lg, L = 1 << lg, CH = kSelNT >> lg, NP = NPT << lg;
  const int I = A.I, N = A.N, c0 = blockIdx.x * CH, nch = min(CH, I - c0);
  float2* ds = reinterpret_cast<float2*>(sel_raw);                       // (dt, dt x) [tok][CH]; later (read-out, -)
  float* bc = reinterpret_cast<float*>(ds + kSelTok * CH);               // B | C, [tok][2 NP]
  T* raw = reinterpret_cast<T*>(bc + kSelTok * 2 * NP);                  // [2 stages][x, dt, z][tok][CH]
  const int cl = tid >> lg, sub = tid & (L - 1), ch = c0 + cl;
  const bool has = cl < nch;
  const T* xp = static_cast<const T*>(A.x) + static_cast<int64_t>(sq.tok0) * A.x_stride + c0;
  const T* dp = static_cast<const T*>(A.dt) + static_cast<int64_t>(sq.tok0) * A.dt_stride + c0;
  const T* zp = static_cast<const T*>(A.z) + static_cast<int64_t>(sq.tok0) * A.z_stride + c0;
  const T* bp = static_cast<const T*>(A.b) + static_cast<int64_t>(sq.tok0) * A.bc_stride;
  const T* cp = static_cast<const T*>(A.c) + static_cast<int64_t>(sq.tok0) * A.bc_stride;
  T* op = static_cast<T*>(A.out) + static_cast<int64_t>(sq.tok0) * A.out_stride + c0;
  float* st = A.state + (static_cast<int64_t>(sq.slot) * I + ch) * N;

  auto load_stage = [&](int t0, int buf) {
    T* dst = raw + buf * 3 * kSelTok * CH;
    const int nt = min(kSelTok, sq.count - t0);
    if (A.vec) {
      constexpr int E = 16 / sizeof(T);
      const int pieces = CH / E;
      for (int e = tid; e < 3 * kSelTok * pieces; e += kSelNT) {
        const int which = e / (kSelTok * pieces), r = e - which * kSelTok * pieces;
        const int t = r / pieces, c = (r - t * pieces) * E;
        const bool ok = t < nt && c < nch;
        const T* src = which == 0 ? xp : (which == 1 ? dp : zp);
        const int64_t stride = which == 0 ? A.x_stride : (which == 1 ? A.dt_stride : A.z_stride);
        sel_copy16(dst + (which * kSelTok + t) * CH + c, ok ? src + static_cast<int64_t>(t0 + t) * stride + c : src, ok);
      }
      asm volatile("cp.async.commit_group;" ::: "memory");
    } else {
      for (int e = tid; e < kSelTok * CH; e += kSelNT) {
        const int t = e / CH, c = e - t * CH;
        if (t < nt && c < nch) {
          dst[t * CH + c] = xp[static_cast<int64_t>(t0 + t) * A.x_stride + c];
          dst[(kSelTok + t) * CH + c] = dp[static_cast<int64_t>(t0 + t) * A.dt_stride + c];
          dst[(2 * kSelTok + t) * CH + c] = zp[static_cast<int64_t>(t0 + t) * A.z_stride + c];
        }
      }
    }
  };
  load_stage(0, 0);
  float S[NPT], a2[NPT];
#pragma unroll
  for (int j = 0; j < NPT; ++j) {
    const int n = sub * NPT + j;
    const bool ok = has && n < N;
    S[j] = (ok && !sq.fresh) ? st[n] : 0.f;
    a2[j] = ok ? -expf(A.a_log[static_cast<int64_t>(ch) * N + n]) * (sizeof(T) == 4 ? 1.0f : 1.4426950408889634f) : 0.f;
  }
  for (int t0 = 0, buf = 0; t0 < sq.count; t0 += kSelTok, buf ^= 1) {
    const int nt = min(kSelTok, sq.count - t0);
    const T* rx = raw + buf * 3 * kSelTok * CH;
    const T* rd = rx + kSelTok * CH;
    const T* rz = rd + kSelTok * CH;
    // B and C of the stage (their slots were last read before the barrier that ended the previous stage)
    for (int e = tid; e < nt * NP; e += kSelNT) {
      const int t = e / NP, n = e - t * NP;
      bc[t * 2 * NP + n] = n < N ? Cvt<T>::to_f32(bp[static_cast<int64_t>(t0 + t) * A.bc_stride + n]) : 0.f;
      bc[t * 2 * NP + NP + n] = n < N ? Cvt<T>::to_f32(cp[static_cast<int64_t>(t0 + t) * A.bc_stride + n]) : 0.f;
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    if (t0 + kSelTok < sq.count) load_stage(t0 + kSelTok, buf ^ 1);
    for (int e = tid; e < nt * CH; e += kSelNT) {
      const int c = e % CH;
      if (c < nch) {
        const float dt = softplus_f(Cvt<T>::to_f32(rd[e]) + A.dt_bias[c0 + c]);
        ds[e] = make_float2(dt, dt * Cvt<T>::to_f32(rx[e]));
      } else {
        ds[e] = make_float2(0.f, 0.f);
      }
    }
    __syncthreads();
    const float* bt = bc + sub * NPT;
#pragma unroll 2
    for (int t = 0; t < nt; ++t) {
      const float2 d = ds[t * CH + cl];
      float B[NPT], C[NPT];
      if constexpr (NPT % 4 == 0) {
#pragma unroll
        for (int j = 0; j < NPT; j += 4) {
          *reinterpret_cast<float4*>(B + j) = *reinterpret_cast<const float4*>(bt + t * 2 * NP + j);
          *reinterpret_cast<float4*>(C + j) = *reinterpret_cast<const float4*>(bt + t * 2 * NP + NP + j);
        }
      } else {
#pragma unroll
        for (int j = 0; j < NPT; j += 2) {
          *reinterpret_cast<float2*>(B + j) = *reinterpret_cast<const float2*>(bt + t * 2 * NP + j);
          *reinterpret_cast<float2*>(C + j) = *reinterpret_cast<const float2*>(bt + t * 2 * NP + NP + j);
        }
      }
      float y0 = 0.f, y1 = 0.f;
#pragma unroll
      for (int j = 0; j < NPT; j += 2) {
        S[j] = decayed<T>(S[j], d.x, a2[j], d.y * B[j]);
        y0 = fmaf(S[j], C[j], y0);
        S[j + 1] = decayed<T>(S[j + 1], d.x, a2[j + 1], d.y * B[j + 1]);
        y1 = fmaf(S[j + 1], C[j + 1], y1);
      }
      float y = y0 + y1;
      if (lg > 0) {
        y += __shfl_xor_sync(0xffffffffu, y, 1);
        if (lg > 1) {
          y += __shfl_xor_sync(0xffffffffu, y, 2);
          if (lg > 2) {
            y += __shfl_xor_sync(0xffffffffu, y, 4);
            if (lg > 3) {
              y += __shfl_xor_sync(0xffffffffu, y, 8);
              if (lg > 4) y += __shfl_xor_sync(0xffffffffu, y, 16);
            }
          }
        }
      }
      // the channel's lanes have read (dt, dt x) of this token: they are in one warp, and the shuffles (or nothing, when a lane
      // is alone) come after their reads
      if (sub == 0) ds[t * CH + cl].x = y;
    }
    __syncthreads();
    for (int e = tid; e < nt * CH; e += kSelNT) {
      const int t = e / CH, c = e - t * CH;
      if (c < nch) {
        const float y = fmaf(A.skip[c0 + c], Cvt<T>::to_f32(rx[e]), ds[e].x);
        op[static_cast<int64_t>(t0 + t) * A.out_stride + c] = Cvt<T>::from_f32(A.gain * y * silu_f(Cvt<T>::to_f32(rz[e])));
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int j = 0; j < NPT; ++j) {
    const int n = sub * NPT + j;
    if (has && n < N) st[n] = S[j];
  }
}

// One token per sequence: bound by the state's bytes, which are read and written once, in 16-byte pieces when V = 4.
template <typename T, int V>
__global__ void __launch_bounds__(128)
selective_step_kernel(const SelArgs A) {
  const SelSeq sq = A.seqs[blockIdx.y];
  const int lg = A.lg, L = 1 << lg, N = A.N;
  const int ch = blockIdx.x * (128 >> lg) + (threadIdx.x >> lg), sub = threadIdx.x & (L - 1);
  const bool has = ch < A.I;
  const int64_t n = sq.tok0;
  float y = 0.f, x = 0.f;
  if (has) {
    x = Cvt<T>::to_f32(static_cast<const T*>(A.x)[n * A.x_stride + ch]);
    const float dt = softplus_f(Cvt<T>::to_f32(static_cast<const T*>(A.dt)[n * A.dt_stride + ch]) + A.dt_bias[ch]);
    const float dx = dt * x;
    const T* bp = static_cast<const T*>(A.b) + n * A.bc_stride;
    const T* cp = static_cast<const T*>(A.c) + n * A.bc_stride;
    float* st = A.state + (static_cast<int64_t>(sq.slot) * A.I + ch) * N;
    const float* al = A.a_log + static_cast<int64_t>(ch) * N;
    for (int i = sub * V; i < N; i += L * V) {
      float s[V], a[V];
      if constexpr (V == 4) {
        const float4 r = *reinterpret_cast<const float4*>(al + i);
        a[0] = r.x; a[1] = r.y; a[2] = r.z; a[3] = r.w;
        const float4 q = sq.fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(st + i);
        s[0] = q.x; s[1] = q.y; s[2] = q.z; s[3] = q.w;
      } else {
        a[0] = al[i];
        s[0] = sq.fresh ? 0.f : st[i];
      }
#pragma unroll
      for (int u = 0; u < V; ++u) {
        s[u] += fmaf(expm1f(-expf(a[u]) * dt), s[u], dx * Cvt<T>::to_f32(bp[i + u]));
        y = fmaf(s[u], Cvt<T>::to_f32(cp[i + u]), y);
      }
      if constexpr (V == 4) *reinterpret_cast<float4*>(st + i) = make_float4(s[0], s[1], s[2], s[3]);
      else st[i] = s[0];
    }
  }
  for (int o = 1; o < L; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
  if (has && sub == 0) {
    y = fmaf(A.skip[ch], x, y);
    const float z = Cvt<T>::to_f32(static_cast<const T*>(A.z)[n * A.z_stride + ch]);
    static_cast<T*>(A.out)[n * A.out_stride + ch] = Cvt<T>::from_f32(A.gain * y * silu_f(z));
  }
}

inline int sel_check(const char* what, const SelArgs& A, int n_seqs) {
  if (n_seqs < 0 || A.I <= 0 || A.N <= 0) return fail(B200_EINVAL, "%s: bad sizes", what);
  if (n_seqs > 65535) return fail(B200_ESHAPE, "%s: %d sequences", what, n_seqs);
  if (n_seqs > 0 && (!A.out || !A.x || !A.dt || !A.dt_bias || !A.a_log || !A.b || !A.c || !A.skip || !A.z || !A.state || !A.seqs))
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
                        const float* dt_bias, const float* a_log, const void* b, const void* c, int64_t bc_stride,
                        const float* skip, const void* z, int64_t z_stride, float gain, float* state, const int32_t* seqs,
                        int n_seqs, int inner, int n_state, int dtype, void* stream) {
  SelArgs A{out, out_stride, x, x_stride, dt, dt_stride, dt_bias, a_log, b, c, bc_stride, skip, z, z_stride, gain, state,
            reinterpret_cast<const SelSeq*>(seqs), inner, n_state, 0, 0};
  if (const int rc = sel_check("b200_selective_scan", A, n_seqs)) return rc;
  if (n_state > 256) return fail(B200_ESHAPE, "b200_selective_scan: %d states per channel beyond 256", n_state);
  if (n_seqs == 0) return 0;
  // lanes per channel: at most 8 states a lane, fewer (down to 2) while the launch has too few warps to fill the GPU
  int lg = 0;
  while ((8 << lg) < n_state) ++lg;
  auto warps = [&](int l) { return static_cast<int64_t>(n_seqs) * ((static_cast<int64_t>(inner) << l) + 127) / 128 * 4; };
  while (lg < 5 && warps(lg) < kNumSMs * 6 && ((n_state + (1 << lg) - 1) >> lg) > 2) ++lg;
  A.lg = lg;
  const int npt = (n_state + (1 << lg) - 1) >> lg;
  const int ch = kSelNT >> lg;
  return selective_by_dtype(dtype, "b200_selective_scan", [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    constexpr int E = 16 / sizeof(T);
    A.vec = ch % E == 0 && inner % E == 0 && x_stride % E == 0 && dt_stride % E == 0 && z_stride % E == 0 && aligned16(x) &&
            aligned16(dt) && aligned16(z);
    auto launch = [&](auto kern, int per_lane) {
      const size_t smem = sel_smem<T>(ch, per_lane << lg);
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
                        const float* dt_bias, const float* a_log, const void* b, const void* c, int64_t bc_stride,
                        const float* skip, const void* z, int64_t z_stride, float gain, float* state, const int32_t* seqs,
                        int n_seqs, int inner, int n_state, int dtype, void* stream) {
  SelArgs A{out, out_stride, x, x_stride, dt, dt_stride, dt_bias, a_log, b, c, bc_stride, skip, z, z_stride, gain, state,
            reinterpret_cast<const SelSeq*>(seqs), inner, n_state, 0, 0};
  if (const int rc = sel_check("b200_selective_step", A, n_seqs)) return rc;
  if (n_seqs == 0) return 0;
  const int per = n_state % 4 == 0 ? n_state / 4 : n_state;      // pieces of a channel's state
  while (A.lg < 5 && (1 << A.lg) < per) ++A.lg;
  const int ch = 128 >> A.lg;
  return selective_by_dtype(dtype, "b200_selective_step", [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    const dim3 grid((inner + ch - 1) / ch, n_seqs);
    auto s = static_cast<cudaStream_t>(stream);
    if (n_state % 4 == 0) selective_step_kernel<T, 4><<<grid, 128, 0, s>>>(A);
    else selective_step_kernel<T, 1><<<grid, 128, 0, s>>>(A);
    return check_launch("b200_selective_step");
  });
}

}  // extern "C"
