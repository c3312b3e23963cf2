// Residual step of pre-normed layer-list decoders (HB_NORM_PRE), with one stream or several copies of it (hyper-connections).
//
// Between two sublayers everything that touches the stream is one launch: the finished sublayer's output joins the copies as
// they are mixed, x_t <- sum_s mix[s][t] x_s + out[t] y, and the next sublayer's input is read from the new copies and normed,
// h = N(sum_t in[t] x_t).  The copies [row][S][W] are read and written once; the read-out u never leaves the registers.  A
// mixture's weighted expert rows are summed here instead of in a pass of their own.  All of it is fp32.
#include <algorithm>

#include "kernels.h"
#include "launch.h"
#include "stack_common.cuh"

namespace hb {
namespace {

constexpr int kChunks = 8;  // float4 chunks of u a thread keeps (W <= 4 * 256 * kChunks)
constexpr int kTop = 8;     // expert rows per token that the in-register form takes

template <typename WT>
__device__ __forceinline__ float4 ld4(const WT* p) {
  if constexpr (sizeof(WT) == 4) return *reinterpret_cast<const float4*>(p);
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ float4 fma4(float a, float4 b, float4 c) {
  return make_float4(fmaf(a, b.x, c.x), fmaf(a, b.y, c.y), fmaf(a, b.z, c.z), fmaf(a, b.w, c.w));
}
__device__ __forceinline__ void st_both(float* f, bf16* b, float4 v) {
  if (f) *reinterpret_cast<float4*>(f) = v;
  if (b) {
    __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    uint2 pk;
    pk.x = *reinterpret_cast<unsigned*>(&lo);
    pk.y = *reinterpret_cast<unsigned*>(&hi);
    *reinterpret_cast<uint2*>(b) = pk;
  }
}

// One block per row, S copies of four neighbouring entries per thread and chunk (W a multiple of 4)
template <typename WT, int S, int CH, bool ROWS>
__global__ void __launch_bounds__(256) stream_step_vec_kernel(StreamStep a) {
  __shared__ float red[32];
  const size_t r = blockIdx.x;
  const int W = a.W;
  float mix[S][S], out[S], in[S];
#pragma unroll
  for (int s = 0; s < S; ++s) {
    out[s] = a.out ? ldf<WT>((const WT*)a.out, s) : 1.f;
    in[s] = a.in ? ldf<WT>((const WT*)a.in, s) : 1.f;
#pragma unroll
    for (int t = 0; t < S; ++t) mix[s][t] = a.mix ? ldf<WT>((const WT*)a.mix, s * S + t) : (s == t ? 1.f : 0.f);
  }
  float wk[ROWS ? kTop : 1];
  int rk[ROWS ? kTop : 1];
  if constexpr (ROWS) {
#pragma unroll
    for (int k = 0; k < kTop; ++k) {
      wk[k] = k < a.top_k ? a.wts[r * a.top_k + k] : 0.f;
      rk[k] = k < a.top_k ? a.row_of[r * a.top_k + k] : 0;
    }
  }
  const bool add = ROWS || a.y;
  float* xr = a.x + r * S * W;
  float4 u[CH];
  float ss = 0.f;
  // all of a thread's loads go out before its first store when its share of the row fits in registers (the stores may alias
  // later loads for all the compiler knows, so it cannot move them itself); a thread only reads what it writes itself
  constexpr int B = S * CH <= 8 ? CH : 1;
  float4 x[B][S], y[B];
  auto load = [&](int c, float4(&xc)[S], float4& yc) {
    const int i = (threadIdx.x + c * 256) * 4;
    yc = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i >= W) return;
#pragma unroll
    for (int s = 0; s < S; ++s) xc[s] = a.x0 ? *reinterpret_cast<const float4*>(a.x0 + r * W + i) : *reinterpret_cast<const float4*>(xr + (size_t)s * W + i);
    if (a.y) yc = *reinterpret_cast<const float4*>(a.y + r * W + i);
    if constexpr (ROWS) {
#pragma unroll
      for (int k = 0; k < kTop; ++k)
        if (k < a.top_k) yc = fma4(wk[k], ld4<bf16>(a.rows + (size_t)rk[k] * W + i), yc);
    }
    if (a.bias) yc = fma4(1.f, ld4<WT>((const WT*)a.bias + i), yc);
  };
  if constexpr (B > 1) {
#pragma unroll
    for (int c = 0; c < CH; ++c) load(c, x[c], y[c]);
  }
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int i = (threadIdx.x + c * 256) * 4;
    if (i >= W) continue;
    if constexpr (B == 1) load(c, x[0], y[0]);
    float4(&xc)[S] = x[B == 1 ? 0 : c];
    const float4 yc = y[B == 1 ? 0 : c];
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (a.x0) {
#pragma unroll
      for (int s = 0; s < S; ++s) {
        *reinterpret_cast<float4*>(xr + (size_t)s * W + i) = xc[s];
        v = fma4(in[s], xc[s], v);
      }
    }
    if (add) {
#pragma unroll
      for (int t = 0; t < S; ++t) {
        float4 n = make_float4(out[t] * yc.x, out[t] * yc.y, out[t] * yc.z, out[t] * yc.w);
#pragma unroll
        for (int s = 0; s < S; ++s) n = fma4(mix[s][t], xc[s], n);
        if (!a.last) *reinterpret_cast<float4*>(xr + (size_t)t * W + i) = n;
        v = fma4(in[t], n, v);
      }
    }
    u[c] = v;
    ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
  float rs = 1.f;
  if (a.w) rs = 1.f / sqrtf(block_sum(ss, red) / (float)W + a.eps);
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int i = (threadIdx.x + c * 256) * 4;
    if (i >= W) continue;
    float4 v = u[c];
    if (a.w) {
      const float4 g = ld4<WT>((const WT*)a.w + i);
      v = make_float4(v.x * rs * g.x, v.y * rs * g.y, v.z * rs * g.z, v.w * rs * g.w);
    }
    st_both(a.h ? a.h + r * W + i : nullptr, a.h16 ? a.h16 + r * W + i : nullptr, v);
  }
}

// The same for any width, number of copies (<= kMaxStreams) and number of expert rows; dynamic smem: u [W]
template <typename WT>
__global__ void __launch_bounds__(256) stream_step_kernel(StreamStep a) {
  extern __shared__ float urow[];
  __shared__ float red[32];
  const size_t r = blockIdx.x;
  const int W = a.W, S = a.S;
  const bool add = a.y || a.top_k > 0;
  float* xr = a.x + r * S * W;
  float ss = 0.f;
  for (int i = threadIdx.x; i < W; i += blockDim.x) {
    float x[kMaxStreams], v = 0.f;
#pragma unroll
    for (int s = 0; s < kMaxStreams; ++s) {
      if (s >= S) break;
      x[s] = a.x0 ? a.x0[r * W + i] : xr[(size_t)s * W + i];
      if (a.x0) {
        xr[(size_t)s * W + i] = x[s];
        v = fmaf(a.in ? ldf<WT>((const WT*)a.in, s) : 1.f, x[s], v);
      }
    }
    if (add) {
      float y = a.y ? a.y[r * W + i] : 0.f;
      for (int k = 0; k < a.top_k; ++k) y = fmaf(a.wts[r * a.top_k + k], __bfloat162float(a.rows[(size_t)a.row_of[r * a.top_k + k] * W + i]), y);
      if (a.bias) y += ldf<WT>((const WT*)a.bias, i);
      for (int t = 0; t < S; ++t) {
        float n = (a.out ? ldf<WT>((const WT*)a.out, t) : 1.f) * y;
#pragma unroll
        for (int s = 0; s < kMaxStreams; ++s) {
          if (s >= S) break;
          n = fmaf(a.mix ? ldf<WT>((const WT*)a.mix, s * S + t) : (s == t ? 1.f : 0.f), x[s], n);
        }
        if (!a.last) xr[(size_t)t * W + i] = n;
        v = fmaf(a.in ? ldf<WT>((const WT*)a.in, t) : 1.f, n, v);
      }
    }
    urow[i] = v;
    ss = fmaf(v, v, ss);
  }
  float rs = 1.f;
  if (a.w) rs = 1.f / sqrtf(block_sum(ss, red) / (float)W + a.eps);
  for (int i = threadIdx.x; i < W; i += blockDim.x) {
    const float v = a.w ? urow[i] * rs * ldf<WT>((const WT*)a.w, i) : urow[i];
    if (a.h) a.h[r * W + i] = v;
    if (a.h16) a.h16[r * W + i] = __float2bfloat16(v);
  }
}

template <typename WT, int S, bool ROWS>
void launch_rows(cudaStream_t s, const StreamStep& a, int rows) {
  if (a.W <= 1024) stream_step_vec_kernel<WT, S, 1, ROWS><<<rows, 256, 0, s>>>(a);
  else if (a.W <= 2048) stream_step_vec_kernel<WT, S, 2, ROWS><<<rows, 256, 0, s>>>(a);
  else if (a.W <= 4096) stream_step_vec_kernel<WT, S, 4, ROWS><<<rows, 256, 0, s>>>(a);
  else stream_step_vec_kernel<WT, S, 8, ROWS><<<rows, 256, 0, s>>>(a);
}
template <typename WT, int S>
void launch_vec(cudaStream_t s, const StreamStep& a, int rows) {
  if (a.top_k > 0) launch_rows<WT, S, true>(s, a, rows);
  else launch_rows<WT, S, false>(s, a, rows);
}

}  // namespace

cudaError_t stack_streams_init() {
  cudaError_t e;
  if ((e = cudaFuncSetAttribute(stream_step_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024)) != cudaSuccess) return e;
  return cudaFuncSetAttribute(stream_step_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
}

cudaError_t stream_step(cudaStream_t s, const StreamStep& a, int rows) {
  if (rows <= 0) return cudaSuccess;
  if (!a.x || a.W <= 0 || a.S < 1 || a.S > kMaxStreams || (a.top_k > 0 && (a.y || !a.rows || !a.row_of || !a.wts))) return cudaErrorInvalidValue;
  if ((a.x0 != nullptr) == (a.y != nullptr || a.top_k > 0)) return cudaErrorInvalidValue;  // the start of a stack, or a sublayer's output
  if (a.S > 1 && !a.x0 && (!a.mix || !a.out)) return cudaErrorInvalidValue;
  const uintptr_t al = (uintptr_t)a.x | (uintptr_t)a.x0 | (uintptr_t)a.y | (uintptr_t)a.bias | (uintptr_t)a.rows | (uintptr_t)a.w | (uintptr_t)a.h | (uintptr_t)a.h16;
  if (a.W % 4 == 0 && a.W <= 4 * 256 * kChunks && (al & 15) == 0 && a.top_k <= kTop && a.S <= 4) {
#define HB_STREAMS(S)                                  \
  if (a.f32) launch_vec<float, S>(s, a, rows);         \
  else launch_vec<bf16, S>(s, a, rows)
    if (a.S == 1) { HB_STREAMS(1); }
    else if (a.S == 2) { HB_STREAMS(2); }
    else if (a.S == 3) { HB_STREAMS(3); }
    else { HB_STREAMS(4); }
#undef HB_STREAMS
    return cudaGetLastError();
  }
  const size_t smem = (size_t)a.W * 4;
  if (smem > 200 * 1024) return cudaErrorInvalidValue;
  if (a.f32) stream_step_kernel<float><<<rows, 256, smem, s>>>(a);
  else stream_step_kernel<bf16><<<rows, 256, smem, s>>>(a);
  return cudaGetLastError();
}

}  // namespace hb
