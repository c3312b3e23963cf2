// Attention over cached latent rows [c (R) | rotated key part (Dr)] without expanding them: single-token steps and short prompt
// portions of latent-attention layers in the bf16 mode.  Queries arrive carried into the latent space (q_h^T W_uk,h), values leave
// as weighted latents, so all heads of a token read the same rows and one pass over them serves up to 32 heads.
//
//   S^T[kv = 64, heads] = K_tile[64 kv x (R + Dr)] (A, K-major smem) . Q^T (B: NQ query heads, zero padded)
//   O^T[r = 128 lanes, heads] += C_tile^T (A, the SAME smem bytes read MN-major, two 64-column sub-tiles) . P^T (B)
//
// Grid (splits, head groups, tokens).  A kv tile is one 64-position page; its 64-column sub-tiles travel in pairs through one
// ring (16 KB slots) and the rotated part through a second ring, so loads of the next tiles overlap the products of this one.
//   warp 0 : TMA producer      warp 1 / warp 6 : issuers of the S / PV products (one warp for both was the bottleneck: an issue
//                takes about 50 cycles whatever the product's size, and a tile needs 36 + 16 of them)
//   warps 2..5 : softmax.  The S^T tile of an M = 64 product sits in lanes 0..15 of every 32-lane quadrant; the running maximum is
//                only reduced when some score passes it by more than 2^8 (the first tile, rarely later), sums stay per thread.
// A second kernel merges the splits.  Further kernels here move rows into the layouts of the per-head products.
#include <math.h>

#include <algorithm>

#include "kernels.h"
#include "launch.h"
#include "ptx.cuh"
#include "tma_host.h"

namespace hb {
namespace {

constexpr int kThreads = 224;
constexpr int PAGE = 64;
constexpr int kSub = PAGE * 128;    // one 64-column sub-tile of a page (bf16)
constexpr int kPair = 2 * kSub;
constexpr int kMaxC = 12, kMaxR = 6;  // ring slots
constexpr float kRescale = 8.0f;      // log2 units
constexpr int kTokRows = kLatentTokRows;
constexpr int kMaxSplits = 32;

__device__ __forceinline__ float fast_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// OR of a predicate over the 128 softmax threads (named barrier 1)
__device__ __forceinline__ bool bar_any(bool v) {
  uint32_t r;
  asm volatile(
      "{\n"
      ".reg .pred p, q;\n"
      "setp.ne.u32 q, %1, 0;\n"
      "barrier.cta.red.or.pred p, 1, 128, q;\n"
      "selp.u32 %0, 1, 0, p;\n"
      "}\n"
      : "=r"(r)
      : "r"((uint32_t)v)
      : "memory");
  return r != 0;
}
template <int NQ>
__device__ __forceinline__ void tmem_ld_cols(uint32_t taddr, uint32_t (&r)[NQ]) {
  if constexpr (NQ == 32) tmem_ld_32x32b_x32(taddr, r);
  else tmem_ld_32x32b_x16(taddr, r);
}

struct Rings { int cs, rs; };  // slots of the latent-pair ring / of the rotated-part ring

template <int NQ>
__global__ void __launch_bounds__(kThreads, 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap map_c, const __grid_constant__ CUtensorMap map_r,
                     const __grid_constant__ CUtensorMap map_ql, const __grid_constant__ CUtensorMap map_qr,
                     const __grid_constant__ LatentDecodeArgs a, Rings rings, int num_splits) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int R = a.R;
  const int nc = (R + 63) / 64, np = (nc + 1) / 2;
  const int CS = rings.cs, RS = rings.rs;
  uint8_t* ring_c = smem;                        // [CS][2][64 rows][128 B]
  uint8_t* ring_r = ring_c + CS * kPair;         // [RS][64 rows][128 B]
  uint8_t* sQ = ring_r + RS * kSub;              // [nc + 1][NQ rows][128 B]
  uint8_t* sP = sQ + (nc + 1) * NQ * 128;        // [2][NQ rows][128 B]
  float* sRed = reinterpret_cast<float*>(sP + 2 * NQ * 128);  // [4 warps][NQ]
  float* sFac = sRed + 4 * NQ;                   // [NQ] rescale factors; at the end the maxima
  uint64_t* bars = reinterpret_cast<uint64_t*>(sFac + NQ);
  uint64_t* c_full = bars;
  uint64_t* c_empty = c_full + kMaxC;
  uint64_t* r_full = c_empty + kMaxC;
  uint64_t* r_empty = r_full + kMaxR;
  uint64_t* s_full = r_empty + kMaxR;   // [2]
  uint64_t* s_empty = s_full + 2;       // [2]
  uint64_t* p_full = s_empty + 2;       // [2]
  uint64_t* pv_done = p_full + 2;       // [2]
  uint64_t* q_ready = pv_done + 2;
  uint32_t* tmem_ptr = reinterpret_cast<uint32_t*>(q_ready + 1);

  const int split = blockIdx.x, hg = blockIdx.y, tq = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int ctx = a.positions[tq] + 1;
  const int kv_lo = a.window > 0 ? max(0, ctx - a.window) : 0;
  const int t_first = kv_lo / PAGE, n_total = (ctx + PAGE - 1) / PAGE;
  const int tps = (n_total - t_first + num_splits - 1) / num_splits;
  const int t_begin = t_first + split * tps;
  const int n_tiles = min(n_total, t_begin + tps) - t_begin;
  const int h0 = hg * NQ, nh = min(NQ, a.H - h0);
  float* ws = a.workspace + (((size_t)tq * gridDim.y + hg) * num_splits + split) * NQ * (R + 2);
  pdl_launch_dependents();
  if (n_tiles <= 0) {
    pdl_wait();  // the partials may still be read by an earlier launch's combine pass
    for (int i = threadIdx.x; i < NQ * (R + 2); i += kThreads) ws[i] = (i % (R + 2) == R) ? -INFINITY : 0.f;
    return;
  }
  const int32_t* pt = a.page_table + (size_t)a.seq_of[tq] * a.max_pages;

  if (threadIdx.x == 0) {
    tma_prefetch_desc(&map_c);
    tma_prefetch_desc(&map_r);
    tma_prefetch_desc(&map_ql);
    tma_prefetch_desc(&map_qr);
    for (int i = 0; i < CS; ++i) { mbar_init(&c_full[i], 1); mbar_init(&c_empty[i], 1); }
    for (int i = 0; i < RS; ++i) { mbar_init(&r_full[i], 1); mbar_init(&r_empty[i], 1); }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&s_full[i], 1);
      mbar_init(&s_empty[i], 4);
      mbar_init(&p_full[i], 4);
      mbar_init(&pv_done[i], 1);
    }
    mbar_init(q_ready, 1);
    fence_barrier_init();
  }
  constexpr uint32_t kCols = NQ == 32 ? 256 : 128;  // two S tiles, up to four O blocks of NQ columns
  if (warp == 1) {
    tmem_alloc(tmem_ptr, kCols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = __shfl_sync(0xffffffffu, *tmem_ptr, 0);
  const uint32_t tmem_S = tmem_base, tmem_O = tmem_base + 2 * NQ;
  pdl_wait();  // launched while the kernel in front of it drains: nothing above depends on it

  if (warp == 0) {
    const bool elected = elect_one_sync();
    int cs = 0, rs = 0;
    uint32_t cph = 0, rph = 0;
    if (elected) {  // the token's queries, one row per head (zeros where a head or an entry does not exist)
      mbar_arrive_expect_tx(q_ready, (nc + 1) * NQ * 128);
      for (int c = 0; c < nc; ++c) tma_load_3d(sQ + c * (NQ * 128), &map_ql, q_ready, c * 64, tq, h0);
      tma_load_3d(sQ + nc * (NQ * 128), &map_qr, q_ready, 0, h0, tq);
    }
    for (int j = 0; j < n_tiles; ++j) {
      const int row = pt[t_begin + j] * PAGE;
      for (int p = 0; p < np; ++p) {
        mbar_wait(&c_empty[cs], cph ^ 1);
        if (elected) {
          const bool two = 2 * p + 1 < nc;  // an odd last sub-tile leaves the pair's second half as it is (its O lanes are unused)
          mbar_arrive_expect_tx(&c_full[cs], two ? kPair : kSub);
          tma_load_2d(ring_c + cs * kPair, &map_c, &c_full[cs], p * 128, row);
          if (two) tma_load_2d(ring_c + cs * kPair + kSub, &map_c, &c_full[cs], p * 128 + 64, row);
        }
        if (++cs == CS) { cs = 0; cph ^= 1; }
      }
      mbar_wait(&r_empty[rs], rph ^ 1);
      if (elected) {
        mbar_arrive_expect_tx(&r_full[rs], kSub);
        tma_load_2d(ring_r + rs * kSub, &map_r, &r_full[rs], 0, row);
      }
      if (++rs == RS) { rs = 0; rph ^= 1; }
    }
  } else if (warp == 1) {
    const bool elected = elect_one_sync();
    constexpr uint32_t idesc_s = umma_idesc_bf16(PAGE, NQ, 0, 0);
    // descriptors are a base per operand plus offsets in 16-byte units (the address field never carries)
    const uint64_t kdesc0 = umma_desc_kmajor_sw128(smem_u32(ring_c)), rdesc0 = umma_desc_kmajor_sw128(smem_u32(ring_r));
    const uint64_t qdesc0 = umma_desc_kmajor_sw128(smem_u32(sQ));
    int cs = 0, rs = 0;  // ring slots of the next latent pair / rotated part
    uint32_t cph = 0, rph = 0;
    auto issue_s = [&](int j) {
      mbar_wait(&s_empty[j & 1], ((j >> 1) & 1) ^ 1);
      const uint32_t d = tmem_S + (j & 1) * NQ;
      uint64_t qd = qdesc0;
      for (int p = 0; p < np; ++p) {
        const bool two = 2 * p + 1 < nc;
        mbar_wait(&c_full[cs], cph);
        tc_fence_after();
        const uint64_t kd = kdesc0 + (uint64_t)(cs * (kPair >> 4));
        if (elected) {
#pragma unroll
          for (int k = 0; k < 4; ++k) umma_f16_ss(d, kd + k * 2, qd + k * 2, idesc_s, k != 0 ? 1u : (p != 0 ? 1u : 0u));
          if (two) {
#pragma unroll
            for (int k = 0; k < 4; ++k) umma_f16_ss(d, kd + (kSub >> 4) + k * 2, qd + (NQ * 128 >> 4) + k * 2, idesc_s, 1u);
          }
        }
        qd += two ? 2 * (NQ * 128 >> 4) : (NQ * 128 >> 4);
        if (++cs == CS) { cs = 0; cph ^= 1; }
      }
      mbar_wait(&r_full[rs], rph);
      tc_fence_after();
      if (elected) {
        const uint64_t rd = rdesc0 + (uint64_t)(rs * (kSub >> 4));
#pragma unroll
        for (int k = 0; k < 4; ++k) umma_f16_ss(d, rd + k * 2, qd + k * 2, idesc_s, 1u);
        umma_commit(&r_empty[rs]);
        umma_commit(&s_full[j & 1]);
      }
      if (++rs == RS) { rs = 0; rph ^= 1; }
    };
    mbar_wait(q_ready, 0);
    tc_fence_after();
    for (int j = 0; j < n_tiles; ++j) issue_s(j);
  } else if (warp == 6) {
    const bool elected = elect_one_sync();
    constexpr uint32_t idesc_o = umma_idesc_bf16(128, NQ, 1, 0);
    const uint64_t pdesc0 = umma_desc_kmajor_sw128(smem_u32(sP)), vdesc0 = umma_desc_mnmajor_sw128(smem_u32(ring_c), kSub, 1024);
    int vs = 0;
    uint32_t vph = 0;
    for (int j = 0; j < n_tiles; ++j) {
      mbar_wait(&p_full[j & 1], (j >> 1) & 1);
      const uint64_t pd = pdesc0 + (uint64_t)((j & 1) * (NQ * 128 >> 4));
      for (int p = 0; p < np; ++p) {
        mbar_wait(&c_full[vs], vph);  // landed long ago (S(j) read it): the wait orders this warp's reads behind the copy
        tc_fence_after();
        if (elected) {
          const uint64_t vd = vdesc0 + (uint64_t)(vs * (kPair >> 4));
#pragma unroll
          for (int k = 0; k < 4; ++k) umma_f16_ss(tmem_O + p * NQ, vd + k * (16 * 128 >> 4), pd + k * 2, idesc_o, k != 0 ? 1u : (j != 0 ? 1u : 0u));
          umma_commit(&c_empty[vs]);
        }
        if (++vs == CS) { vs = 0; vph ^= 1; }
      }
      if (elected) umma_commit(&pv_done[j & 1]);
    }
  } else {
    const int qd = warp & 3;
    const int t = qd * 32 + lane;
    const uint32_t lane_sel = static_cast<uint32_t>(qd * 32) << 16;
    // lanes 0..15 hold the rows of S^T; lane l + 16 takes the upper half of the heads of lane l's row
    constexpr int HN = NQ / 2;
    const int kv = qd * 16 + (lane & 15);  // position within the tile
    const int g0 = lane < 16 ? 0 : HN;     // first head of this lane
    float m_used[HN], l_run[HN];
#pragma unroll
    for (int g = 0; g < HN; ++g) { m_used[g] = -INFINITY; l_run[g] = 0.f; }
    const float scale_log2 = a.scale * 1.4426950408889634f;
    for (int j = 0; j < n_tiles; ++j) {
      mbar_wait(&s_full[j & 1], (j >> 1) & 1);
      tc_fence_after();
      uint32_t sv[NQ];
      tmem_ld_cols<NQ>(tmem_S + lane_sel + (j & 1) * NQ, sv);
      tmem_ld_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&s_empty[j & 1]);
      const int pos = (t_begin + j) * PAGE + kv;
      const bool valid = pos < ctx && pos >= kv_lo;
      float sc[HN];
      bool need = j == 0;
#pragma unroll
      for (int g = 0; g < HN; ++g) {
        const uint32_t up = __shfl_sync(0xffffffffu, sv[HN + g], lane & 15);
        sc[g] = valid ? __uint_as_float(lane < 16 ? sv[g] : up) * scale_log2 : -INFINITY;
        need |= sc[g] > m_used[g] + kRescale;
      }
      if (j >= 2) {  // the P buffer is free
        mbar_wait(&pv_done[j & 1], ((j >> 1) - 1) & 1);
        tc_fence_after();
      }
      if (bar_any(need)) {
#pragma unroll
        for (int g = 0; g < HN; ++g) {
          float mx = sc[g];
#pragma unroll
          for (int o = 8; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
          if ((lane & 15) == 0) sRed[qd * NQ + g0 + g] = mx;
        }
        bar_sync(1, 128);
#pragma unroll
        for (int g = 0; g < HN; ++g) {
          const int h = g0 + g;
          const float tm = fmaxf(fmaxf(sRed[h], sRed[NQ + h]), fmaxf(sRed[2 * NQ + h], sRed[3 * NQ + h]));
          float f = 1.f;
          if (tm > m_used[g] + kRescale) {  // the first tile too (m_used = -inf; some position of every tile is visible)
            f = m_used[g] == -INFINITY ? 0.f : fast_exp2(m_used[g] - tm);
            m_used[g] = tm;
            l_run[g] *= f;
          }
          if (qd == 0 && (lane & 15) == 0) sFac[h] = f;
        }
        bar_sync(1, 128);  // sRed may be rewritten, sFac is complete
        if (j > 0) {
          mbar_wait(&pv_done[(j - 1) & 1], ((j - 1) >> 1) & 1);  // O^T is consistent
          tc_fence_after();
          for (int p = 0; p < np; ++p) {
            uint32_t o[NQ];
            tmem_ld_cols<NQ>(tmem_O + lane_sel + p * NQ, o);
            tmem_ld_wait();
#pragma unroll
            for (int g = 0; g < NQ; ++g) o[g] = __float_as_uint(__uint_as_float(o[g]) * sFac[g]);
            tmem_st_32x32b_x16(tmem_O + lane_sel + p * NQ, *reinterpret_cast<uint32_t(*)[16]>(&o[0]));
            if constexpr (NQ == 32) tmem_st_32x32b_x16(tmem_O + lane_sel + p * NQ + 16, *reinterpret_cast<uint32_t(*)[16]>(&o[16]));
          }
          tmem_st_wait();
        }
      }
      uint8_t* dst = sP + (j & 1) * (NQ * 128) + g0 * 128 + (kv & 7) * 2;
#pragma unroll
      for (int g = 0; g < HN; ++g) {  // g0 is a multiple of 8: the swizzle phase of row g0 + g is g & 7
        const float pr = fast_exp2(sc[g] - m_used[g]);
        l_run[g] += pr;
        *reinterpret_cast<bf16*>(dst + g * 128 + (((kv >> 3) ^ (g & 7)) << 4)) = __float2bfloat16(pr);
      }
      fence_proxy_async_smem();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[j & 1]);
    }
    // ---- epilogue: O^T lane r, column g; l over all positions of the split
#pragma unroll
    for (int g = 0; g < HN; ++g) {
      float v = l_run[g];
#pragma unroll
      for (int o = 8; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
      if ((lane & 15) == 0) sRed[qd * NQ + g0 + g] = v;
      if (qd == 0 && (lane & 15) == 0) sFac[g0 + g] = m_used[g];
    }
    bar_sync(1, 128);
    if (t < NQ) sRed[t] = (sRed[t] + sRed[NQ + t]) + (sRed[2 * NQ + t] + sRed[3 * NQ + t]);
    bar_sync(1, 128);
    mbar_wait(&pv_done[(n_tiles - 1) & 1], ((n_tiles - 1) >> 1) & 1);
    tc_fence_after();
    for (int p = 0; p < np; ++p) {
      uint32_t o[NQ];
      tmem_ld_cols<NQ>(tmem_O + lane_sel + p * NQ, o);
      tmem_ld_wait();
      const int r = p * 128 + t;
      if (r < R) {
        if (num_splits == 1) {
#pragma unroll
          for (int g = 0; g < NQ; ++g) {
            if (g >= nh) break;
            float lg = sRed[g];
            if (a.sink) lg += fast_exp2(__bfloat162float(a.sink[h0 + g]) * 1.4426950408889634f - sFac[g]);
            a.ctx[((size_t)(h0 + g) * kTokRows + tq) * R + r] = __float2bfloat16(__uint_as_float(o[g]) / lg);
          }
        } else {
#pragma unroll
          for (int g = 0; g < NQ; ++g) ws[(size_t)g * (R + 2) + r] = __uint_as_float(o[g]);
        }
      }
    }
    if (num_splits > 1 && t < NQ) {
      ws[(size_t)t * (R + 2) + R] = sFac[t];
      ws[(size_t)t * (R + 2) + R + 1] = sRed[t];
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, kCols);
  }
}

// merges the splits of one (head, token): every thread weighs the splits itself (their maxima and sums are a few loads that all
// threads share), then sums four latent entries per pass
__global__ void __launch_bounds__(128) latent_combine_kernel(const float* __restrict__ ws, bf16* __restrict__ ctx, const bf16* __restrict__ sink,
                                                             int R, int NQ, int groups, int num_splits) {
  __shared__ float wts[kMaxSplits];
  pdl_wait();
  const int h = blockIdx.x, tq = blockIdx.y, hg = h / NQ, g = h % NQ;
  const float* base = ws + ((size_t)tq * groups + hg) * num_splits * NQ * (R + 2) + (size_t)g * (R + 2);
  const size_t stride = (size_t)NQ * (R + 2);
  if (threadIdx.x < 32) {
    const int s = threadIdx.x;
    const float ms = s < num_splits ? base[s * stride + R] : -INFINITY, ls = s < num_splits ? base[s * stride + R + 1] : 0.f;
    float m = ms;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
    const float w = ms == -INFINITY ? 0.f : fast_exp2(ms - m);
    float l = w * ls;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
    if (sink) l += fast_exp2(__bfloat162float(sink[h]) * 1.4426950408889634f - m);
    wts[s] = w / l;
  }
  __syncthreads();
  for (int r = threadIdx.x * 2; r < R; r += 256) {  // R is a multiple of 8
    float2 o = make_float2(0.f, 0.f);
#pragma unroll 4
    for (int s = 0; s < num_splits; ++s) {
      const float2 v = *reinterpret_cast<const float2*>(base + s * stride + r);
      o.x = fmaf(wts[s], v.x, o.x);
      o.y = fmaf(wts[s], v.y, o.y);
    }
    *reinterpret_cast<__nv_bfloat162*>(ctx + ((size_t)h * kTokRows + tq) * R + r) = __floats2bfloat162_rn(o.x, o.y);
  }
}

// expanded rows: c[row] and k_rot[row] copied from the cache rows of the runs' positions, 16 bytes per thread
__global__ void __launch_bounds__(128) latent_rows_kernel(const bf16* __restrict__ cache, const int32_t* __restrict__ page_table, int max_pages,
                                                          int R, int Dr, bf16* __restrict__ c, bf16* __restrict__ kr,
                                                          const __grid_constant__ LatentRuns runs) {
  const int row = blockIdx.x;
  int b = 0;
  while (b + 1 < runs.n && row >= runs.row0[b + 1]) ++b;
  const int pos = runs.pos0[b] + row - runs.row0[b];
  const size_t src = ((size_t)page_table[(size_t)runs.seq[b] * max_pages + pos / PAGE] * PAGE + pos % PAGE) * (R + Dr);
  for (int i = threadIdx.x * 8; i < R + Dr; i += 128 * 8) {
    const uint4 v = *reinterpret_cast<const uint4*>(cache + src + i);
    *reinterpret_cast<uint4*>(i < R ? c + (size_t)row * R + i : kr + (size_t)row * Dr + (i - R)) = v;
  }
}

// qh[h][tq][:] = q[tq][h * (Dk + Dr) : + Dk]
__global__ void __launch_bounds__(128) latent_q_heads_kernel(const bf16* __restrict__ q, int ldq, bf16* __restrict__ qh, int H, int Dk, int Dr) {
  const int tq = blockIdx.x, per = Dk / 8;
  for (int i = threadIdx.x; i < H * per; i += 128) {
    const int h = i / per, e = i % per * 8;
    *reinterpret_cast<uint4*>(qh + ((size_t)h * kTokRows + tq) * Dk + e) = *reinterpret_cast<const uint4*>(q + (size_t)tq * ldq + (size_t)h * (Dk + Dr) + e);
  }
}

template <int NQ>
bool pick_rings(int nc, int np, Rings* rings, size_t* smem) {
  const size_t fixed = (size_t)(nc + 1) * NQ * 128 + 2 * NQ * 128 + 5 * NQ * 4 + (2 * kMaxC + 2 * kMaxR + 9) * 8 + 16 + 1024;
  const size_t total = 227 * 1024;
  if (fixed >= total) return false;
  const size_t room = total - fixed, tile = (size_t)np * kPair + kSub;
  // about as many rotated parts as tiles of latents; at least two tiles of both (S of the next tile is issued while this tile's
  // latents are held)
  int rs = std::min<int>(kMaxR, (int)((room + tile - 1) / tile));
  while (rs > 2 && (room - (size_t)rs * kSub) / kPair < (size_t)2 * np) --rs;
  if (rs < 2 || room < (size_t)rs * kSub + (size_t)2 * np * kPair) return false;
  rings->rs = rs;
  rings->cs = std::min<int>(kMaxC, (int)((room - (size_t)rs * kSub) / kPair));
  *smem = fixed + (size_t)rings->cs * kPair + (size_t)rings->rs * kSub;
  return true;
}

int pick_nq(int H) { return H <= 16 ? 16 : 32; }

template <int NQ>
cudaError_t launch_decode(cudaStream_t s, const LatentDecodeArgs& a) {
  const int nc = (a.R + 63) / 64, np = (nc + 1) / 2, groups = (a.H + NQ - 1) / NQ;
  Rings rings;
  size_t smem = 0;
  if (!pick_rings<NQ>(nc, np, &rings, &smem)) return cudaErrorInvalidValue;
  CUtensorMap mc, mr, mql, mqr;
  const uint64_t rows = (uint64_t)a.num_pages * PAGE, stride = (uint64_t)(a.R + a.Dr) * 2;
  if (!make_tmap_2d(&mc, a.cache, TM_BF16, a.R, rows, stride, 64, PAGE)) return cudaErrorInvalidValue;
  if (!make_tmap_2d(&mr, a.cache + a.R, TM_BF16, a.Dr, rows, stride, 64, PAGE)) return cudaErrorInvalidValue;
  const uint64_t qs = (uint64_t)(a.Dk + a.Dr) * 2;
  if (!make_tmap_3d(&mql, a.q_lat, TM_BF16, a.R, kTokRows, a.H, (uint64_t)a.R * 2, (uint64_t)kTokRows * a.R * 2, 64, 1, NQ)) return cudaErrorInvalidValue;
  if (!make_tmap_3d(&mqr, a.q + a.Dk, TM_BF16, a.Dr, a.H, a.T, qs, (uint64_t)a.ldq * 2, 64, NQ, 1)) return cudaErrorInvalidValue;
  cudaError_t e = launch_k(latent_decode_kernel<NQ>, dim3(a.num_splits, groups, a.T), dim3(kThreads), smem, s, true, mc, mr, mql, mqr, a, rings, a.num_splits);
  if (e != cudaSuccess || a.num_splits == 1) return e;
  return launch_k(latent_combine_kernel, dim3(a.H, a.T), dim3(128), 0, s, true, (const float*)a.workspace, a.ctx, a.sink, a.R, NQ, groups, a.num_splits);
}

}  // namespace

bool latent_decode_ok(int Dk, int R, int Dr) {
  return Dk > 0 && Dk % 8 == 0 && R > 0 && R % 8 == 0 && R <= 512 && Dr > 0 && Dr % 8 == 0 && Dr <= 64;
}
int latent_decode_splits(int T, int H, int max_keys, int sms) {
  const int blocks = T * ((H + pick_nq(H) - 1) / pick_nq(H));
  const int tiles = std::max(1, (max_keys + PAGE - 1) / PAGE);
  return std::max(1, std::min(std::min(kMaxSplits, (tiles + 1) / 2), sms / std::max(1, blocks)));
}
size_t latent_decode_ws_floats(int T, int H, int R, int splits) {
  return splits <= 1 ? 0 : (size_t)T * ((H + pick_nq(H) - 1) / pick_nq(H)) * splits * pick_nq(H) * (R + 2);
}

cudaError_t attn_latent_init() {
  cudaError_t e = cudaFuncSetAttribute(latent_decode_kernel<16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
  return e != cudaSuccess ? e : cudaFuncSetAttribute(latent_decode_kernel<32>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
}

cudaError_t latent_decode(cudaStream_t s, const LatentDecodeArgs& a) {
  if (a.T <= 0) return cudaSuccess;
  if (a.T > kTokRows || !latent_decode_ok(a.Dk, a.R, a.Dr) || a.page_size != PAGE || a.num_splits < 1 || a.num_splits > kMaxSplits || a.num_pages <= 0 || a.window < 0 ||
      a.ldq % 8 || (a.num_splits > 1 && !a.workspace))
    return cudaErrorInvalidValue;
  return pick_nq(a.H) == 16 ? launch_decode<16>(s, a) : launch_decode<32>(s, a);
}

cudaError_t latent_rows(cudaStream_t s, const bf16* cache, const int32_t* page_table, int max_pages, int R, int Dr, bf16* c, bf16* k_rot,
                        const LatentRuns& runs, int rows) {
  if (rows <= 0) return cudaSuccess;
  if (R % 8 || Dr % 8 || runs.n <= 0 || runs.n > AttnRuns::kMax) return cudaErrorInvalidValue;
  latent_rows_kernel<<<rows, 128, 0, s>>>(cache, page_table, max_pages, R, Dr, c, k_rot, runs);
  return cudaGetLastError();
}

cudaError_t latent_q_heads(cudaStream_t s, const bf16* q, int ldq, bf16* qh, int T, int H, int Dk, int Dr) {
  if (T <= 0) return cudaSuccess;
  if (T > kTokRows || Dk % 8 || Dr % 8 || ldq % 8) return cudaErrorInvalidValue;
  latent_q_heads_kernel<<<T, 128, 0, s>>>(q, ldq, qh, H, Dk, Dr);
  return cudaGetLastError();
}

}  // namespace hb
