// Linear attention with one constant decay per head over long prompt portions, on the tensor cores (HB_MIXER_LIGHTNING, bf16
// mode).  With chunks of 128 tokens, i / j counted inside the chunk, n tokens in it and S the state behind the chunk before:
//
//   A = Q K^T                                   o_i = sum_(j <= i) a^(i-j) A_ij v_j + a^(i+1) S^T q_i
//   S <- a^n S + sum_j a^(n-1-j) k_j v_j^T
//
// q, k, v are bf16 rows (the activations' own rounding); everything behind them is fp32: the decay-weighted scores, the weighted
// values and the state travel through the bf16 tensor-core operands as two terms each, x = hi + lo with hi = bf16(x) and
// lo = bf16(x - hi) (16 significant bits), products accumulate in fp32, and the state itself stays an fp32 accumulator in TMEM
// from the first chunk to the last.
//
// One CTA per (entry, head, NV value columns) walks the entry's chunks; an entry that starts at position 0 starts from zeros.
//   warp 8    : TMA loads (Q single, K / V in two slots) and all products
//   warps 0-7 : thread (row r = 32 (warp & 3) + lane, half warp >> 2) turns S into operand tiles and decays it in TMEM, weighs
//               a row of A in place (P, the A operand of P V, stays in TMEM), weighs a row of V, and writes output rows
// TMEM columns: [S (NV) | A, then P hi | P lo (128) | S^T q (NV) | P V (NV)].
// Waits are bounded: one that runs out marks the launch as failed (the host reads the flag behind the step), and the block runs
// on without loads, products or stores until it has given its TMEM back.
#include <math.h>

#include <algorithm>

#include "kernels.h"
#include "launch.h"
#include "ptx.cuh"
#include "tma_host.h"

namespace hb {
namespace {

constexpr int C = 128;            // tokens per chunk
constexpr int kThreads = 288;
constexpr int kSubTile = C * 128;  // 64 bf16 columns of 128 rows
constexpr long long kWaitCycles = 2000000000ll;

template <int NV>
struct Cfg {
  static constexpr int Q = 2 * kSubTile, K = 2 * kSubTile, V = NV / 64 * kSubTile;
  static constexpr int W = 2 * V;  // S hi | S lo, then the weighted values hi | lo
  static constexpr int TILES = Q + 2 * (K + V) + W;
  static constexpr int SMEM = 1024 + TILES + 256 * 4 + 16 * 8;
  static constexpr uint32_t COLS = 512;
};

struct Bars {
  uint64_t *q_full, *kv_full, *a_full, *m2_done, *o_full, *s_done, *s_ready, *p_ready, *vd_ready, *o_free;
};

template <int NV>
__global__ void __launch_bounds__(kThreads, 1)
lin_chunk_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                 const __grid_constant__ CUtensorMap map_v, const __grid_constant__ LinChunkArgs a) {
  using G = Cfg<NV>;
  constexpr int VC = NV / 2;  // value columns per thread
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = smem;
  uint8_t* sK = sQ + G::Q;         // [2]
  uint8_t* sV = sK + 2 * G::K;     // [2]
  uint8_t* sW = sV + 2 * G::V;     // [hi | lo][NV / 64 sub-tiles][128 rows][128 B]
  float* tz = reinterpret_cast<float*>(sW + G::W);  // tz[127 + d] = decay^d, 0 for d < 0
  const float* pw = tz + 127;
  uint64_t* bars = reinterpret_cast<uint64_t*>(tz + 256);
  const Bars B{bars, bars + 1, bars + 3, bars + 4, bars + 5, bars + 6, bars + 7, bars + 8, bars + 9, bars + 10};
  uint32_t* tmem_ptr = reinterpret_cast<uint32_t*>(bars + 11);
  volatile int* dead = reinterpret_cast<volatile int*>(tmem_ptr + 1);

  const int b = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * NV;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t0 = a.cu[b], n_tok = a.cu[b + 1] - t0;
  if (n_tok <= 0) return;
  const int chunks = (n_tok + C - 1) / C;

  if (threadIdx.x == 0) {
    *dead = 0;
    mbar_init(B.q_full, 1);
    mbar_init(B.kv_full, 1);
    mbar_init(B.kv_full + 1, 1);
    mbar_init(B.a_full, 1);
    mbar_init(B.m2_done, 1);
    mbar_init(B.o_full, 1);
    mbar_init(B.s_done, 1);
    mbar_init(B.s_ready, 8);
    mbar_init(B.p_ready, 8);
    mbar_init(B.vd_ready, 8);
    mbar_init(B.o_free, 8);
    fence_barrier_init();
  }
  if (warp == 8) {
    tma_prefetch_desc(&map_q);
    tma_prefetch_desc(&map_k);
    tma_prefetch_desc(&map_v);
    tmem_alloc(tmem_ptr, G::COLS);
    tmem_relinquish();
  }
  for (int i = threadIdx.x; i < 256; i += kThreads) tz[i] = i < 127 ? 0.f : (float)pow((double)a.decay[h], (double)(i - 127));
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = __shfl_sync(0xffffffffu, *tmem_ptr, 0);
  const uint32_t tS = tmem, tA = tmem + NV, tO1 = tA + C, tO2 = tO1 + NV;

  auto wait = [&](uint64_t* bar, uint32_t parity) {
    if (*dead || mbar_try_wait(bar, parity)) return;
    const long long c0 = clock64();
    while (!mbar_try_wait(bar, parity)) {
      if (*dead) return;
      if (clock64() - c0 > kWaitCycles) {
        *dead = 1;
        *a.error = 1;
        return;
      }
    }
  };

  if (warp == 8) {
    const bool leader = elect_one_sync();
    constexpr uint32_t id_qk = umma_idesc_bf16(C, C, 0, 0), id_mn = umma_idesc_bf16(C, NV, 0, 1), id_upd = umma_idesc_bf16(128, NV, 1, 1);
    const uint64_t qd = umma_desc_kmajor_sw128(smem_u32(sQ)), kd0 = umma_desc_kmajor_sw128(smem_u32(sK));
    const uint64_t kt0 = umma_desc_mnmajor_sw128(smem_u32(sK), kSubTile, 1024), vd0 = umma_desc_mnmajor_sw128(smem_u32(sV), kSubTile, 1024);
    const uint64_t wd = umma_desc_mnmajor_sw128(smem_u32(sW), kSubTile, 1024);
    const int nk = a.Dk <= 64 ? 4 : 8;  // 16-channel steps of the products over the key channels
    auto load_q = [&](int c) {
      if (leader && !*dead) {
        mbar_arrive_expect_tx(B.q_full, G::Q);
        for (int s = 0; s < 2; ++s) tma_load_3d(sQ + s * kSubTile, &map_q, B.q_full, s * 64, h, t0 + c * C);
      }
    };
    auto load_kv = [&](int c) {
      const int s = c & 1;
      if (leader && !*dead) {
        mbar_arrive_expect_tx(B.kv_full + s, G::K + G::V);
        for (int i = 0; i < 2; ++i) tma_load_3d(sK + s * G::K + i * kSubTile, &map_k, B.kv_full + s, i * 64, h, t0 + c * C);
        for (int i = 0; i < NV / 64; ++i) tma_load_3d(sV + s * G::V + i * kSubTile, &map_v, B.kv_full + s, v0 + i * 64, h, t0 + c * C);
      }
    };
    load_q(0);
    load_kv(0);
    for (int c = 0; c < chunks; ++c) {
      const int s = c & 1;
      const uint32_t ph = c & 1;
      wait(B.kv_full + s, (c >> 1) & 1);
      wait(B.q_full, ph);
      tc_fence_after();
      if (leader && !*dead) {
        const uint64_t kd = kd0 + (uint64_t)(s * (G::K >> 4));
        for (int k = 0; k < nk; ++k) {
          const uint64_t o = ((k >> 2) * kSubTile + (k & 3) * 32) >> 4;
          umma_f16_ss(tA, qd + o, kd + o, id_qk, k != 0);
        }
        umma_commit(B.a_full);
      }
      wait(B.s_ready, ph);  // the state's operand tiles; the chunk before has left the other K / V slot
      if (c + 1 < chunks) load_kv(c + 1);
      if (c > 0) wait(B.o_free, (c - 1) & 1);
      tc_fence_after();
      if (leader && !*dead) {
        for (int k = 0; k < 2 * nk; ++k) {
          const int kk = k % nk;
          umma_f16_ss(tO1, qd + (((kk >> 2) * kSubTile + (kk & 3) * 32) >> 4), wd + (((k / nk) * G::V + kk * 16 * 128) >> 4), id_mn, k != 0);
        }
        umma_commit(B.m2_done);
      }
      wait(B.p_ready, ph);
      tc_fence_after();
      if (leader && !*dead) {
        const uint64_t vd = vd0 + (uint64_t)(s * (G::V >> 4));
#pragma unroll
        for (int k = 0; k < 16; ++k) umma_f16_ts(tO2, tA + k * 8, vd + (((k & 7) * 16 * 128) >> 4), id_mn, k != 0);
        umma_commit(B.o_full);
      }
      wait(B.m2_done, ph);  // nothing reads Q any more
      if (c + 1 < chunks) load_q(c + 1);
      wait(B.vd_ready, ph);
      tc_fence_after();
      if (leader && !*dead) {
        const uint64_t kt = kt0 + (uint64_t)(s * (G::K >> 4));
#pragma unroll
        for (int k = 0; k < 16; ++k)
          umma_f16_ss(tS, kt + (((k & 7) * 16 * 128) >> 4), wd + (((k >> 3) * G::V + (k & 7) * 16 * 128) >> 4), id_upd, 1u);
        umma_commit(B.s_done);
      }
    }
    wait(B.s_done, (chunks - 1) & 1);
    if (*dead) {  // copies and products already issued get time to land before the block's memory goes away
      const long long c0 = clock64();
      while (clock64() - c0 < 20000000ll) {}
    }
  } else {
    const int r = (warp & 3) * 32 + lane, hf = warp >> 2;
    const uint32_t lanes = (uint32_t)(warp & 3) << 21;  // this warp's 32 TMEM lanes
    const int vc0 = hf * VC;                            // first value column of this thread
    const uint32_t row_off = (uint32_t)(vc0 / 64) * kSubTile + (uint32_t)r * 128;
    const int ch0 = vc0 % 64 / 8;                       // its first 16-byte piece inside the 128-byte row
    float* st = a.state + (size_t)a.slots[b] * a.slot_stride + (size_t)h * a.Dk * a.Dv + (size_t)r * a.Dv + v0 + vc0;
    const bool fresh = a.first_pos[b] == 0;
    auto arrive = [&](uint64_t* bar) {
      __syncwarp();
      if (lane == 0) mbar_arrive(bar);
    };
    // x[8] as two bf16 terms into the same 16-byte piece of both halves of the operand tiles
    auto put_split = [&](int piece, const float (&x)[8]) {
      uint4 hi, lo;
      uint32_t* hp = &hi.x;
      uint32_t* lp = &lo.x;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        hp[e] = pack_bf16x2(x[2 * e], x[2 * e + 1]);
        const float2 f = unpack_bf16x2(hp[e]);
        lp[e] = pack_bf16x2(x[2 * e] - f.x, x[2 * e + 1] - f.y);
      }
      uint8_t* d = sW + row_off + (((ch0 + piece) ^ (r & 7)) << 4);
      *reinterpret_cast<uint4*>(d) = hi;
      *reinterpret_cast<uint4*>(d + G::V) = lo;
    };
    for (int c = 0; c < chunks; ++c) {
      const uint32_t ph = c & 1;
      const int n = min(C, n_tok - c * C);
      // ---- the state: operand tiles, then decayed in place
      if (c > 0) {
        wait(B.s_done, (c - 1) & 1);
        tc_fence_after();
      }
      const float dec = pw[n];
#pragma unroll
      for (int p = 0; p < VC / 32; ++p) {
        uint32_t x[32];
        if (c > 0) {
          tmem_ld_32x32b_x32(tS + lanes + vc0 + p * 32, x);
          tmem_ld_wait();
        } else {
#pragma unroll
          for (int q = 0; q < 8; ++q) {
            float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
            if (!fresh && r < a.Dk && v0 + vc0 + p * 32 + q * 4 < a.Dv) f = *reinterpret_cast<const float4*>(st + p * 32 + q * 4);
            x[4 * q] = __float_as_uint(f.x); x[4 * q + 1] = __float_as_uint(f.y); x[4 * q + 2] = __float_as_uint(f.z); x[4 * q + 3] = __float_as_uint(f.w);
          }
        }
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          float f[8];
#pragma unroll
          for (int e = 0; e < 8; ++e) f[e] = __uint_as_float(x[8 * q + e]);
          put_split(p * 4 + q, f);
        }
#pragma unroll
        for (int e = 0; e < 32; ++e) x[e] = __float_as_uint(__uint_as_float(x[e]) * dec);
        tmem_st_32x32b_x16(tS + lanes + vc0 + p * 32, *reinterpret_cast<uint32_t(*)[16]>(&x[0]));
        tmem_st_32x32b_x16(tS + lanes + vc0 + p * 32 + 16, *reinterpret_cast<uint32_t(*)[16]>(&x[16]));
      }
      tmem_st_wait();
      fence_proxy_async_smem();
      tc_fence_before();
      arrive(B.s_ready);
      // ---- P_ij = a^(i-j) A_ij (zero above the diagonal), j in this thread's half of the row
      wait(B.a_full, ph);
      tc_fence_after();
      {
        uint32_t hi[32], lo[32];
        const float* tw = pw + r - hf * 64;
#pragma unroll
        for (int p = 0; p < 2; ++p) {
          uint32_t x[32];
          tmem_ld_32x32b_x32(tA + lanes + hf * 64 + p * 32, x);
          tmem_ld_wait();
#pragma unroll
          for (int e = 0; e < 16; ++e) {
            const int j = p * 32 + 2 * e;
            const float f0 = __uint_as_float(x[2 * e]) * tw[-j], f1 = __uint_as_float(x[2 * e + 1]) * tw[-j - 1];
            hi[p * 16 + e] = pack_bf16x2(f0, f1);
            const float2 f = unpack_bf16x2(hi[p * 16 + e]);
            lo[p * 16 + e] = pack_bf16x2(f0 - f.x, f1 - f.y);
          }
        }
        tc_fence_before();
        bar_sync(1, 256);  // both halves of every row have been read: P takes A's columns
        tc_fence_after();
        const uint32_t d = tA + lanes + hf * 32;
        tmem_st_32x32b_x16(d, *reinterpret_cast<uint32_t(*)[16]>(&hi[0]));
        tmem_st_32x32b_x16(d + 16, *reinterpret_cast<uint32_t(*)[16]>(&hi[16]));
        tmem_st_32x32b_x16(d + 64, *reinterpret_cast<uint32_t(*)[16]>(&lo[0]));
        tmem_st_32x32b_x16(d + 80, *reinterpret_cast<uint32_t(*)[16]>(&lo[16]));
        tmem_st_wait();
        tc_fence_before();
        arrive(B.p_ready);
      }
      // ---- a^(n-1-j) v_j into the tiles the state's product has left
      wait(B.m2_done, ph);
      wait(B.kv_full + (c & 1), (c >> 1) & 1);
      {
        const float w = r < n ? pw[n - 1 - r] : 0.f;
        const uint8_t* src = sV + (c & 1) * G::V + row_off;
#pragma unroll
        for (int q = 0; q < VC / 8; ++q) {
          const uint4 u = *reinterpret_cast<const uint4*>(src + (((ch0 + q) ^ (r & 7)) << 4));
          float f[8];
          unpack_bf16x8(u, f);
#pragma unroll
          for (int e = 0; e < 8; ++e) f[e] *= w;
          put_split(q, f);
        }
        fence_proxy_async_smem();
        arrive(B.vd_ready);
      }
      // ---- output rows
      wait(B.o_full, ph);
      tc_fence_after();
      const float w1 = pw[r + 1];
      float* o = a.out + (size_t)(t0 + c * C + r) * a.ldo + (size_t)h * a.Dv + v0 + vc0;
#pragma unroll
      for (int p = 0; p < VC / 16; ++p) {
        uint32_t x1[16], x2[16];
        tmem_ld_32x32b_x16(tO1 + lanes + vc0 + p * 16, x1);
        tmem_ld_32x32b_x16(tO2 + lanes + vc0 + p * 16, x2);
        tmem_ld_wait();
        if (r < n && !*dead) {
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            float4 f;
            f.x = fmaf(w1, __uint_as_float(x1[4 * q]), __uint_as_float(x2[4 * q]));
            f.y = fmaf(w1, __uint_as_float(x1[4 * q + 1]), __uint_as_float(x2[4 * q + 1]));
            f.z = fmaf(w1, __uint_as_float(x1[4 * q + 2]), __uint_as_float(x2[4 * q + 2]));
            f.w = fmaf(w1, __uint_as_float(x1[4 * q + 3]), __uint_as_float(x2[4 * q + 3]));
            if (v0 + vc0 + p * 16 + q * 4 < a.Dv) *reinterpret_cast<float4*>(o + p * 16 + q * 4) = f;
          }
        }
      }
      tc_fence_before();
      arrive(B.o_free);
    }
    wait(B.s_done, (chunks - 1) & 1);
    tc_fence_after();
#pragma unroll
    for (int p = 0; p < VC / 16; ++p) {
      uint32_t x[16];
      tmem_ld_32x32b_x16(tS + lanes + vc0 + p * 16, x);
      tmem_ld_wait();
      if (r < a.Dk && !*dead) {
#pragma unroll
        for (int q = 0; q < 4; ++q)
          if (v0 + vc0 + p * 16 + q * 4 < a.Dv)
            *reinterpret_cast<float4*>(st + p * 16 + q * 4) = make_float4(__uint_as_float(x[4 * q]), __uint_as_float(x[4 * q + 1]), __uint_as_float(x[4 * q + 2]),
                                                                          __uint_as_float(x[4 * q + 3]));
      }
    }
    tc_fence_before();
  }
  __syncthreads();
  if (warp == 8) {
    tc_fence_after();
    tmem_dealloc(tmem, G::COLS);
  }
}

template <int NV>
cudaError_t launch(cudaStream_t s, const LinChunkArgs& a) {
  CUtensorMap mq, mk, mv;
  const uint64_t ld = (uint64_t)a.ld * 2, T = a.T, H = a.H;
  if (!make_tmap_3d(&mq, a.q, TM_BF16, a.Dk, H, T, (uint64_t)a.Dk * 2, ld, 64, 1, C)) return cudaErrorInvalidValue;
  if (!make_tmap_3d(&mk, a.k, TM_BF16, a.Dk, H, T, (uint64_t)a.Dk * 2, ld, 64, 1, C)) return cudaErrorInvalidValue;
  if (!make_tmap_3d(&mv, a.v, TM_BF16, a.Dv, H, T, (uint64_t)a.Dv * 2, ld, 64, 1, C)) return cudaErrorInvalidValue;
  lin_chunk_kernel<NV><<<dim3(a.B, a.H, (a.Dv + NV - 1) / NV), kThreads, Cfg<NV>::SMEM, s>>>(mq, mk, mv, a);
  return cudaGetLastError();
}

}  // namespace

static_assert(Cfg<128>::SMEM <= 227 * 1024, "shared memory of one CTA");

bool lin_chunk_ok(int Dk, int Dv) { return Dk > 0 && Dv > 0 && Dk <= 128 && Dk % 8 == 0 && Dv % 8 == 0; }

cudaError_t stack_lightning_init() {
  cudaError_t e = cudaFuncSetAttribute(lin_chunk_kernel<64>, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg<64>::SMEM);
  if (e != cudaSuccess) return e;
  return cudaFuncSetAttribute(lin_chunk_kernel<128>, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg<128>::SMEM);
}

cudaError_t lin_chunk(cudaStream_t s, const LinChunkArgs& a) {
  if (a.B <= 0 || a.T <= 0) return cudaSuccess;
  if (!lin_chunk_ok(a.Dk, a.Dv) || a.H <= 0 || a.ld % 8 || a.ldo % 4 || a.slot_stride % 4 || !a.error ||
      (((uintptr_t)a.q | (uintptr_t)a.k | (uintptr_t)a.v | (uintptr_t)a.out | (uintptr_t)a.state) & 15))
    return cudaErrorInvalidValue;
  return a.Dv <= 64 ? launch<64>(s, a) : launch<128>(s, a);
}

}  // namespace hb
