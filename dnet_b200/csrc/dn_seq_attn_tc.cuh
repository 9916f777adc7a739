// dn_seq_attn_tc.cuh -- attention with sigmoid weights for prompt portions on the 5th-generation tensor cores
// (tcgen05 + TMEM + TMA), libdnet_b200_seq.so, bf16.
//
// A key's weight depends on its own score alone, so there is no running maximum, no rescaling and no sum: the output
// accumulates in TMEM over all key tiles of a row without being read in between.  A CTA takes one key / value head, up to
// SG_HEADS of its query heads and TB = floor(128 / heads) consecutive tokens of one entry: the 128 MMA rows are heads x
// tokens, so that a staged key / value tile serves the whole group.  Per tile of 128 keys (two pages, by TMA through the
// block table):
//   S = Q K^T       A = Q [128 x DK] K-major, B = K tile [128 x DK] K-major          TMEM columns 0-127 / 128-255 in turn
//   P = weights     sixteen warps, four per TMEM lane quarter (a quarter of the columns each): one score = one fused
//                   multiply-add with the tabled bias, one exponential, half a reciprocal (two weights share one)
//   O += P V        A = P as a bf16 pair hi + lo (16 bits of each weight's mantissa), B = V tile, MN-major     TMEM 256-383
// S of tile j + 1 is formed while the weights of tile j are; S, K and V have two buffers each, P one.
// Per row the tiles are visited in ascending position; a tile that a row does not see adds zeros.
// Roles: warp 0 TMA producer, warp 1 MMA issuer, warp 2 TMEM allocator, warps 4-19 weights and output.
#pragma once
#include "dn_gemm_tc.cuh"
#include "dn_seq_kernels.cuh"

namespace dnseq {

constexpr int SG_HEADS = 16, SG_THREADS = 640, SG_HALF = 16384;      // SG_HALF: bytes of 128 rows x 64 columns
constexpr float SG_LOG2E = 1.4426950408889634f;

struct SigParams {
  const bf16* q;          // [N][H][DK]
  bf16* out;              // [N][H][DV]
  const float* tab;       // [H][D]: (bias at distance d - offset_h) log2(e)
  const float* gate;      // [N][H] pre-activations (null: none)
  int H, G, chunk, window, D, hpc;      // hpc: query heads of a CTA
  float scale;
  unsigned int* err;
};

// exponential and reciprocal of the special-function unit (a few units in the last place of fp32, far inside what the bf16
// operands carry)
__device__ __forceinline__ float sg_ex2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ float sg_rcp(float x) { float y; asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
// 32 lanes x 32 consecutive fp32 columns of this warp's TMEM quarter
__device__ __forceinline__ void sg_ld32(uint32_t taddr, float (&v)[32]) {
  uint32_t r[32];
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x32.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31}, [%32];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]), "=r"(r[10]), "=r"(r[11]),
        "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]), "=r"(r[16]), "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]), "=r"(r[21]), "=r"(r[22]),
        "=r"(r[23]), "=r"(r[24]), "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]), "=r"(r[30]), "=r"(r[31])
      : "r"(taddr));
  asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
  for (int i = 0; i < 32; ++i) v[i] = __uint_as_float(r[i]);
}

// tab[h][d] = (r1_h ln(1 + r2_h d) - off_h) log2(e)
__global__ void k_dist_table(const bf16* __restrict__ r1, const bf16* __restrict__ r2, const bf16* __restrict__ off, int D, float* __restrict__ tab) {
  const int h = blockIdx.y, d = blockIdx.x * blockDim.x + threadIdx.x;
  if (d >= D) return;
  const float b = r1 ? ldf(r1 + h) * log1pf(ldf(r2 + h) * (float)d) : 0.f;
  tab[(size_t)h * D + d] = (b - ldf(off + h)) * SG_LOG2E;
}

__host__ __device__ constexpr size_t sg_smem(int DK, int DV) { return (size_t)(3 * (DK / 64) + 2 * (DV / 64) + 4) * SG_HALF + 1024 + 256; }

template <int DK, int DV>
__global__ void __launch_bounds__(SG_THREADS, 1) k_sig_attn_tc(const __grid_constant__ CUtensorMap mapK, const __grid_constant__ CUtensorMap mapV, Batch b, SigParams p) {
  constexpr int KB = DK / 64 * SG_HALF, VB = DV / 64 * SG_HALF;      // bytes of a K (Q) and a V tile
  extern __shared__ __align__(1024) unsigned char sg_raw[];
  unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(sg_raw) + 1023) & ~(uintptr_t)1023);
  unsigned char *sQ = smem, *sK = sQ + KB, *sV = sK + 2 * KB, *sPh = sV + 2 * VB, *sPl = sPh + 2 * SG_HALF;
  uint64_t* bars = reinterpret_cast<uint64_t*>(sPl + 2 * SG_HALF);
  uint64_t *k_full = bars, *k_empty = bars + 2, *s_full = bars + 4, *s_empty = bars + 6, *v_full = bars + 8, *v_empty = bars + 10, *p_full = bars + 12,
           *p_empty = bars + 13, *o_full = bars + 14;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 15);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  // which entry, which of its blocks of TB tokens, which heads
  const int TB = 128 / p.hpc;
  int e = 0, t = blockIdx.x;
  for (; e < b.E; e++) {
    const int nt = (b.ent_start[e + 1] - b.ent_start[e] + TB - 1) / TB;
    if (t < nt) break;
    t -= nt;
  }
  if (e >= b.E) return;
  const int R = p.H / p.G, per = (R + p.hpc - 1) / p.hpc, g = blockIdx.y / per, h0 = g * R + (blockIdx.y % per) * p.hpc, nh = min(p.hpc, (g + 1) * R - h0);
  const int s0 = b.ent_start[e] + t * TB, nq = min(TB, b.ent_start[e + 1] - s0);
  const int p_first = b.ent_pos0[e] + t * TB, kv_max = p_first + nq;      // keys up to the last query's position
  const int32_t* bt = b.bt + (size_t)b.ent_slot[e] * b.max_pages;
  const int page0 = attn_lo(p_first, p.chunk, p.window) / PAGE, pages = (kv_max + PAGE - 1) / PAGE, n_tiles = (pages - page0 + 1) / 2;

  if (threadIdx.x == 0) {
    constexpr int WW = SG_THREADS / 32 - 4;      // warps that form weights
    for (int i = 0; i < 2; i++) {
      dn::mbar_init(&k_full[i], 1); dn::mbar_init(&k_empty[i], 1); dn::mbar_init(&s_full[i], 1); dn::mbar_init(&s_empty[i], WW);
      dn::mbar_init(&v_full[i], 1); dn::mbar_init(&v_empty[i], 1);
    }
    dn::mbar_init(p_full, WW); dn::mbar_init(p_empty, 1); dn::mbar_init(o_full, 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 2) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], 512;" ::"r"(dn::smem_u32(tmem_slot)) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  // Q rows (head, token), zero where there is none, in the layout TMA's 128-byte swizzle gives
  for (int i = threadIdx.x; i < 128 * (DK / 8); i += SG_THREADS) {
    const int r = i / (DK / 8), c = i % (DK / 8), hr = r / TB, tr = r % TB;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (hr < nh && tr < nq) v = *reinterpret_cast<const uint4*>(p.q + ((size_t)(s0 + tr) * p.H + h0 + hr) * DK + c * 8);
    *reinterpret_cast<uint4*>(sQ + dn::at_swz(r, c)) = v;
  }
  asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  dn::tc_fence_before();
  __syncthreads();
  dn::tc_fence_after();
  const uint32_t tmem = *tmem_slot, tO = tmem + 256;

  if (warp == 0) {
    if (lane == 0) {
      for (int j = 0; j <= n_tiles; j++) {
        if (j < n_tiles) {
          const int st = j & 1;
          const int pg0 = bt[page0 + 2 * j], pg1 = page0 + 2 * j + 1 < pages ? bt[page0 + 2 * j + 1] : pg0;      // an unused half is masked
          unsigned char* dst = sK + st * KB;
          dn::mbar_wait(&k_empty[st], ((j >> 1) & 1) ^ 1u, p.err);
          dn::mbar_arrive_expect_tx(&k_full[st], KB);
#pragma unroll
          for (int hf = 0; hf < DK / 64; hf++) {
            dn::tma_load_2d(dst + hf * SG_HALF, &mapK, g * DK + hf * 64, pg0 * PAGE, &k_full[st]);
            dn::tma_load_2d(dst + hf * SG_HALF + SG_HALF / 2, &mapK, g * DK + hf * 64, pg1 * PAGE, &k_full[st]);
          }
        }
        if (j > 0) {
          const int jv = j - 1, st = jv & 1;
          unsigned char* dst = sV + st * VB;
          const int pg0 = bt[page0 + 2 * jv], pg1 = page0 + 2 * jv + 1 < pages ? bt[page0 + 2 * jv + 1] : pg0;
          dn::mbar_wait(&v_empty[st], ((jv >> 1) & 1) ^ 1u, p.err);
          dn::mbar_arrive_expect_tx(&v_full[st], VB);
#pragma unroll
          for (int hf = 0; hf < DV / 64; hf++) {
            dn::tma_load_2d(dst + hf * SG_HALF, &mapV, g * DV + hf * 64, pg0 * PAGE, &v_full[st]);
            dn::tma_load_2d(dst + hf * SG_HALF + SG_HALF / 2, &mapV, g * DV + hf * 64, pg1 * PAGE, &v_full[st]);
          }
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t idesc_s = dn::tc_instr_desc(128, 128), idesc_o = dn::tc_instr_desc(128, DV) | (1u << 16);      // V is MN-major
      for (int j = 0; j <= n_tiles; j++) {
        if (j < n_tiles) {
          const int st = j & 1;
          const uint32_t ph = (j >> 1) & 1;
          dn::mbar_wait(&k_full[st], ph, p.err);
          dn::mbar_wait(&s_empty[st], ph ^ 1u, p.err);
          dn::tc_fence_after();
#pragma unroll
          for (int hf = 0; hf < DK / 64; hf++) {
            const uint64_t ad = dn::tc_smem_desc(sQ + hf * SG_HALF), bd = dn::tc_smem_desc(sK + st * KB + hf * SG_HALF);
#pragma unroll
            for (int k = 0; k < 4; k++) dn::tc_mma(tmem + st * 128, ad + (uint64_t)(2 * k), bd + (uint64_t)(2 * k), idesc_s, (hf | k) ? 1u : 0u);
          }
          dn::tc_commit(&k_empty[st]);
          dn::tc_commit(&s_full[st]);
        }
        if (j > 0) {
          const int st = (j - 1) & 1;
          dn::mbar_wait(p_full, st, p.err);
          dn::mbar_wait(&v_full[st], ((j - 1) >> 1) & 1, p.err);
          dn::tc_fence_after();
          const uint64_t vd = dn::tc_smem_desc_mn(sV + st * VB, SG_HALF, 1024);
#pragma unroll
          for (int part = 0; part < 2; part++) {
#pragma unroll
            for (int kk = 0; kk < 8; kk++) {
              const uint64_t ad = dn::tc_smem_desc((part ? sPl : sPh) + (kk >> 2) * SG_HALF) + (uint64_t)(2 * (kk & 3));
              dn::tc_mma(tO, ad, vd + (uint64_t)(kk * (2048 >> 4)), idesc_o, (j > 1 || part || kk) ? 1u : 0u);
            }
          }
          dn::tc_commit(&v_empty[st]);
          dn::tc_commit(p_empty);
        }
      }
      dn::tc_commit(o_full);
    }
  } else if (warp >= 4) {
    const int qd = warp & 3, cq = (warp - 4) >> 2, r = qd * 32 + lane;      // TMEM lane quarter, quarter of the columns, this thread's row
    const int hr = r / TB, tr = r % TB;
    const bool ok = hr < nh && tr < nq;
    const int pos = p_first + tr, lo = ok ? attn_lo(pos, p.chunk, p.window) : 0, hi_pos = ok ? pos : -1;
    const uint32_t lane_off = (uint32_t)(qd * 32) << 16;
    const float ns = -p.scale * SG_LOG2E;
    const float* tab = p.tab + (size_t)(h0 + (ok ? hr : 0)) * p.D;
    uint32_t hi[16], lw[16];
    // weights of columns 2 k, 2 k + 1 from z = (bias - offset - score) log2(e): 1 / (1 + 2^z); two denominators share a reciprocal
    // (z is capped where 2^-60 stands for zero)
    auto weigh = [&](int k, float za, float zb, bool sa, bool sb) {
      const float a = 1.f + sg_ex2(fminf(za, 60.f)), c = 1.f + sg_ex2(fminf(zb, 60.f)), rc = sg_rcp(a * c);
      const float wa = sa ? rc * c : 0.f, wb = sb ? rc * a : 0.f;
      hi[k] = pack_bf16(wa, wb);
      lw[k] = pack_bf16(wa - __uint_as_float(hi[k] << 16), wb - __uint_as_float(hi[k] & 0xffff0000u));
    };
    for (int j = 0; j < n_tiles; j++) {
      const int st = j & 1, key0 = (page0 + 2 * j) * PAGE + cq * 32, d0 = pos - key0;      // this thread's 32 keys; the first one's distance
      // every key of the quarter is seen by every live row of the warp (rows without a query compute something that is not stored)
      const bool inner = __all_sync(0xffffffffu, !ok || (key0 >= lo && key0 + 31 <= pos));
      float tv[32], v[32];
      if (inner) {
        const float* tp = tab + (ok ? d0 : 31);
#pragma unroll
        for (int i = 0; i < 32; i++) tv[i] = __ldg(tp - i);
      } else {
#pragma unroll
        for (int i = 0; i < 32; i++) tv[i] = __ldg(tab + min(max(d0 - i, 0), p.D - 1));
      }
      dn::mbar_wait(&s_full[st], (j >> 1) & 1, p.err);
      dn::tc_fence_after();
      sg_ld32(tmem + st * 128 + lane_off + cq * 32, v);
      dn::tc_fence_before();
      __syncwarp();
      if (lane == 0) dn::mbar_arrive(&s_empty[st]);
      if (inner) {
#pragma unroll
        for (int i = 0; i < 32; i += 2) weigh(i / 2, fmaf(v[i], ns, tv[i]), fmaf(v[i + 1], ns, tv[i + 1]), true, true);
      } else {
#pragma unroll
        for (int i = 0; i < 32; i += 2) {
          const int ka = key0 + i;
          weigh(i / 2, fmaf(v[i], ns, tv[i]), fmaf(v[i + 1], ns, tv[i + 1]), ka >= lo && ka <= hi_pos, ka + 1 >= lo && ka + 1 <= hi_pos);
        }
      }
      dn::mbar_wait(p_empty, (j & 1) ^ 1u, p.err);      // the product with the previous tile's weights has read them
#pragma unroll
      for (int c = 0; c < 4; c++) {
        *reinterpret_cast<uint4*>(sPh + dn::at_swz(r, cq * 4 + c)) = make_uint4(hi[4 * c], hi[4 * c + 1], hi[4 * c + 2], hi[4 * c + 3]);
        *reinterpret_cast<uint4*>(sPl + dn::at_swz(r, cq * 4 + c)) = make_uint4(lw[4 * c], lw[4 * c + 1], lw[4 * c + 2], lw[4 * c + 3]);
      }
      const int valid = kv_max - (page0 + 2 * j) * PAGE;      // value rows from here on belong to no key: whatever the page holds, it must not enter
      if (valid < 128) {
        dn::mbar_wait(&v_full[st], (j >> 1) & 1, p.err);
        const int per_row = 8 * (DV / 64);
        for (int i = threadIdx.x - 128; i < (128 - valid) * per_row; i += SG_THREADS - 128) {
          const int row = valid + i / per_row, c = i % per_row;
          *reinterpret_cast<uint4*>(sV + st * VB + (c >> 3) * SG_HALF + row * 128 + (c & 7) * 16) = make_uint4(0u, 0u, 0u, 0u);
        }
      }
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
      __syncwarp();
      if (lane == 0) dn::mbar_arrive(p_full);
    }
    dn::mbar_wait(o_full, 0, p.err);
    dn::tc_fence_after();
    const float og = ok && p.gate ? sigmoid_f(p.gate[(size_t)(s0 + tr) * p.H + h0 + hr]) : 1.f;
    bf16* dst = p.out + ((size_t)(s0 + (ok ? tr : 0)) * p.H + h0 + (ok ? hr : 0)) * DV + cq * (DV / 4);
#pragma unroll
    for (int c = 0; c < DV / 64; c++) {
      float v[16];
      dn::tc_ld16(tO + lane_off + cq * (DV / 4) + c * 16, v);
      if (ok) {
#pragma unroll
        for (int x = 0; x < 2; x++) {
          uint4 w;
          w.x = pack_bf16(v[8 * x] * og, v[8 * x + 1] * og); w.y = pack_bf16(v[8 * x + 2] * og, v[8 * x + 3] * og);
          w.z = pack_bf16(v[8 * x + 4] * og, v[8 * x + 5] * og); w.w = pack_bf16(v[8 * x + 6] * og, v[8 * x + 7] * og);
          *reinterpret_cast<uint4*>(dst + c * 16 + 8 * x) = w;
        }
      }
    }
    dn::tc_fence_before();
  }
  __syncthreads();
  if (warp == 2) {
    dn::tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, 512;" ::"r"(tmem) : "memory");
  }
}

}  // namespace dnseq
