// dn_seq_attn_diff.cuh -- differential attention of prompt portions on the 5th-generation tensor cores (tcgen05 + TMEM + TMA),
// libdnet_b200_seq.so, bf16.
//
// A head has two maps -- a query and a key each -- over one value:  o = a1 - lambda a2, then (1 - diff) rms(o).  The two maps are the two
// halves of a software pipeline: while one's softmax weights are formed, the tensor cores run the other's products.  A CTA takes one key /
// value head, up to DA_HEADS of its query heads and TB = floor(128 / heads) consecutive tokens of one entry: the 128 MMA rows are heads x
// tokens.  Per tile of 128 keys (two pages of the row block's list, by TMA through the block table) and map m:
//   S_m = Q_m K_m^T      A = Q_m [128 x DK], B = K_m [128 x DK], both K-major in shared memory       TMEM columns 128 m .. 128 m + 127
//   P_m = weights        four warps a map, a thread a row; P takes the place of S_m in TMEM: of each 32 columns the first 16 hold 32
//                        weights as bf16, the other 16 what bf16 left of them (16 bits of each weight's mantissa)
//   O_m += P_m V         A = P_m out of TMEM, B = V tile [128 x DV], MN-major                          TMEM columns 256 + DV m ..
// A row's weights are 2^(score - reference); the reference is a running maximum that is only moved (and O_m scaled by the row's own thread)
// when a score exceeds it by 8 or more, so that scaling is rare and every sum stays in range.  The value tile is read once for both maps.
// At the end the maps' sums meet in shared memory, the eight warps subtract, norm and store half of the columns each.
// The page list of a row block: the pages of the kept first tokens, then the window's; a page half a row does not see is masked.
// Roles: warp 0 TMA producer, warp 1 MMA issuer, warp 2 TMEM allocator, warps 4-7 map 0, warps 8-11 map 1.
#pragma once
#include "dn_seq_attn_tc.cuh"

namespace dnseq {

constexpr int DA_HEADS = 16, DA_THREADS = 384;
constexpr float DA_SLACK = 8.f;      // how far (log2) a score may exceed the reference before the row is rescaled

struct DiffParams {
  const bf16* q;          // [N][2 H][DK]
  bf16* out;              // [N][H][DV]
  const float* lam;
  int H, G, chunk, window, keep, hpc;      // heads and key heads (pairs of maps count once); hpc: query heads of a CTA
  float scale, post, eps;
  unsigned int* err;
};

// 32 consecutive 32-bit columns of this warp's TMEM quarter; the registers are valid after tm_ready
__device__ __forceinline__ void tm_ld32(uint32_t taddr, uint32_t (&r)[32]) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x32.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31}, [%32];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]), "=r"(r[10]), "=r"(r[11]),
        "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]), "=r"(r[16]), "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]), "=r"(r[21]), "=r"(r[22]),
        "=r"(r[23]), "=r"(r[24]), "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]), "=r"(r[30]), "=r"(r[31])
      : "r"(taddr));
}
__device__ __forceinline__ void tm_wait_ld() { asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory"); }
// no use of r moves above this point
__device__ __forceinline__ void tm_pin(uint32_t (&r)[32]) {
#pragma unroll
  for (int i = 0; i < 32; i += 8)
    asm volatile("" : "+r"(r[i]), "+r"(r[i + 1]), "+r"(r[i + 2]), "+r"(r[i + 3]), "+r"(r[i + 4]), "+r"(r[i + 5]), "+r"(r[i + 6]), "+r"(r[i + 7]));
}
__device__ __forceinline__ void tm_wait_st() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }
// D[tmem] (+)= A[tmem] . B[smem]^T   (kind::f16; A: bf16 pairs, one row a lane)
__device__ __forceinline__ void tc_mma_ts(uint32_t tmem_d, uint32_t tmem_a, uint64_t bdesc, uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}"
      ::"r"(tmem_d), "r"(tmem_a), "l"(bdesc), "r"(idesc), "r"(accumulate)
      : "memory");
}

// pages a row block reads: 0 .. kept - 1, then w0 .. (count in all)
struct DiffPages { int kept, w0, count; };
__device__ __forceinline__ DiffPages diff_pages(int p_first, int p_last, int chunk, int window, int keep) {
  const int lo = attn_lo(p_first, chunk, window);
  DiffPages d;
  d.kept = (min(keep, lo) + PAGE - 1) / PAGE;
  d.w0 = max(lo / PAGE, d.kept);
  d.count = d.kept + max(0, p_last / PAGE - d.w0 + 1);
  return d;
}
__host__ __device__ constexpr int da_kst(int DK) { return DK == 64 ? 2 : 1; }      // stages of the key tile
__host__ __device__ constexpr size_t da_smem(int DK, int DV) { return (size_t)(2 * (1 + da_kst(DK)) * (DK / 64) + 2 * (DV / 64)) * SG_HALF + 1024 + 4096; }

template <int DK, int DV>
__global__ void __launch_bounds__(DA_THREADS, 1) k_diff_attn_tc(const __grid_constant__ CUtensorMap mapK, const __grid_constant__ CUtensorMap mapV, Batch b, DiffParams p) {
  constexpr int KST = da_kst(DK), KB = DK / 64 * SG_HALF, VB = DV / 64 * SG_HALF;      // bytes of one map's key (query) tile and of a value tile
  extern __shared__ __align__(1024) unsigned char da_raw[];
  unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(da_raw) + 1023) & ~(uintptr_t)1023);
  unsigned char *sQ = smem, *sK = sQ + 2 * KB, *sV = sK + KST * 2 * KB;
  float* xch = reinterpret_cast<float*>(sV + 2 * VB);      // [2][128] reciprocal sums of the maps, [2][128] partial sums of squares
  uint64_t* bars = reinterpret_cast<uint64_t*>(xch + 512);
  uint64_t *k_full = bars, *k_empty = bars + 2, *v_full = bars + 4, *v_empty = bars + 6, *s_full = bars + 8, *p_full = bars + 10, *o_full = bars + 12;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 13);
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
  const int p_first = b.ent_pos0[e] + t * TB, p_last = p_first + nq - 1;
  const int32_t* bt = b.bt + (size_t)b.ent_slot[e] * b.max_pages;
  const DiffPages pg = diff_pages(p_first, p_last, p.chunk, p.window, p.keep);
  const int n_tiles = (pg.count + 1) / 2;
  auto page_at = [&](int i) { return i < pg.kept ? i : pg.w0 + i - pg.kept; };      // the sequence's page at place i of the list

  if (threadIdx.x == 0) {
    for (int i = 0; i < 2; i++) {
      dn::mbar_init(&k_full[i], 1); dn::mbar_init(&k_empty[i], 1); dn::mbar_init(&v_full[i], 1); dn::mbar_init(&v_empty[i], 1);
      dn::mbar_init(&s_full[i], 1); dn::mbar_init(&p_full[i], 4);
    }
    dn::mbar_init(o_full, 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 2) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], 512;" ::"r"(dn::smem_u32(tmem_slot)) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  // Q rows (head, token) of both maps, zero where there is none, in the layout TMA's 128-byte swizzle gives
  for (int i = threadIdx.x; i < 2 * 128 * (DK / 8); i += DA_THREADS) {
    const int m = i / (128 * (DK / 8)), x = i % (128 * (DK / 8)), r = x / (DK / 8), c = x % (DK / 8), hr = r / TB, tr = r % TB;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (hr < nh && tr < nq) v = *reinterpret_cast<const uint4*>(p.q + (((size_t)(s0 + tr) * p.H + h0 + hr) * 2 + m) * DK + c * 8);
    *reinterpret_cast<uint4*>(sQ + m * KB + dn::at_swz(r, c)) = v;
  }
  asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  dn::tc_fence_before();
  __syncthreads();
  dn::tc_fence_after();
  const uint32_t tmem = *tmem_slot, tO = tmem + 256;

  if (warp == 0) {
    if (lane == 0) {
      for (int j = 0; j < n_tiles; j++) {
        // the second half of the last tile may have no page: any page, masked
        const int pg0 = bt[page_at(2 * j)] * PAGE, pg1 = 2 * j + 1 < pg.count ? bt[page_at(2 * j + 1)] * PAGE : pg0;
        const int ks = j % KST, vs = j & 1;
        unsigned char* dk = sK + ks * 2 * KB;
        dn::mbar_wait(&k_empty[ks], ((j / KST) & 1) ^ 1u, p.err);
        dn::mbar_arrive_expect_tx(&k_full[ks], 2 * KB);
#pragma unroll
        for (int hf = 0; hf < 2 * DK / 64; hf++) {      // both maps' columns lie side by side in a key row
          dn::tma_load_2d(dk + hf * SG_HALF, &mapK, g * 2 * DK + hf * 64, pg0, &k_full[ks]);
          dn::tma_load_2d(dk + hf * SG_HALF + SG_HALF / 2, &mapK, g * 2 * DK + hf * 64, pg1, &k_full[ks]);
        }
        unsigned char* dv = sV + vs * VB;
        dn::mbar_wait(&v_empty[vs], ((j >> 1) & 1) ^ 1u, p.err);
        dn::mbar_arrive_expect_tx(&v_full[vs], VB);
#pragma unroll
        for (int hf = 0; hf < DV / 64; hf++) {
          dn::tma_load_2d(dv + hf * SG_HALF, &mapV, g * DV + hf * 64, pg0, &v_full[vs]);
          dn::tma_load_2d(dv + hf * SG_HALF + SG_HALF / 2, &mapV, g * DV + hf * 64, pg1, &v_full[vs]);
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t idesc_s = dn::tc_instr_desc(128, 128), idesc_o = dn::tc_instr_desc(128, DV) | (1u << 16);      // V is MN-major
      auto scores = [&](int j, int m) {
        const int ks = j % KST;
        if (m == 0) dn::mbar_wait(&k_full[ks], (j / KST) & 1, p.err);
        dn::tc_fence_after();
#pragma unroll
        for (int hf = 0; hf < DK / 64; hf++) {
          const uint64_t ad = dn::tc_smem_desc(sQ + m * KB + hf * SG_HALF), bd = dn::tc_smem_desc(sK + (ks * 2 + m) * KB + hf * SG_HALF);
#pragma unroll
          for (int k = 0; k < 4; k++) dn::tc_mma(tmem + m * 128, ad + (uint64_t)(2 * k), bd + (uint64_t)(2 * k), idesc_s, (hf | k) ? 1u : 0u);
        }
        dn::tc_commit(&s_full[m]);
        if (m == 1) dn::tc_commit(&k_empty[ks]);
      };
      scores(0, 0);
      scores(0, 1);
      for (int j = 0; j < n_tiles; j++) {
        const int vs = j & 1;
        dn::mbar_wait(&v_full[vs], (j >> 1) & 1, p.err);
        const uint64_t vd = dn::tc_smem_desc_mn(sV + vs * VB, SG_HALF, 1024);
#pragma unroll
        for (int m = 0; m < 2; m++) {
          dn::mbar_wait(&p_full[m], j & 1, p.err);
          dn::tc_fence_after();
#pragma unroll
          for (int kk = 0; kk < 8; kk++) {
#pragma unroll
            for (int part = 0; part < 2; part++)
              tc_mma_ts(tO + m * DV, tmem + m * 128 + 32 * (kk >> 1) + 8 * (kk & 1) + 16 * part, vd + (uint64_t)(kk * (2048 >> 4)), idesc_o, (j | kk | part) ? 1u : 0u);
          }
          if (m == 1) dn::tc_commit(&v_empty[vs]);
          if (j + 1 < n_tiles) scores(j + 1, m);      // into the columns that P_m has just been read from: products run in order
        }
      }
      dn::tc_commit(o_full);
    }
  } else if (warp >= 4) {
    const int m = (warp - 4) >> 2, qd = warp & 3, r = qd * 32 + lane;      // map, TMEM lane quarter, this thread's row
    const int hr = r / TB, tr = r % TB;
    const bool ok = hr < nh && tr < nq;
    const int pos = p_first + tr, lo = ok ? attn_lo(pos, p.chunk, p.window) : 0, hi_pos = ok ? pos : -1;
    const uint32_t lane_off = (uint32_t)(qd * 32) << 16, tS = tmem + m * 128 + lane_off, tOm = tO + m * DV + lane_off;
    const float sc2 = p.scale * SG_LOG2E;
    float ref = -INFINITY, l = 0.f;      // ref: scaled, log2
    for (int j = 0; j < n_tiles; j++) {
      const int kb0 = page_at(2 * j) * PAGE, kb1 = 2 * j + 1 < pg.count ? page_at(2 * j + 1) * PAGE : 0x7fffffff - PAGE;      // first positions of the halves
      uint32_t v[4][32];
      dn::mbar_wait(&s_full[m], j & 1, p.err);
      __syncwarp();
      dn::tc_fence_after();
#pragma unroll
      for (int c = 0; c < 4; c++) tm_ld32(tS + c * 32, v[c]);
      tm_wait_ld();
#pragma unroll
      for (int c = 0; c < 4; c++) tm_pin(v[c]);
      float mx = -INFINITY;
#pragma unroll
      for (int hf = 0; hf < 2; hf++) {
        const int kb = hf ? kb1 : kb0;
        // every key of the half is seen by every live row of the warp (rows without a query compute something that is not stored)
        const bool inner = __all_sync(0xffffffffu, !ok || (kb + PAGE - 1 <= pos && (kb >= lo || kb + PAGE - 1 < p.keep)));
        if (!inner) {
#pragma unroll
          for (int c = 0; c < 2; c++)
#pragma unroll
            for (int i = 0; i < 32; i++) {
              const int key = kb + c * 32 + i;
              if (!(key <= hi_pos && (key >= lo || key < p.keep))) v[2 * hf + c][i] = 0xff800000u;      // -inf
            }
        }
#pragma unroll
        for (int c = 0; c < 2; c++)
#pragma unroll
          for (int i = 0; i < 32; i++) mx = fmaxf(mx, __uint_as_float(v[2 * hf + c][i]));
      }
      mx *= sc2;      // (the scale is positive)
      const bool move = mx > ref + DA_SLACK || (ref == -INFINITY && mx > -INFINITY);
      if (__any_sync(0xffffffffu, move)) {
        const float f = move ? sg_ex2(ref - mx) : 1.f;      // 0 for a row that has seen nothing yet
        if (move) { ref = mx; l *= f; }
        if (j > 0) {      // (the tile before's product with V is complete: the scores were issued behind it)
#pragma unroll 1
          for (int c = 0; c < DV / 32; c++) {
            uint32_t o[32];
            tm_ld32(tOm + c * 32, o);
            tm_wait_ld();
            tm_pin(o);
#pragma unroll
            for (int i = 0; i < 32; i++) o[i] = __float_as_uint(__uint_as_float(o[i]) * f);
            dn::tmem_st32(tOm + c * 32, o);
          }
        }
      }
      const float nref = ref == -INFINITY ? 0.f : -ref;
      float l0 = 0.f, l1 = 0.f;
#pragma unroll
      for (int c = 0; c < 4; c++) {
        uint32_t w[32];
#pragma unroll
        for (int i = 0; i < 16; i++) {
          const float a = sg_ex2(fmaf(__uint_as_float(v[c][2 * i]), sc2, nref)), d = sg_ex2(fmaf(__uint_as_float(v[c][2 * i + 1]), sc2, nref));
          l0 += a; l1 += d;
          w[i] = pack_bf16(a, d);
          w[16 + i] = pack_bf16(a - __uint_as_float(w[i] << 16), d - __uint_as_float(w[i] & 0xffff0000u));
        }
        dn::tmem_st32(tS + c * 32, w);
      }
      l += l0 + l1;
      if (m == 0 && j == n_tiles - 1) {      // value rows that belong to no key: whatever the page holds, it must not enter
        const int n0 = min(PAGE, p_last - kb0 + 1), n1 = kb1 <= p_last ? min(PAGE, p_last - kb1 + 1) : 0;
        if (n0 + n1 < 2 * PAGE) {
          dn::mbar_wait(&v_full[j & 1], (j >> 1) & 1, p.err);
          constexpr int per_row = 8 * (DV / 64);
          for (int i = threadIdx.x - 128; i < 128 * per_row; i += 128) {
            const int row = i / per_row, c = i % per_row;
            if ((row & 63) >= (row < 64 ? n0 : n1))
              *reinterpret_cast<uint4*>(sV + (j & 1) * VB + (c >> 3) * SG_HALF + row * 128 + (c & 7) * 16) = make_uint4(0u, 0u, 0u, 0u);
          }
          asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
        }
      }
      tm_wait_st();
      dn::tc_fence_before();
      __syncwarp();
      if (lane == 0) dn::mbar_arrive(&p_full[m]);
    }
    xch[m * 128 + r] = 1.f / l;
    dn::mbar_wait(o_full, 0, p.err);
    __syncwarp();
    dn::tc_fence_after();
    asm volatile("bar.sync 1, 256;" ::: "memory");
    // the thread's row, half of its columns: o = a1 - lambda a2
    const float i0 = xch[r], i1 = *p.lam * xch[128 + r];
    constexpr int HC = DV / 2;
    uint32_t o[HC / 32][32];
    float ss = 0.f;
#pragma unroll
    for (int c = 0; c < HC / 32; c++) {
      uint32_t a2[32];
      tm_ld32(tO + lane_off + m * HC + c * 32, o[c]);
      tm_ld32(tO + lane_off + DV + m * HC + c * 32, a2);
      tm_wait_ld();
      tm_pin(o[c]);
      tm_pin(a2);
#pragma unroll
      for (int i = 0; i < 32; i++) {
        const float x = __uint_as_float(o[c][i]) * i0 - __uint_as_float(a2[i]) * i1;
        o[c][i] = __float_as_uint(x);
        ss += x * x;
      }
    }
    xch[256 + m * 128 + r] = ss;
    asm volatile("bar.sync 1, 256;" ::: "memory");
    const float f = p.post / sqrtf((xch[256 + r] + xch[384 + r]) / (float)DV + p.eps);
    if (ok) {
      bf16* dst = p.out + ((size_t)(s0 + tr) * p.H + h0 + hr) * DV + m * HC;
#pragma unroll
      for (int c = 0; c < HC / 8; c++) {
        const uint32_t* x = &o[c / 4][(c % 4) * 8];
        uint4 w;
        w.x = pack_bf16(__uint_as_float(x[0]) * f, __uint_as_float(x[1]) * f); w.y = pack_bf16(__uint_as_float(x[2]) * f, __uint_as_float(x[3]) * f);
        w.z = pack_bf16(__uint_as_float(x[4]) * f, __uint_as_float(x[5]) * f); w.w = pack_bf16(__uint_as_float(x[6]) * f, __uint_as_float(x[7]) * f);
        *reinterpret_cast<uint4*>(dst + c * 8) = w;
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
