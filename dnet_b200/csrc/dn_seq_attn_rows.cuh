// dn_seq_attn_rows.cuh -- attention of a step with few rows (decode steps and small portions), libdnet_b200_seq.so.
//
// What k_attn computes, arranged for latency: a block takes one token, up to HB (1, 2 or 4) query heads of one key / value head
// and every nz-th run of 128 keys; each of its four warps stages a tile of 32 keys *and* their values in shared memory by
// asynchronous copies -- one trip to memory after the block table, whole rows, read once for all the block's heads -- and
// works from there: a lane scores one key, then owns ceil(dv / 32) adjacent output dims.  The warps' partials join in warp
// order; rows with several splits leave theirs in scratch, and the last block of a row to finish (an atomic count, nobody
// waits) joins them in split order.  A row's split, tiles and order of sums depend on its own position only.
// MAPS = 2 (differential attention): heads 2 i and 2 i + 1 are one pair of maps, key heads 2 g and 2 g + 1 lie side by side in a key
// row and share value head g; a block stages both maps' keys as one row, and the join subtracts the maps and norms the head.
// Head sizes up to 128 (a pair's keys count as one row) whose rows start on 16-byte boundaries; no pooled blocks (k_attn does those).
#pragma once
#include "dn_seq_kernels.cuh"

namespace dnseq {

constexpr int AR_WARPS = 4, AR_KEYS = AR_WARPS * 32;
__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d), "l"(src) : "memory");
}
// bytes of one tile (32 keys and values): key rows are padded by 16 bytes, so that the lanes' 16-byte reads of one column
// of 32 rows fall into different banks
__host__ __device__ __forceinline__ size_t ar_tile_bytes(int dk, int dv, int esz, bool vk) { return (size_t)32 * (dk * esz + 16) + (vk ? 0 : (size_t)32 * dv * esz); }
// (dk: the whole staged key row; HB heads of `maps` rows of partials each)
__host__ __device__ __forceinline__ size_t ar_smem_bytes(int dk, int dv, int esz, bool vk, int stages, int HB, int maps) {
  const size_t part = (size_t)AR_WARPS * HB * maps * (2 + (dv + 31) / 32 * 32) * 4;
  return (size_t)HB * dk * 4 + ((part + 15) & ~(size_t)15) + (size_t)AR_WARPS * stages * ar_tile_bytes(dk, dv, esz, vk);
}
__device__ __forceinline__ int ar_splits(int keys, int zmax) { return min(zmax, max(1, (keys + AR_KEYS - 1) / AR_KEYS)); }

// (a head's result does not depend on HB: small grids take fewer heads a block)
template <class T, bool SIG, int HB, int MAPS>
__global__ void __launch_bounds__(AR_WARPS * 32) k_attn_rows(Batch b, const T* __restrict__ q, const T* __restrict__ kpool, const T* __restrict__ vpool, int H,
                                                             int G, int dk, int dv, int chunk, float scale, int stages, AttnExtra ex, T* __restrict__ out,
                                                             float* __restrict__ part_g, unsigned int* __restrict__ count) {
  extern __shared__ __align__(16) unsigned char smb[];
  __shared__ uint32_t rows_s[AR_WARPS][32];
  __shared__ bool last_s;
  __shared__ float fz[HB * MAPS][AT_MAX_SPLITS];
  constexpr int V = Vec16<T>::n, ESZ = (int)sizeof(T), NV = HB * MAPS;      // NV: score rows of the block (head i, map m: i MAPS + m)
  H /= MAPS; G /= MAPS;                                      // heads and key heads with all their maps
  const int dk1 = dk;
  dk *= MAPS;                                                // numbers of a staged key row, and of a head's query
  const int VPL = (dv + 31) / 32, dvp = VPL * 32, PL = 2 + dvp;
  float* qs = reinterpret_cast<float*>(smb);                       // [HB][dk]
  float* part = qs + HB * dk;                                // [AR_WARPS][NV][2 + dvp]
  unsigned char* tiles = smb + (size_t)HB * dk * 4 + (((size_t)AR_WARPS * NV * PL * 4 + 15) & ~(size_t)15);
  const int n = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int R = H / G, per = (R + HB - 1) / HB;        // heads of a key head; blocks they take
  const int g = blockIdx.y / per, h0 = g * R + (blockIdx.y % per) * HB, nh = min(HB, (g + 1) * R - h0);
  const int slot = b.slot[n], p = b.pos[n];
  const int lo = attn_lo(p, chunk, ex.window), kept = attn_kept(lo, ex), nkeys = kept + p - lo + 1;
  const int zmax = gridDim.z, nz = ar_splits(nkeys, zmax), z = blockIdx.z;
  if (z >= nz) return;
  const bool vk = vpool == kpool;
  const int Ck = G * dk, Cv = ex.v_ld > 0 ? ex.v_ld : G * dv;
  const int ldk = dk * ESZ + 16, ldv_ = vk ? ldk : dv * ESZ;       // row strides of a tile in bytes
  const size_t tile_b = ar_tile_bytes(dk, dv, ESZ, vk);
  unsigned char* mine = tiles + (size_t)warp * stages * tile_b;
  const int32_t* bt = b.bt + (size_t)slot * b.max_pages;
  const int step = nz * AR_KEYS, first = (z * AR_WARPS + warp) * 32;
  // a lane's walk over the 16-byte pieces of a tile's rows: first row and piece, and what 32 pieces further means
  const int ck = dk * ESZ / 16, cv = dv * ESZ / 16;
  const int kr0 = lane / ck, kc0 = lane - kr0 * ck, kdr = 32 / ck, kdc = 32 - kdr * ck;
  const int vr0 = lane / cv, vc0 = lane - vr0 * cv, vdr = 32 / cv, vdc = 32 - vdr * cv;
  auto stage = [&](int s, int j0) {      // this warp's tile at key j0 into buffer s
    unsigned char* kt = mine + (size_t)s * tile_b;
    unsigned char* vt = vk ? kt : kt + (size_t)32 * ldk;
    const int cnt = min(32, nkeys - j0);
    if (lane < cnt) {
      const int v = j0 + lane, j = v < kept ? v : lo + v - kept;      // kept first tokens, then the tokens lo .. p
      rows_s[warp][lane] = (uint32_t)bt[j / PAGE] * PAGE + (uint32_t)(j % PAGE);
    }
    __syncwarp();
    for (int r = kr0, c = kc0; r < cnt;) {
      cp_async16(kt + r * ldk + c * 16, kpool + (size_t)rows_s[warp][r] * Ck + g * dk + c * V);
      r += kdr; c += kdc;
      if (c >= ck) { c -= ck; r++; }
    }
    if (!vk)
      for (int r = vr0, c = vc0; r < cnt;) {
        cp_async16(vt + r * ldv_ + c * 16, vpool + (size_t)rows_s[warp][r] * Cv + g * dv + c * V);
        r += vdr; c += vdc;
        if (c >= cv) { c -= cv; r++; }
      }
    cp_async_commit();
    __syncwarp();
  };
  if (first < nkeys) stage(0, first);
  for (int e = threadIdx.x; e < HB * dk; e += blockDim.x) qs[e] = e < nh * dk ? ldf(q + ((size_t)n * H + h0) * dk + e) : 0.f;
  float r1[HB], r2[HB], soff[HB];
#pragma unroll
  for (int i = 0; i < HB; i++) {
    const int h = h0 + min(i, nh - 1);
    r1[i] = ex.r1 ? ldf((const T*)ex.r1 + h) : 0.f;
    r2[i] = ex.r1 ? ldf((const T*)ex.r2 + h) : 0.f;
    soff[i] = SIG ? ldf((const T*)ex.off + h) : 0.f;
  }
  __syncthreads();
  float m[NV], l[NV], acc[NV][4];
#pragma unroll
  for (int i = 0; i < NV; i++) {
    m[i] = -INFINITY; l[i] = 0.f;
#pragma unroll
    for (int x = 0; x < 4; x++) acc[i][x] = 0.f;
  }
  const int vcnt = min(VPL, max(0, dv - lane * VPL));
  int s = 0;
  for (int j0 = first; j0 < nkeys; j0 += step) {
    const bool more = j0 + step < nkeys;
    if (more && stages > 1) { stage(s ^ 1, j0 + step); cp_async_wait<1>(); }
    else cp_async_wait<0>();
    __syncwarp();
    const unsigned char* kt = mine + (size_t)s * tile_b;
    const unsigned char* vt = vk ? kt : kt + (size_t)32 * ldk;
    const int cnt = min(32, nkeys - j0), j = j0 + lane;
    float sc[NV];
#pragma unroll
    for (int i = 0; i < NV; i++) sc[i] = 0.f;
    if (lane < cnt) {
      const T* kr = reinterpret_cast<const T*>(kt + (size_t)lane * ldk);
#pragma unroll
      for (int mp = 0; mp < MAPS; mp++) {
#pragma unroll 4
        for (int d1 = 0; d1 < dk1; d1 += V) {
          const int d = mp * dk1 + d1;
          float kv[V];
          ldv(kr + d, kv);
#pragma unroll
          for (int i = 0; i < HB; i++) {
            float& s1 = sc[i * MAPS + mp];
#pragma unroll
            for (int x = 0; x < V; x += 4) {
              const float4 q4 = *reinterpret_cast<const float4*>(qs + i * dk + d + x);
              s1 = fmaf(q4.x, kv[x], s1); s1 = fmaf(q4.y, kv[x + 1], s1);
              s1 = fmaf(q4.z, kv[x + 2], s1); s1 = fmaf(q4.w, kv[x + 3], s1);
            }
          }
        }
      }
    }
    float pw[NV];
#pragma unroll
    for (int i = 0; i < NV; i++) {
      float a = sc[i] * scale;
      if (ex.softcap > 0.f) a = ex.softcap * tanhf(a / ex.softcap);
      if (ex.r1) a -= r1[i / MAPS] * log1pf(r2[i / MAPS] * (float)max(0, j < kept ? p - j : nkeys - 1 - j));
      if (SIG) { pw[i] = lane < cnt ? sigmoid_f(a + soff[i / MAPS]) : 0.f; continue; }
      a = lane < cnt ? a : -INFINITY;
      const float mn = fmaxf(m[i], warp_max(a)), corr = expf(m[i] - mn);
      pw[i] = lane < cnt ? expf(a - mn) : 0.f;
      l[i] = l[i] * corr + warp_sum(pw[i]);
#pragma unroll
      for (int x = 0; x < 4; x++) acc[i][x] *= corr;
      m[i] = mn;
    }
#pragma unroll 4
    for (int t = 0; t < cnt; t++) {
      const T* vr = reinterpret_cast<const T*>(vt + (size_t)t * ldv_) + lane * VPL;
      float v[4] = {0.f, 0.f, 0.f, 0.f};
      if (VPL == 4 && vcnt == 4 && (dv & 3) == 0) ld4(vr, v);
      else {
#pragma unroll
        for (int x = 0; x < 4; x++) if (x < vcnt) v[x] = ldf(vr + x);
      }
#pragma unroll
      for (int i = 0; i < NV; i++) {
        const float pt = __shfl_sync(0xffffffffu, pw[i], t);
#pragma unroll
        for (int x = 0; x < 4; x++) acc[i][x] = fmaf(pt, v[x], acc[i][x]);
      }
    }
    __syncwarp();
    if (stages > 1) s ^= 1;
    else if (more) stage(0, j0 + step);
  }
#pragma unroll
  for (int i = 0; i < NV; i++) {
    float* pr = part + ((size_t)warp * NV + i) * PL;
    if (lane == 0) { pr[0] = m[i]; pr[1] = l[i]; }
#pragma unroll
    for (int x = 0; x < 4; x++) if (x < VPL) pr[2 + lane * VPL + x] = acc[i][x];
  }
  __syncthreads();
  const bool split = nz > 1;
  // row i's (head's) output from the warps' partials at stride `st` floats
  float* os = reinterpret_cast<float*>(tiles);      // MAPS = 2: [NV][dv], the maps' outputs (the tiles have been read out)
  auto finish = [&](int i, int d, const float* pr, size_t st) {
    constexpr int cnt = AR_WARPS;
    if (MAPS == 2) {
      float M = -INFINITY, L = 0.f, a = 0.f;
      for (int w = 0; w < cnt; w++) M = fmaxf(M, pr[w * st]);
      for (int w = 0; w < cnt; w++) {
        const float f = expf(pr[w * st] - M);
        L += pr[w * st + 1] * f;
        a += pr[w * st + 2 + d] * f;
      }
      os[i * dv + d] = a / L;
      return;
    }
    const int h = h0 + i;
    const float og = ex.gate ? sigmoid_f(ex.gate[(size_t)n * H + h]) : 1.f;
    float a = 0.f;
    if (SIG) {
      for (int w = 0; w < cnt; w++) a += pr[w * st + 2 + d];
      stf(out + ((size_t)n * H + h) * dv + d, a * og);
      return;
    }
    const float snk = ex.sink ? ldf((const T*)ex.sink + h) : -INFINITY;
    float M = snk;
    for (int w = 0; w < cnt; w++) M = fmaxf(M, pr[w * st]);
    float L = ex.sink ? expf(snk - M) : 0.f;
    for (int w = 0; w < cnt; w++) {
      const float f = expf(pr[w * st] - M);      // a warp without a tile has maximum -inf and weight 0
      L += pr[w * st + 1] * f;
      a += pr[w * st + 2 + d] * f;
    }
    stf(out + ((size_t)n * H + h) * dv + d, a / L * og);
  };
  // MAPS = 2: a warp a head subtracts the maps, norms and stores
  auto diff_out = [&]() {
    __syncthreads();
    const float lm = *ex.lam;
    for (int i = warp; i < nh; i += AR_WARPS) {
      const float *a1 = os + 2 * i * dv, *a2 = a1 + dv;
      float ss = 0.f;
      for (int d = lane; d < dv; d += 32) { const float o = a1[d] - lm * a2[d]; ss += o * o; }
      const float f = ex.post / sqrtf(warp_sum(ss) / (float)dv + ex.eps);
      for (int d = lane; d < dv; d += 32) stf(out + ((size_t)n * H + h0 + i) * dv + d, (a1[d] - lm * a2[d]) * f);
    }
  };
  const int nrows = nh * MAPS;
  if (!split) {
    for (int e = threadIdx.x; e < nrows * dv; e += blockDim.x) finish(e / dv, e % dv, part + (size_t)(e / dv) * PL, (size_t)NV * PL);
    if (MAPS == 2) diff_out();
    return;
  }
  for (int e = threadIdx.x; e < nrows * dv; e += blockDim.x) {
    const int i = e / dv, d = e % dv;
    const float* pr = part + (size_t)i * PL;
    float* pg = part_g + (((size_t)n * H * MAPS + h0 * MAPS + i) * zmax + z) * PL;
    float M = -INFINITY, L = 0.f, a = 0.f;
    if (!SIG)
      for (int w = 0; w < AR_WARPS; w++) M = fmaxf(M, pr[(size_t)w * NV * PL]);
    for (int w = 0; w < AR_WARPS; w++) {
      const float* pq = pr + (size_t)w * NV * PL;
      const float f = SIG ? 1.f : expf(pq[0] - M);
      if (!SIG) L += pq[1] * f;
      a += pq[2 + d] * f;
    }
    pg[2 + d] = a;
    if (d == 0) { pg[0] = M; pg[1] = L; }
  }
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) last_s = atomicAdd(count + (size_t)n * gridDim.y + blockIdx.y, 1u) == (unsigned)nz - 1;
  __syncthreads();
  if (!last_s) return;
  __threadfence();
  if (threadIdx.x == 0) count[(size_t)n * gridDim.y + blockIdx.y] = 0;      // ready for the next launch
  // a warp a row turns the splits' maxima and sums into one factor a split (a lane each), then every thread adds its numbers over the
  // splits, all loads in flight at once
  const float* rows_g = part_g + ((size_t)n * H + h0) * MAPS * zmax * PL;
  for (int i = warp; i < nrows; i += AR_WARPS) {
    const float* pr = rows_g + (size_t)i * zmax * PL;
    float f = lane < nz ? 1.f : 0.f;
    if (!SIG) {
      const float snk = MAPS == 1 && ex.sink ? ldf((const T*)ex.sink + h0 + i) : -INFINITY;
      const float mz = lane < nz ? __ldcg(pr + (size_t)lane * PL) : -INFINITY, lz = lane < nz ? __ldcg(pr + (size_t)lane * PL + 1) : 0.f;
      const float M = fmaxf(warp_max(mz), snk);
      f = lane < nz ? expf(mz - M) : 0.f;
      f /= warp_sum(lz * f) + (MAPS == 1 && ex.sink ? expf(snk - M) : 0.f);
    }
    if (MAPS == 1 && ex.gate) f *= sigmoid_f(ex.gate[(size_t)n * H + h0 + i]);
    if (lane < AT_MAX_SPLITS) fz[i][lane] = f;
  }
  __syncthreads();
  for (int e = threadIdx.x; e < nrows * dv; e += blockDim.x) {
    const int i = e / dv, d = e - i * dv;
    const float* pr = rows_g + (size_t)i * zmax * PL + 2 + d;
    float v[AT_MAX_SPLITS], a = 0.f;
#pragma unroll
    for (int z1 = 0; z1 < AT_MAX_SPLITS; z1++) v[z1] = z1 < nz ? __ldcg(pr + (size_t)z1 * PL) : 0.f;
#pragma unroll
    for (int z1 = 0; z1 < AT_MAX_SPLITS; z1++) a = fmaf(v[z1], fz[i][z1], a);
    if (MAPS == 2) os[i * dv + d] = a;
    else stf(out + ((size_t)n * H + h0 + i) * dv + d, a);
  }
  if (MAPS == 2) diff_out();
}

}  // namespace dnseq
