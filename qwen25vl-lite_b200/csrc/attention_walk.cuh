// Device code shared by the attention kernels over a window beside kept first tokens (attention_biased.cu,
// attention_differential.cu): which key tiles a piece of work walks, a tile's copy into shared memory, and one tile of
// FlashAttention-style attention (mma.sync m16n8k16, float accumulators).
#pragma once

#include "attention_decode.cuh"

// sigmoid of two neighbouring gate channels (an even channel offset: one 32-bit load).
__device__ __forceinline__ float2 gate_pair(const bf16* g) {
  const float2 z = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(g));
  return make_float2(1.0f / (1.0f + __expf(-z.x)), 1.0f / (1.0f + __expf(-z.y)));
}
__device__ __forceinline__ float gate_one(const bf16* g) { return 1.0f / (1.0f + __expf(-__bfloat162float(*g))); }

// The tiles of keys that queries at positions p_first .. p_last walk.
struct KeyWalk {
  int kept, lo, hi, sink_tiles, win_key0, n_tiles;
  __device__ __forceinline__ void set(int p_first, int p_last, int window, int keep_first, int bn) {
    lo = window > 0 ? max(0, p_first - window + 1) : 0;
    if (lo <= keep_first) lo = 0;
    kept = lo > 0 ? keep_first : 0;
    hi = p_last;
    sink_tiles = (kept + bn - 1) / bn;
    win_key0 = lo / bn * bn;
    n_tiles = sink_tiles + (hi - win_key0) / bn + 1;
  }
  // first key of tile i, and the range of keys [rl, rh] that count in it
  __device__ __forceinline__ void tile(int i, int bn, int& key0, int& rl, int& rh) const {
    if (i < sink_tiles) { key0 = i * bn; rl = 0; rh = kept - 1; }
    else { key0 = win_key0 + (i - sink_tiles) * bn; rl = lo; rh = hi; }
  }
};

// Copies keys [key0, key0 + BN) of one kv head into K and V tiles (zeros past `last`), by NT threads:
// NT / BN threads share a key, so a thread looks one page up and takes that row's 16-byte chunks
// (of the key and of the value) in turn.
// a: anything with the pages, nkv, page_size and v_row of BiasedArgs.
template <int DK, int DV, int BN, int NT, typename Args>
__device__ __forceinline__ void biased_load_tile(unsigned char* ks, unsigned char* vs, const Args& a, const int* table, int kvh,
                                                 int key0, int last, int tid) {
  constexpr int CK = DK / 8, CV = DV / 8, TPK = NT / BN;
  static_assert(NT % BN == 0 && CK % TPK == 0 && CV % TPK == 0, "the chunks of a row divide among its threads");
  const int key = tid / TPK, part = tid % TPK;
  const int kidx = key0 + key;
  const bool valid = kidx <= last;
  const int kc = valid ? kidx : last;                       // a readable address also for the zero-filled rows
  const int page = table[kc / a.page_size];
  const size_t row = ((size_t)page * a.nkv + kvh) * a.page_size + kc % a.page_size;
  const bf16* kr = a.kpages + row * DK;
  const bf16* vr = a.vpages + row * a.v_row;
#pragma unroll
  for (int i = 0; i < CK / TPK; ++i) {
    const int ch = part + i * TPK;
    cp_async16(ks + key * Tile<DK>::PITCH + ch * 16, kr + ch * 8, valid);
  }
#pragma unroll
  for (int i = 0; i < CV / TPK; ++i) {
    const int ch = part + i * TPK;
    cp_async16(vs + key * Tile<DV>::PITCH + ch * 16, vr + ch * 8, valid);
  }
}

// One tile of keys for the warp's 16 rows.  p0/p1: positions of rows g and g+8 (-1: no such row);
// b1x/b2x: the bias numbers of the rows' heads; [rl, rh]: the keys of the tile that count.  FULL: the
// caller has seen that every key of the tile counts for every row of the warp, so nothing is masked.
// TABLE: the rows' heads add tab0 / tab1 [min(distance, dist_rows - 1) * nq] to their scores (a build of
// its own, so that the kernels without a table carry none of it).  PLAIN: a build whose scores are scaled and nothing
// else (no bias, no squashing).  KROW: channels of a key row in shared memory, when the keys at ks are part of wider rows.
template <int DK, int DV, int BN, bool FULL, bool TABLE, bool PLAIN = false, int KROW = DK>
__device__ __forceinline__ void biased_tile(const unsigned (&qf)[DK / 16][4], const unsigned char* ks, const unsigned char* vs,
                                            int key0, int rl, int rh, int p0, int p1, int window, int keep_first, float scale_log2,
                                            float cap_log2, float scale_over_cap, float b10, float b20, float b11, float b21,
                                            const float* __restrict__ tab0, const float* __restrict__ tab1, int dist_rows, int nq,
                                            float (&m)[2], float (&l)[2], float (&o)[DV / 8][4]) {
  constexpr int PK = Tile<KROW>::PITCH, PV = Tile<DV>::PITCH;
  const int lane = threadIdx.x & 31, t = lane & 3;
  float s[BN / 8][4];
#pragma unroll
  for (int j = 0; j < BN / 8; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.f;
#pragma unroll
  for (int kk = 0; kk < DK / 16; ++kk) {
    unsigned b[BN / 8][2];
#pragma unroll
    for (int j = 0; j < BN / 8; ++j) ldmatrix_x2(b[j], ks + (j * 8 + (lane & 7)) * PK + (kk * 16 + 8 * ((lane >> 3) & 1)) * 2);
#pragma unroll
    for (int j = 0; j < BN / 8; ++j) mma_bf16(s[j], qf[kk], b[j][0], b[j][1]);
  }
  // distance of the row's query to the thread's first key of the tile, as a float; the other keys
  // of the thread lie constants further on
  const float d0 = (float)(p0 - key0 - 2 * t), d1 = (float)(p1 - key0 - 2 * t);
  // the distance table: a row whose nearest key of the tile lies at the table's last row or beyond adds one number
  // to all its scores; the table's entries are natural-log scores, the kernel's live in the base-2 domain
  constexpr float LOG2E = 1.4426950408889634f;
  const int last_row = dist_rows - 1;
  const bool far0 = TABLE && p0 - (key0 + BN - 1) >= last_row, far1 = TABLE && p1 - (key0 + BN - 1) >= last_row;
  const float fb0 = far0 ? tab0[(size_t)last_row * nq] * LOG2E : 0.f, fb1 = far1 ? tab1[(size_t)last_row * nq] * LOG2E : 0.f;
  float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
  for (int j = 0; j < BN / 8; ++j) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float fd = (e < 2 ? d0 : d1) - (float)(j * 8 + (e & 1));
      const float b1 = e < 2 ? b10 : b11, b2 = e < 2 ? b20 : b21;
      float v = PLAIN ? s[j][e] * scale_log2
                : cap_log2 > 0.f ? cap_log2 * tanhf(s[j][e] * scale_over_cap) - b1 * __log2f(fmaf(b2, fd, 1.0f))
                                 : fmaf(s[j][e], scale_log2, -b1 * __log2f(fmaf(b2, fd, 1.0f)));
      if (TABLE) {
        if (e < 2 ? far0 : far1) {
          v += e < 2 ? fb0 : fb1;
        } else {
          const int dist = (e < 2 ? p0 : p1) - (key0 + j * 8 + 2 * t + (e & 1));
          v = fmaf((e < 2 ? tab0 : tab1)[(size_t)min(max(dist, 0), last_row) * nq], LOG2E, v);
        }
      }
      if (!FULL) {
        const int kidx = key0 + j * 8 + 2 * t + (e & 1);
        const int dist = (e < 2 ? p0 : p1) - kidx;
        const bool ok = kidx >= rl && kidx <= rh && dist >= 0 && (window <= 0 || dist < window || kidx < keep_first);
        v = ok ? v : -INFINITY;
      }
      s[j][e] = v;
    }
    mx0 = fmaxf(mx0, fmaxf(s[j][0], s[j][1]));
    mx1 = fmaxf(mx1, fmaxf(s[j][2], s[j][3]));
  }
  mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
  mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
  mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
  mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
  const float mn0 = fmaxf(m[0], mx0), mn1 = fmaxf(m[1], mx1);
  const float ms0 = mn0 == -INFINITY ? 0.f : mn0, ms1 = mn1 == -INFINITY ? 0.f : mn1;  // nothing seen yet
  const float c0 = exp2f(m[0] - ms0), c1 = exp2f(m[1] - ms1);
  m[0] = mn0;
  m[1] = mn1;
  float sum0 = 0.f, sum1 = 0.f;
#pragma unroll
  for (int j = 0; j < BN / 8; ++j) {
    s[j][0] = exp2f(s[j][0] - ms0);
    s[j][1] = exp2f(s[j][1] - ms0);
    s[j][2] = exp2f(s[j][2] - ms1);
    s[j][3] = exp2f(s[j][3] - ms1);
    sum0 += s[j][0] + s[j][1];
    sum1 += s[j][2] + s[j][3];
  }
  l[0] = l[0] * c0 + sum0;  // per-thread partial sums; the quad is reduced once at the end
  l[1] = l[1] * c1 + sum1;
#pragma unroll
  for (int nb = 0; nb < DV / 8; ++nb) {
    o[nb][0] *= c0;
    o[nb][1] *= c0;
    o[nb][2] *= c1;
    o[nb][3] *= c1;
  }
#pragma unroll
  for (int kk = 0; kk < BN / 16; ++kk) {
    unsigned pa[4];
    pa[0] = pack_bf16(s[2 * kk][0], s[2 * kk][1]);
    pa[1] = pack_bf16(s[2 * kk][2], s[2 * kk][3]);
    pa[2] = pack_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1]);
    pa[3] = pack_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3]);
    const unsigned char* vrow = vs + (kk * 16 + (lane & 7) + 8 * ((lane >> 3) & 1)) * PV;
#pragma unroll
    for (int np = 0; np < DV / 16; ++np) {
      unsigned b[4];
      ldmatrix_x4_trans(b, vrow + (np * 16 + 8 * (lane >> 4)) * 2);
      mma_bf16(o[2 * np], pa, b[0], b[1]);
      mma_bf16(o[2 * np + 1], pa, b[2], b[3]);
    }
  }
}

// Whether every key of the tile [key0, key0 + bn) counts for every query of positions p_min .. p_max.
__device__ __forceinline__ bool tile_is_full(int key0, int bn, int rl, int rh, int p_min, int p_max, int window, int keep_first) {
  const int last = key0 + bn - 1;
  return p_min >= 0 && last <= p_min && key0 >= rl && last <= rh && (window <= 0 || p_max - key0 < window || last < keep_first);
}
