// Differential attention over the paged cache: every head has two maps, each a softmax attention of its own over the
// same values, and the second map's result is subtracted from the first's.
//
//   a_m(i) = softmax_j((q_m,i . k_m,j) * scale) v_j  for m = 1, 2, over j <= i and i - j < window (window 0: all j <= i)
//   o_i    = a_1(i) - lam * a_2(i);   o_i <- o_i / sqrt(mean(o_i^2) + eps) * gain * sigmoid(gate_i)   per head
//
// A token's row holds its queries ordered by (kv head, map, head of the group), D channels each.  A key row of the cache
// holds the kv head's keys of both maps side by side, 2 * D channels, over one value row of Dv channels.  Scores, softmax
// state, both maps' results, the difference, its norm and the gate are float; the maps' weights are rounded to bfloat16
// for the tensor cores' product with the values, nothing else is before the result.
//
// The general kernel (float or bfloat16, keys of any size, values of up to 512 channels): a warp per (token, head) walks
// the keys once for both maps, in tiles of 32 aligned to the absolute key index.
//
// The bfloat16 tensor-core kernels (mma.sync m16n8k16), for the sizes listed below:
//   * runs: a CTA of 4 warps takes 32 (token, head of the group) pairs of one entry and kv head; warps 0 and 1 hold the
//     pairs' first map, warps 2 and 3 the second, all share the key and value tiles (64 keys, two stages of cp.async);
//     at the end the second map's rows go through shared memory to the first map's warps, which finish the heads;
//   * single tokens: the 4 warps hold the token's heads on both maps (up to 16 rows: the key row is read whole, a map's
//     query has zeros where the other map's channels are), take 32-key tiles in turn and merge through shared memory;
//     with more than one key range per token the ranges leave (max, sum, unnormalised output) in scratch memory and a
//     second kernel adds them up in order.
#include "attention_walk.cuh"

#define DIFF_WARPS 4
#define DIFF_MAX_D 512

struct DiffArgs {
  const void* q;            // [N, q_stride]
  int q_stride;
  const void* gate;         // [N, gate_stride], heads * Dv channels
  int gate_stride;
  void* out;                // [N, heads * Dv]
  const bf16* kpages;       // [pages, nkv, page_size, 2 * D]
  const bf16* vpages;       // [pages, nkv, page_size, Dv]
  const int* block_table;
  int table_width;
  const int* cu_q;
  const int* q_start_pos;
  const int* items;         // runs: (entry, row tile) pairs; single tokens: entry indices
  int heads, nkv, page_size, window;
  int v_row;
  float scale_log2, lam, gain, eps;
  int n_splits;
  float* part_o;            // [items, 2 * heads, splits, Dv]
  float* part_ml;           // [items, 2 * heads, splits, 2]
};

template <typename T>
__global__ void diff_attention_generic_kernel(DiffArgs a, const T* __restrict__ kpages, const T* __restrict__ vpages, const int* __restrict__ token_seq,
                                              int n_tokens, int dk, int dv, float scale) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ __align__(16) unsigned char diff_smem[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const size_t per_warp = (size_t)(2 * dk + 64) * sizeof(float) + 32 * sizeof(size_t);
  unsigned char* base = diff_smem + warp * per_warp;
  size_t* voff = reinterpret_cast<size_t*>(base);
  float* qs = reinterpret_cast<float*>(base + 32 * sizeof(size_t));          // both maps' queries
  float* ps = qs + 2 * dk;                                                    // both maps' weights of a tile
  const long long item = (long long)blockIdx.x * DIFF_WARPS + warp;
  if (item >= (long long)n_tokens * a.heads) return;
  const int token = (int)(item / a.heads), head = (int)(item % a.heads);
  const int group = a.heads / a.nkv, kvh = head / group, in_group = head % group;
  const int seq = token_seq[token];
  if (seq < 0) return;
  const int p = a.q_start_pos[seq] + token - a.cu_q[seq];
  const int lo = a.window > 0 ? max(0, p - a.window + 1) : 0;
  const T* q = (const T*)a.q + (size_t)token * a.q_stride;
  for (int m = 0; m < 2; ++m)
    for (int c = lane; c < dk; c += 32) qs[m * dk + c] = to_f32(q[(size_t)((kvh * 2 + m) * group + in_group) * dk + c]);
  __syncwarp();
  float mx[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  float acc[2][DIFF_MAX_D / 32];
#pragma unroll
  for (int i = 0; i < DIFF_MAX_D / 32; ++i) acc[0][i] = acc[1][i] = 0.f;
  const int* table = a.block_table + (size_t)seq * a.table_width;
  for (int t0 = lo & ~31; t0 <= p; t0 += 32) {
    const int key = t0 + lane;
    const bool valid = key >= lo && key <= p;
    float s[2] = {-INFINITY, -INFINITY};
    size_t off = 0;
    if (valid) {
      const size_t row = ((size_t)table[key / a.page_size] * a.nkv + kvh) * a.page_size + key % a.page_size;
      off = row * dv;
      const T* kr = kpages + row * 2 * dk;
      for (int m = 0; m < 2; ++m) {
        float dot = 0.f;
        for (int c = 0; c < dk; ++c) dot = fmaf(qs[m * dk + c], to_f32(kr[m * dk + c]), dot);
        s[m] = dot * scale;
      }
    }
    float corr[2];
    for (int m = 0; m < 2; ++m) {
      const float m_new = fmaxf(mx[m], warp_max(s[m]));       // finite: every tile holds at least one valid key
      const float pexp = valid ? expf(s[m] - m_new) : 0.f;
      corr[m] = expf(mx[m] - m_new);
      l[m] = l[m] * corr[m] + warp_sum(pexp);
      mx[m] = m_new;
      ps[m * 32 + lane] = pexp;
    }
    voff[lane] = off;
    __syncwarp();
    const int kmin = max(0, lo - t0), kmax = min(32, p - t0 + 1);
#pragma unroll
    for (int i = 0; i < DIFF_MAX_D / 32; ++i) {
      const int c = lane + 32 * i;
      if (c < dv) {
        float a0 = acc[0][i] * corr[0], a1 = acc[1][i] * corr[1];
        for (int kk = kmin; kk < kmax; ++kk) {
          const float v = to_f32(vpages[voff[kk] + c]);
          a0 = fmaf(ps[kk], v, a0);
          a1 = fmaf(ps[32 + kk], v, a1);
        }
        acc[0][i] = a0;
        acc[1][i] = a1;
      }
    }
    __syncwarp();
  }
  float sq = 0.f;
#pragma unroll
  for (int i = 0; i < DIFF_MAX_D / 32; ++i) {
    const int c = lane + 32 * i;
    if (c < dv) {
      acc[0][i] = acc[0][i] / l[0] - a.lam * (acc[1][i] / l[1]);
      sq = fmaf(acc[0][i], acc[0][i], sq);
    }
  }
  const float f = a.gain / sqrtf(warp_sum(sq) / (float)dv + a.eps);
  T* o = (T*)a.out + ((size_t)token * a.heads + head) * dv;
  const T* gate = (const T*)a.gate + (size_t)token * a.gate_stride + (size_t)head * dv;
#pragma unroll
  for (int i = 0; i < DIFF_MAX_D / 32; ++i) {
    const int c = lane + 32 * i;
    if (c < dv) o[c] = from_f32<T>(acc[0][i] * f / (1.0f + expf(-to_f32(gate[c]))));
  }
}

// ---- tensor cores ---------------------------------------------------------------------------------------------------

template <int DK, int DV>
__global__ void __launch_bounds__(128) diff_prefill_kernel(DiffArgs a) {
  pdl_trigger();
  pdl_wait();
  constexpr int BN = 64, KW = 2 * DK, KT = BN * Tile<KW>::PITCH, VT = BN * Tile<DV>::PITCH, SLAB = DV + 4;
  extern __shared__ __align__(16) unsigned char smem[];     // two stages of (K tile, V tile); reused for the second map's rows
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int map = warp >> 1;
  const int entry = a.items[2 * blockIdx.x], row_tile = a.items[2 * blockIdx.x + 1];
  const int kvh = blockIdx.y;
  const int group = a.heads / a.nkv;
  const int first = a.cu_q[entry], n = a.cu_q[entry + 1] - first, start = a.q_start_pos[entry];
  const int rows = n * group;
  const int tile_row0 = row_tile * 32;
  const int t_first = tile_row0 / group, t_last = min(tile_row0 + 31, rows - 1) / group;
  KeyWalk walk;
  walk.set(start + t_first, start + t_last, a.window, 0, BN);
  const int* table = a.block_table + (size_t)entry * a.table_width;
  const int w_row0 = tile_row0 + (warp & 1) * 16;
  const int r0 = w_row0 + g, r1 = r0 + 8;
  const int tok0 = r0 < rows ? r0 / group : -1, tok1 = r1 < rows ? r1 / group : -1;
  const int p0 = tok0 < 0 ? -1 : start + tok0, p1 = tok1 < 0 ? -1 : start + tok1;
  const bf16* q = (const bf16*)a.q;
  unsigned qf[DK / 16][4];
  load_q<DK>(qf, [&](int r) -> const bf16* {
    const int rr = w_row0 + r;
    return rr < rows ? q + (size_t)(first + rr / group) * a.q_stride + (size_t)((kvh * 2 + map) * group + rr % group) * DK : nullptr;
  });
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  float o[DV / 8][4];
#pragma unroll
  for (int i = 0; i < DV / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  const int wp_min = w_row0 + 15 < rows ? start + w_row0 / group : -1, wp_max = start + min(w_row0 + 15, rows - 1) / group;

  int key0, rl, rh;
  walk.tile(0, BN, key0, rl, rh);
  biased_load_tile<KW, DV, BN, 128>(smem, smem + KT, a, table, kvh, key0, walk.hi, threadIdx.x);
  cp_async_commit();
  for (int i = 0; i < walk.n_tiles; ++i) {
    unsigned char* cur = smem + (i & 1) * (KT + VT);
    if (i + 1 < walk.n_tiles) {
      int nk0, nrl, nrh;
      walk.tile(i + 1, BN, nk0, nrl, nrh);
      unsigned char* nxt = smem + ((i + 1) & 1) * (KT + VT);
      biased_load_tile<KW, DV, BN, 128>(nxt, nxt + KT, a, table, kvh, nk0, walk.hi, threadIdx.x);
      cp_async_commit();
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    walk.tile(i, BN, key0, rl, rh);
    const unsigned char* ks = cur + map * DK * 2;
    if (tile_is_full(key0, BN, rl, rh, wp_min, wp_max, a.window, 0))
      biased_tile<DK, DV, BN, true, false, true, KW>(qf, ks, cur + KT, key0, rl, rh, p0, p1, a.window, 0, a.scale_log2, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, nullptr, nullptr, 1, 0, m, l, o);
    else
      biased_tile<DK, DV, BN, false, false, true, KW>(qf, ks, cur + KT, key0, rl, rh, p0, p1, a.window, 0, a.scale_log2, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, nullptr, nullptr, 1, 0, m, l, o);
    __syncthreads();
  }
  const float l0 = quad_sum(l[0]), l1 = quad_sum(l[1]);
  const float i0 = l0 > 0.f ? 1.0f / l0 : 0.f, i1 = l1 > 0.f ? 1.0f / l1 : 0.f;
  float* slab = reinterpret_cast<float*>(smem);              // [32 rows][SLAB]; everybody is done with the tiles
  const int s0 = (warp & 1) * 16 + g;
  if (map == 1) {
#pragma unroll
    for (int nb = 0; nb < DV / 8; ++nb) {
      const int c = nb * 8 + 2 * t;
      *reinterpret_cast<float2*>(slab + s0 * SLAB + c) = make_float2(o[nb][0] * i0, o[nb][1] * i0);
      *reinterpret_cast<float2*>(slab + (s0 + 8) * SLAB + c) = make_float2(o[nb][2] * i1, o[nb][3] * i1);
    }
  }
  __syncthreads();
  if (map == 1) return;
  float q0 = 0.f, q1 = 0.f;
#pragma unroll
  for (int nb = 0; nb < DV / 8; ++nb) {
    const int c = nb * 8 + 2 * t;
    const float2 b0 = *reinterpret_cast<const float2*>(slab + s0 * SLAB + c), b1 = *reinterpret_cast<const float2*>(slab + (s0 + 8) * SLAB + c);
    o[nb][0] = fmaf(-a.lam, b0.x, o[nb][0] * i0); o[nb][1] = fmaf(-a.lam, b0.y, o[nb][1] * i0);
    o[nb][2] = fmaf(-a.lam, b1.x, o[nb][2] * i1); o[nb][3] = fmaf(-a.lam, b1.y, o[nb][3] * i1);
    q0 = fmaf(o[nb][0], o[nb][0], q0); q0 = fmaf(o[nb][1], o[nb][1], q0);
    q1 = fmaf(o[nb][2], o[nb][2], q1); q1 = fmaf(o[nb][3], o[nb][3], q1);
  }
  const float f0 = a.gain / sqrtf(quad_sum(q0) / (float)DV + a.eps), f1 = a.gain / sqrtf(quad_sum(q1) / (float)DV + a.eps);
  const int h0 = kvh * group + (tok0 >= 0 ? r0 % group : 0), h1 = kvh * group + (tok1 >= 0 ? r1 % group : 0);
  const bf16* gate = (const bf16*)a.gate;
  bf16* out = (bf16*)a.out;
#pragma unroll
  for (int nb = 0; nb < DV / 8; ++nb) {
    const int c = nb * 8 + 2 * t;
    if (tok0 >= 0) {
      const float2 z = gate_pair(gate + (size_t)(first + tok0) * a.gate_stride + (size_t)h0 * DV + c);
      *reinterpret_cast<unsigned*>(out + ((size_t)(first + tok0) * a.heads + h0) * DV + c) = pack_bf16(o[nb][0] * f0 * z.x, o[nb][1] * f0 * z.y);
    }
    if (tok1 >= 0) {
      const float2 z = gate_pair(gate + (size_t)(first + tok1) * a.gate_stride + (size_t)h1 * DV + c);
      *reinterpret_cast<unsigned*>(out + ((size_t)(first + tok1) * a.heads + h1) * DV + c) = pack_bf16(o[nb][2] * f1 * z.x, o[nb][3] * f1 * z.y);
    }
  }
}

// One head's two finished maps -> its channels of the result, by a warp: y(map, c) gives channel c of a map.
template <int DV, typename Y>
__device__ __forceinline__ void diff_finish_head(const DiffArgs& a, int token, int head, Y y) {
  const int lane = threadIdx.x & 31;
  float v[DV / 32], sq = 0.f;
#pragma unroll
  for (int i = 0; i < DV / 32; ++i) {
    v[i] = y(0, lane + 32 * i) - a.lam * y(1, lane + 32 * i);
    sq = fmaf(v[i], v[i], sq);
  }
  const float f = a.gain / sqrtf(warp_sum(sq) / (float)DV + a.eps);
  const bf16* gate = (const bf16*)a.gate + (size_t)token * a.gate_stride + (size_t)head * DV;
  bf16* out = (bf16*)a.out + ((size_t)token * a.heads + head) * DV;
#pragma unroll
  for (int i = 0; i < DV / 32; ++i) out[lane + 32 * i] = __float2bfloat16_rn(v[i] * f * gate_one(gate + lane + 32 * i));
}

// Single tokens: blockIdx.x = item, blockIdx.y = kv head, blockIdx.z = key range.  Rows: (map, head of the group).
template <int DK, int DV>
__global__ void __launch_bounds__(128) diff_decode_kernel(DiffArgs a) {
  pdl_trigger();
  pdl_wait();
  constexpr int BN = 32, KW = 2 * DK, KT = BN * Tile<KW>::PITCH, VT = BN * Tile<DV>::PITCH, WARP_BYTES = 2 * (KT + VT);
  constexpr int SLAB = DV + 4;
  extern __shared__ __align__(16) unsigned char smem[];     // per warp two stages of (K, V); reused for the merge
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int item = blockIdx.x, kvh = blockIdx.y, split = blockIdx.z;
  const int entry = a.items[item];
  const int group = a.heads / a.nkv, rows = 2 * group;
  const int token = a.cu_q[entry], p = a.q_start_pos[entry];
  KeyWalk walk;
  walk.set(p, p, a.window, 0, BN);
  const int per = (walk.n_tiles + a.n_splits - 1) / a.n_splits;
  const int t_begin = split * per, t_end = min(walk.n_tiles, t_begin + per);
  const int* table = a.block_table + (size_t)entry * a.table_width;
  const int p0 = g < rows ? p : -1, p1 = g + 8 < rows ? p : -1;
  unsigned qf[KW / 16][4];
  {
    const bf16* q = (const bf16*)a.q + (size_t)token * a.q_stride + (size_t)kvh * rows * DK;
    const bf16* q0 = g < rows ? q + (size_t)g * DK : nullptr;
    const bf16* q1 = g + 8 < rows ? q + (size_t)(g + 8) * DK : nullptr;
    const int m0 = g >= group, m1 = g + 8 >= group;
#pragma unroll
    for (int ks = 0; ks < KW / 16; ++ks) {
      const int c = (ks % (DK / 16)) * 16 + 2 * t, of = ks / (DK / 16);
      const bool in0 = q0 && m0 == of, in1 = q1 && m1 == of;
      qf[ks][0] = in0 ? *reinterpret_cast<const unsigned*>(q0 + c) : 0u;
      qf[ks][1] = in1 ? *reinterpret_cast<const unsigned*>(q1 + c) : 0u;
      qf[ks][2] = in0 ? *reinterpret_cast<const unsigned*>(q0 + c + 8) : 0u;
      qf[ks][3] = in1 ? *reinterpret_cast<const unsigned*>(q1 + c + 8) : 0u;
    }
  }
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  float o[DV / 8][4];
#pragma unroll
  for (int i = 0; i < DV / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  unsigned char* mine = smem + warp * WARP_BYTES;
  int key0, rl, rh;
  int i = t_begin + warp;
  if (i < t_end) {
    walk.tile(i, BN, key0, rl, rh);
    biased_load_tile<KW, DV, BN, 32>(mine, mine + KT, a, table, kvh, key0, walk.hi, lane);
  }
  cp_async_commit();
  for (int stage = 0; i < t_end; i += 4, stage ^= 1) {
    unsigned char* cur = mine + stage * (KT + VT);
    if (i + 4 < t_end) {
      int nk0, nrl, nrh;
      walk.tile(i + 4, BN, nk0, nrl, nrh);
      unsigned char* nxt = mine + (stage ^ 1) * (KT + VT);
      biased_load_tile<KW, DV, BN, 32>(nxt, nxt + KT, a, table, kvh, nk0, walk.hi, lane);
      cp_async_commit();
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncwarp();
    walk.tile(i, BN, key0, rl, rh);
    biased_tile<KW, DV, BN, false, false, true>(qf, cur, cur + KT, key0, rl, rh, p0, p1, a.window, 0, a.scale_log2, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, nullptr, nullptr, 1, 0, m, l, o);
    __syncwarp();
  }
  cp_async_wait<0>();
  __syncthreads();                                           // every warp is done with its tiles
  float* ml = reinterpret_cast<float*>(smem);                // [4 warps][16 rows][2]
  float* slab = ml + 4 * 16 * 2;                             // [4 warps][16 rows][SLAB]
  const float l0 = quad_sum(l[0]), l1 = quad_sum(l[1]);
  if (t == 0) {
    ml[(warp * 16 + g) * 2] = m[0]; ml[(warp * 16 + g) * 2 + 1] = l0;
    ml[(warp * 16 + g + 8) * 2] = m[1]; ml[(warp * 16 + g + 8) * 2 + 1] = l1;
  }
#pragma unroll
  for (int nb = 0; nb < DV / 8; ++nb) {
    const int c = nb * 8 + 2 * t;
    *reinterpret_cast<float2*>(slab + (warp * 16 + g) * SLAB + c) = make_float2(o[nb][0], o[nb][1]);
    *reinterpret_cast<float2*>(slab + (warp * 16 + g + 8) * SLAB + c) = make_float2(o[nb][2], o[nb][3]);
  }
  __syncthreads();
  // the warps' shares of a row added up: (max, sum, channel c)
  auto merge = [&](int r, int c, float& mm, float& sum) {
    mm = -INFINITY;
    for (int w = 0; w < 4; ++w) mm = fmaxf(mm, ml[(w * 16 + r) * 2]);
    float acc = 0.f;
    sum = 0.f;
    for (int w = 0; w < 4; ++w) {
      const float mw = ml[(w * 16 + r) * 2];
      const float f = mw == -INFINITY ? 0.f : exp2f(mw - mm);
      sum = fmaf(ml[(w * 16 + r) * 2 + 1], f, sum);
      acc = fmaf(slab[(w * 16 + r) * SLAB + c], f, acc);
    }
    return acc;
  };
  if (a.n_splits == 1) {
    for (int h = warp; h < group; h += 4)
      diff_finish_head<DV>(a, token, kvh * group + h, [&](int map, int c) {
        float mm, sum;
        const float acc = merge(map * group + h, c, mm, sum);
        return sum > 0.f ? acc / sum : 0.f;
      });
  } else {
    for (int x = threadIdx.x; x < rows * DV; x += 128) {
      const int r = x / DV, c = x % DV;
      float mm, sum;
      const float acc = merge(r, c, mm, sum);
      const size_t at = ((size_t)item * 2 * a.heads + kvh * rows + r) * a.n_splits + split;
      a.part_o[at * DV + c] = acc;
      if (c == 0) { a.part_ml[at * 2] = mm; a.part_ml[at * 2 + 1] = sum; }
    }
  }
}

// Adds the key ranges of a token's maps up, in order, and finishes the heads: a warp per (item, head), DV / 32 neighbouring
// channels a lane.  A lane holds the (max, sum) of up to two ranges of each map; both maps' ranges are in flight together.
#define DIFF_MAX_SPLITS 64
template <int DV>
__global__ void __launch_bounds__(128) diff_combine_kernel(DiffArgs a) {
  pdl_trigger();
  pdl_wait();
  constexpr int CPL = DV / 32;
  const int item = blockIdx.x, head = blockIdx.y * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (head >= a.heads) return;
  const int group = a.heads / a.nkv, kvh = head / group;
  const int token = a.cu_q[a.items[item]];
  float w[2][2], acc[2][CPL], inv[2];
  size_t base[2];
#pragma unroll
  for (int map = 0; map < 2; ++map) {
    base[map] = ((size_t)item * 2 * a.heads + (kvh * 2 + map) * group + head % group) * a.n_splits;
    float2 ml[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int s = lane + 32 * i;
      ml[i] = s < a.n_splits ? *reinterpret_cast<const float2*>(a.part_ml + (base[map] + s) * 2) : make_float2(-INFINITY, 0.f);
    }
    const float mm = warp_max(fmaxf(ml[0].x, ml[1].x));
#pragma unroll
    for (int i = 0; i < 2; ++i) w[map][i] = ml[i].x == -INFINITY ? 0.f : exp2f(ml[i].x - mm);
    const float sum = warp_sum(fmaf(ml[0].y, w[map][0], ml[1].y * w[map][1]));
    inv[map] = sum > 0.f ? 1.0f / sum : 0.f;
#pragma unroll
    for (int c = 0; c < CPL; ++c) acc[map][c] = 0.f;
  }
#pragma unroll 4
  for (int s = 0; s < a.n_splits; ++s)
#pragma unroll
    for (int map = 0; map < 2; ++map) {
      const float f = __shfl_sync(0xffffffffu, s < 32 ? w[map][0] : w[map][1], s & 31);
      const float* o = a.part_o + (base[map] + s) * DV + lane * CPL;
      float v[CPL];
      if constexpr (CPL == 4) { const float4 t = *reinterpret_cast<const float4*>(o); v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w; }
      else if constexpr (CPL == 2) { const float2 t = *reinterpret_cast<const float2*>(o); v[0] = t.x; v[1] = t.y; }
      else v[0] = o[0];
#pragma unroll
      for (int c = 0; c < CPL; ++c) acc[map][c] = fmaf(v[c], f, acc[map][c]);
    }
  float y[CPL], sq = 0.f;
#pragma unroll
  for (int c = 0; c < CPL; ++c) { y[c] = acc[0][c] * inv[0] - a.lam * (acc[1][c] * inv[1]); sq = fmaf(y[c], y[c], sq); }
  const float f = a.gain / sqrtf(warp_sum(sq) / (float)DV + a.eps);
  const bf16* gate = (const bf16*)a.gate + (size_t)token * a.gate_stride + (size_t)head * DV + lane * CPL;
  bf16* out = (bf16*)a.out + ((size_t)token * a.heads + head) * DV + lane * CPL;
#pragma unroll
  for (int c = 0; c < CPL; ++c) out[c] = __float2bfloat16_rn(y[c] * f * gate_one(gate + c));
}

template <int DK, int DV>
static int diff_mma_launch(const DiffArgs& a, int n_tiles, int n_items, const int* tiles, const int* items, cudaStream_t s) {
  if (n_tiles > 0) {
    constexpr int TILES = 2 * 64 * (Tile<2 * DK>::PITCH + Tile<DV>::PITCH), MAP2 = 32 * (DV + 4) * 4;
    constexpr int SMEM = TILES > MAP2 ? TILES : MAP2;
    if (SMEM > 48 * 1024) {
      const cudaError_t e = cudaFuncSetAttribute(diff_prefill_kernel<DK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM);
      if (e != cudaSuccess) return (int)e;
    }
    DiffArgs b = a;
    b.items = tiles;
    launch(diff_prefill_kernel<DK, DV>, dim3(n_tiles, a.nkv), dim3(128), SMEM, s, b);
  }
  if (n_items > 0) {
    constexpr int TILES = 4 * 2 * 32 * (Tile<2 * DK>::PITCH + Tile<DV>::PITCH), MERGE = (4 * 16 * 2 + 4 * 16 * (DV + 4)) * 4;
    constexpr int SMEM = TILES > MERGE ? TILES : MERGE;
    if (SMEM > 48 * 1024) {
      const cudaError_t e = cudaFuncSetAttribute(diff_decode_kernel<DK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM);
      if (e != cudaSuccess) return (int)e;
    }
    DiffArgs b = a;
    b.items = items;
    launch(diff_decode_kernel<DK, DV>, dim3(n_items, a.nkv, a.n_splits), dim3(128), SMEM, s, b);
    if (a.n_splits > 1) launch(diff_combine_kernel<DV>, dim3(n_items, (a.heads + 3) / 4), dim3(128), 0, s, b);
  }
  return launch_status();
}

// Sizes the tensor-core kernels are built for: a map's keys of 32, 64 or 128 channels over values of 32, 64 or 128.
#define DIFF_SIZES(X) X(32, 32) X(32, 64) X(32, 128) X(64, 32) X(64, 64) X(64, 128) X(128, 32) X(128, 64) X(128, 128)

static void diff_fill(DiffArgs& a, const void* q, int q_stride, const void* gate, int gate_stride, void* out, const void* kp, const void* vp, const int* bt,
                      int tw, const int* cu, const int* sp, int heads, int nkv, int dv, int ps, int window, float scale, float lam, float gain, float eps) {
  a.q = q; a.q_stride = q_stride; a.gate = gate; a.gate_stride = gate_stride; a.out = out; a.kpages = (const bf16*)kp; a.vpages = (const bf16*)vp;
  a.block_table = bt; a.table_width = tw; a.cu_q = cu; a.q_start_pos = sp; a.items = nullptr; a.heads = heads; a.nkv = nkv; a.page_size = ps;
  a.window = window; a.v_row = dv; a.scale_log2 = scale * 1.4426950408889634f; a.lam = lam; a.gain = gain; a.eps = eps; a.n_splits = 1;
  a.part_o = a.part_ml = nullptr;
}

// tiles: (entry, tile of 32 (token, head) pairs) of the runs; items: the entries of one token (groups of up to 8 heads).
Q25_EXPORT int q25_differential_attention_mma_bf16(const void* q, int q_stride, const void* gate, int gate_stride, void* out, const void* kp, const void* vp,
                                                   const int* bt, int tw, const int* cu, const int* sp, const int* tiles, int n_tiles, const int* items,
                                                   int n_items, int heads, int nkv, int dk, int dv, int ps, int window, float scale, float lam, float gain,
                                                   float eps, int n_splits, float* part_o, float* part_ml, void* stream) {
  if (n_tiles <= 0 && n_items <= 0) return 0;
  if (nkv <= 0 || heads <= 0 || heads % nkv || ps <= 0 || window < 0 || n_splits < 1 || n_splits > DIFF_MAX_SPLITS || (((uintptr_t)part_o | (uintptr_t)part_ml) & 15) || (n_items > 0 && heads / nkv > 8) || q_stride % 2 || gate_stride % 2 ||
      (((uintptr_t)q | (uintptr_t)gate | (uintptr_t)out) & 3) || (((uintptr_t)kp | (uintptr_t)vp) & 15) || (n_splits > 1 && (!part_o || !part_ml)))
    return (int)cudaErrorInvalidValue;
  DiffArgs a;
  diff_fill(a, q, q_stride, gate, gate_stride, out, kp, vp, bt, tw, cu, sp, heads, nkv, dv, ps, window, scale, lam, gain, eps);
  a.n_splits = n_splits; a.part_o = part_o; a.part_ml = part_ml;
#define DIFF_CASE(K, V) if (dk == K && dv == V) return diff_mma_launch<K, V>(a, n_tiles, n_items, tiles, items, (cudaStream_t)stream);
  DIFF_SIZES(DIFF_CASE)
#undef DIFF_CASE
  return (int)cudaErrorInvalidValue;
}

template <typename T>
static int diff_generic(const void* q, int q_stride, const void* gate, int gate_stride, void* out, const void* kp, const void* vp, const int* bt, int tw,
                        const int* ts, const int* cu, const int* sp, int n_tokens, int heads, int nkv, int dk, int dv, int ps, int window, float scale,
                        float lam, float gain, float eps, void* stream) {
  if (n_tokens <= 0) return 0;
  if (nkv <= 0 || heads <= 0 || heads % nkv || ps <= 0 || window < 0 || dk <= 0 || dk > 2048 || dv <= 0 || dv > DIFF_MAX_D) return (int)cudaErrorInvalidValue;
  DiffArgs a;
  diff_fill(a, q, q_stride, gate, gate_stride, out, kp, vp, bt, tw, cu, sp, heads, nkv, dv, ps, window, scale, lam, gain, eps);
  const unsigned blocks = (unsigned)(((long long)n_tokens * heads + DIFF_WARPS - 1) / DIFF_WARPS);
  // room for the longer of the offsets first: every warp's part starts on an 8-byte boundary
  const size_t smem = DIFF_WARPS * ((size_t)(2 * dk + 64) * sizeof(float) + 32 * sizeof(size_t));
  if (smem > 48 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(diff_attention_generic_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  launch(diff_attention_generic_kernel<T>, dim3(blocks), dim3(DIFF_WARPS * 32), smem, (cudaStream_t)stream, a, (const T*)kp, (const T*)vp, ts, n_tokens, dk, dv,
         scale);
  return launch_status();
}
Q25_EXPORT int q25_differential_attention_generic_f32(const void* q, int qs, const void* g, int gs, void* out, const void* kp, const void* vp, const int* bt, int tw,
        const int* ts, const int* cu, const int* sp, int n, int heads, int nkv, int dk, int dv, int ps, int window, float scale, float lam, float gain, float eps, void* s) {
  return diff_generic<float>(q, qs, g, gs, out, kp, vp, bt, tw, ts, cu, sp, n, heads, nkv, dk, dv, ps, window, scale, lam, gain, eps, s);
}
Q25_EXPORT int q25_differential_attention_generic_bf16(const void* q, int qs, const void* g, int gs, void* out, const void* kp, const void* vp, const int* bt, int tw,
        const int* ts, const int* cu, const int* sp, int n, int heads, int nkv, int dk, int dv, int ps, int window, float scale, float lam, float gain, float eps, void* s) {
  return diff_generic<bf16>(q, qs, g, gs, out, kp, vp, bt, tw, ts, cu, sp, n, heads, nkv, dk, dv, ps, window, scale, lam, gain, eps, s);
}
