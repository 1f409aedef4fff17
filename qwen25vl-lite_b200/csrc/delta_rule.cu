// The gated delta rule (Yang, Kautz, Hatamizadeh, "Gated Delta Networks: Improving Mamba2 with Delta Rule"): per head a
// state S [D, V] in float, carried from token to token,
//
//   S <- g_t S,   u_t = beta_t (v_t - S^T k_t),   S <- S + k_t u_t^T,   o_t = S^T q_t
//
// with k_t = k'_t / |k'_t|, q_t = q_scale q'_t / |q'_t| (unit_eps inside the root), g_t = exp(-exp(A_log) softplus(a_t +
// dt_bias)) and beta_t = sigmoid(b_t).  q', k' and v are the rows a convolution leaves ([q' | k' | v] in T; q' and k'
// shared by groups of consecutive heads); a and b come as floats, [N, H of a | H of b].  Everything else is float.
//
// The walk (delta_walk_kernel, any sizes, float or bfloat16 rows): a CTA owns a request's run of tokens, one head and a tile
// of columns of S, which stay in registers: a thread has CPT neighbouring columns in RPT neighbouring rows.  Since
// S_t^T q = (g S)^T q + (k . q) u, a token needs one pass over S for both products with it and one barrier.  When a tile is
// the whole head, the CTA also finishes the head: o / rms(o) * weight * silu(gate).
//
// Runs on tensor cores (bfloat16 rows, D of 32, 64 or 128), in chunks of L = 64 tokens.  With c_t the sum of log g up to t
// within the chunk and S the state before it,
//
//   (I + A) U = diag(beta) (V - diag(e^c) K S),   A_tj = beta_t e^(c_t - c_j) (k_t . k_j) below the diagonal
//   o_t = e^(c_t) S^T q_t + sum_(j <= t) e^(c_t - c_j) (q_t . k_j) u_j
//   S  <- e^(c_L) S + sum_j e^(c_L - c_j) k_j u_j^T
//
// so with T = (I + A)^-1 diag(beta), U = T V - (T diag(e^c) K) S = Uv - Y S.  delta_prepare_kernel makes Y, Uv and the scores M
// of every chunk and head at once (they do not depend on S); delta_run_kernel follows a run's chunks, a CTA per head and
// columns, S in its accumulators: U = Uv - Y S and Q S, then o and the new S.
//
// Products are mma.sync with float accumulators.  The raw k', q' and v are bfloat16 and go in as they are; the norms are
// factors of rows.  What is float by nature (T, Y, M, S, U and its weighted copy) enters as a sum of two bfloat16 numbers,
// the rounded value and what the rounding left, in two products (three where both operands are sums: the product of the two
// rests is left out), which carries 16 bits of mantissa.  The inverse is float: the four 16 x 16 blocks on the diagonal by
// forward substitution, the blocks below from them.
#include "mma.cuh"

struct DeltaArgs {
  const void* x;            // [N, x_stride] in T: q' of all kv heads, k' of all kv heads, v of all heads
  int x_stride, k_off, v_off;
  const float* gates;       // [N, 2 H]
  const float* step_bias;   // [H]
  const float* rate_log;    // [H]
  float* state;             // slot * slot_floats + [H][D][V]
  size_t slot_floats;
  const int* cu_q;
  const int* slot_ids;
  const int* items;         // (first token row, end, entry); nullptr: entry y of cu_q
  float* o_raw;             // [N, H, V]; nullptr: the walk finishes the heads itself
  const void* gate;         // [N, gate_stride] in T
  int gate_stride;
  const float* weight;      // [H, V]
  void* out;                // [N, out_stride] in T
  int out_stride;
  float norm_eps, q_scale, unit_eps;
  int H, share, D, V;
};

__device__ __forceinline__ float delta_log_decay(float a, float bias, float rate_log) {
  const float z = a + bias;
  return -expf(rate_log) * (fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))));
}

#define DW_TOKENS 8          // tokens staged at a time

// blockDim = (column groups, row groups).  Shared memory: k, q [DW_TOKENS][Dp], (g, beta, k . q, -) [DW_TOKENS][4], partial
// products [2][row groups][2][columns], results [DW_TOKENS][columns].
template <typename T, int CPT, int RPT>
__global__ void __launch_bounds__(CPT == 4 ? 512 : 1024) delta_walk_kernel(DeltaArgs p) {
  pdl_trigger();
  extern __shared__ __align__(16) float dw_smem[];
  const int CG = blockDim.x, RG = blockDim.y, cols = CG * CPT, Dp = RG * RPT;
  const int cg = threadIdx.x, rg = threadIdx.y, tid = rg * CG + cg, n_threads = CG * RG;
  const int head = blockIdx.x, col0 = blockIdx.z * cols, c0 = cg * CPT, r0 = rg * RPT;
  float* k_s = dw_smem;
  float* q_s = k_s + DW_TOKENS * Dp;
  float* sc = q_s + DW_TOKENS * Dp;
  float* part = sc + DW_TOKENS * 4;
  float* o_s = part + 2 * RG * 2 * cols;
  const float bias = p.step_bias[head], rate = p.rate_log[head];
  int begin, end, entry = blockIdx.y;
  if (p.items) { const int* it = p.items + 3 * blockIdx.y; begin = it[0]; end = it[1]; entry = it[2]; }
  else { begin = p.cu_q[entry]; end = p.cu_q[entry + 1]; }
  pdl_wait();
  float* st = p.state + (size_t)p.slot_ids[entry] * p.slot_floats + (size_t)head * p.D * p.V + col0;
  const T* x = (const T*)p.x;
  const int left = p.V - col0;                            // columns of this tile that exist
  float S[RPT][CPT];
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int r = r0 + i;
    if (CPT == 4) {
      const float4 v = (r < p.D && c0 < left) ? *reinterpret_cast<const float4*>(st + (size_t)r * p.V + c0) : make_float4(0.f, 0.f, 0.f, 0.f);
      S[i][0] = v.x; S[i][CPT > 1 ? 1 : 0] = v.y; S[i][CPT > 2 ? 2 : 0] = v.z; S[i][CPT > 3 ? 3 : 0] = v.w;
    } else {
      S[i][0] = (r < p.D && c0 < left) ? st[(size_t)r * p.V + c0] : 0.f;
    }
  }
  const size_t q_at = (size_t)(head / p.share) * p.D, k_at = p.k_off + q_at, v_at = p.v_off + (size_t)head * p.V + col0;
  const int warp = tid >> 5, lane = tid & 31, full_warps = n_threads >> 5;
  for (int t0 = begin; t0 < end; t0 += DW_TOKENS) {
    const int nt = min(DW_TOKENS, end - t0);
    __syncthreads();
    // a warp per token: unit vectors and the token's numbers (the last warp may be partly filled: it stays out)
    if (warp < full_warps) {
      for (int t = warp; t < nt; t += full_warps) {
        const T* row = x + (size_t)(t0 + t) * p.x_stride;
        float kk = 0.f, qq = 0.f, kq = 0.f;
        for (int r = lane; r < Dp; r += 32) {
          const float kv = r < p.D ? to_f32(row[k_at + r]) : 0.f, qv = r < p.D ? to_f32(row[q_at + r]) : 0.f;
          k_s[t * Dp + r] = kv; q_s[t * Dp + r] = qv;
          kk = fmaf(kv, kv, kk); qq = fmaf(qv, qv, qq); kq = fmaf(kv, qv, kq);
        }
        kk = warp_sum(kk); qq = warp_sum(qq); kq = warp_sum(kq);
        const float ik = 1.0f / sqrtf(kk + p.unit_eps), iq = p.q_scale / sqrtf(qq + p.unit_eps);
        for (int r = lane; r < Dp; r += 32) { k_s[t * Dp + r] *= ik; q_s[t * Dp + r] *= iq; }
        if (lane == 0) {
          const float* gt = p.gates + (size_t)(t0 + t) * 2 * p.H + head;
          sc[t * 4] = expf(delta_log_decay(gt[0], bias, rate));
          sc[t * 4 + 1] = 1.0f / (1.0f + expf(-gt[p.H]));
          sc[t * 4 + 2] = kq * ik * iq;
        }
      }
    }
    __syncthreads();
    for (int t = 0; t < nt; ++t) {
      const float g = sc[t * 4], beta = sc[t * 4 + 1], kq = sc[t * 4 + 2];
      float v[CPT], pk[CPT], pq[CPT];
#pragma unroll
      for (int c = 0; c < CPT; ++c) {
        v[c] = c0 + c < left ? to_f32(x[(size_t)(t0 + t) * p.x_stride + v_at + c0 + c]) : 0.f;
        pk[c] = pq[c] = 0.f;
      }
      const float *kt = k_s + t * Dp + r0, *qt = q_s + t * Dp + r0;
#pragma unroll
      for (int i = 0; i < RPT; ++i) {
        const float kv = kt[i], qv = qt[i];
#pragma unroll
        for (int c = 0; c < CPT; ++c) {
          S[i][c] *= g;
          pk[c] = fmaf(S[i][c], kv, pk[c]);
          pq[c] = fmaf(S[i][c], qv, pq[c]);
        }
      }
      float* mine = part + (t & 1) * RG * 2 * cols;
#pragma unroll
      for (int c = 0; c < CPT; ++c) { mine[(rg * 2) * cols + c0 + c] = pk[c]; mine[(rg * 2 + 1) * cols + c0 + c] = pq[c]; }
      __syncthreads();
      float u[CPT];
#pragma unroll
      for (int c = 0; c < CPT; ++c) u[c] = pq[c] = 0.f;
      for (int s = 0; s < RG; ++s) {
#pragma unroll
        for (int c = 0; c < CPT; ++c) { u[c] += mine[(s * 2) * cols + c0 + c]; pq[c] += mine[(s * 2 + 1) * cols + c0 + c]; }
      }
#pragma unroll
      for (int c = 0; c < CPT; ++c) u[c] = beta * (v[c] - u[c]);
#pragma unroll
      for (int i = 0; i < RPT; ++i) {
        const float kv = kt[i];
#pragma unroll
        for (int c = 0; c < CPT; ++c) S[i][c] = fmaf(kv, u[c], S[i][c]);
      }
      if (rg == 0) {
#pragma unroll
        for (int c = 0; c < CPT; ++c) {
          const float o = fmaf(kq, u[c], pq[c]);
          if (!p.o_raw) o_s[t * cols + c0 + c] = o;
          else if (c0 + c < left) p.o_raw[((size_t)(t0 + t) * p.H + head) * p.V + col0 + c0 + c] = o;
        }
      }
    }
    if (!p.o_raw) {                                       // this tile is the whole head
      __syncthreads();
      if (warp < full_warps)
        for (int t = warp; t < nt; t += full_warps) {
          float sq = 0.f;
          for (int c = lane; c < p.V; c += 32) sq = fmaf(o_s[t * cols + c], o_s[t * cols + c], sq);
          const float inv = 1.0f / sqrtf(warp_sum(sq) / (float)p.V + p.norm_eps);
          const T* gate = (const T*)p.gate + (size_t)(t0 + t) * p.gate_stride + (size_t)head * p.V;
          T* dst = (T*)p.out + (size_t)(t0 + t) * p.out_stride + (size_t)head * p.V;
          for (int c = lane; c < p.V; c += 32) {
            const float z = to_f32(gate[c]);
            dst[c] = from_f32<T>(o_s[t * cols + c] * inv * p.weight[(size_t)head * p.V + c] * (z / (1.0f + expf(-z))));
          }
        }
    }
  }
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int r = r0 + i;
    if (r < p.D && c0 < left) {
      if (CPT == 4) *reinterpret_cast<float4*>(st + (size_t)r * p.V + c0) = make_float4(S[i][0], S[i][CPT > 1 ? 1 : 0], S[i][CPT > 2 ? 2 : 0], S[i][CPT > 3 ? 3 : 0]);
      else st[(size_t)r * p.V + c0] = S[i][0];
    }
  }
}

template <typename T, int CPT, int RPT>
static int delta_walk_shape(const DeltaArgs& p, int n_items, cudaStream_t s) {
  int CG = (p.V + CPT - 1) / CPT;
  if (CG > 32) CG = 32;
  int RG = (p.D + RPT - 1) / RPT;
  while (CG * RG < 32) ++RG;                              // a whole warp at least (the rows past D are empty)
  if (CG * RG > (CPT == 4 ? 512 : 1024)) return (int)cudaErrorInvalidValue;
  const int cols = CG * CPT, Dp = RG * RPT, tiles = (p.V + cols - 1) / cols;
  if (!p.o_raw && tiles != 1) return (int)cudaErrorInvalidValue;
  const size_t smem = ((size_t)2 * DW_TOKENS * Dp + DW_TOKENS * 4 + (size_t)4 * RG * cols + (size_t)DW_TOKENS * cols) * sizeof(float);
  if (smem > 200 * 1024 || tiles > 65535 || n_items > 65535) return (int)cudaErrorInvalidValue;
  if (smem > 48 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(delta_walk_kernel<T, CPT, RPT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  launch(delta_walk_kernel<T, CPT, RPT>, dim3(p.H, n_items, tiles), dim3(CG, RG), smem, s, p);
  return launch_status();
}

// Columns of a head that one CTA of the walk takes at most: up to there it can finish the head.
Q25_EXPORT int q25_delta_walk_columns(int V, int D) { return (V % 4 == 0 && D <= 256) ? 128 : 32; }

template <typename T>
static int delta_walk(const void* x, int x_stride, int k_off, int v_off, const float* gates, const float* step_bias, const float* rate_log, float* state,
                      long long slot_floats, const int* cu_q, const int* slot_ids, const int* items, int n_items, float* o_raw, const void* gate,
                      int gate_stride, const float* weight, float norm_eps, void* out, int out_stride, int H, int G, int D, int V, float q_scale,
                      float unit_eps, void* stream) {
  if (n_items <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || D <= 0 || D > 512 || V <= 0 || (!o_raw && (!gate || !weight || !out))) return (int)cudaErrorInvalidValue;
  DeltaArgs p;
  p.x = x; p.x_stride = x_stride; p.k_off = k_off; p.v_off = v_off; p.gates = gates; p.step_bias = step_bias; p.rate_log = rate_log; p.state = state;
  p.slot_floats = (size_t)slot_floats; p.cu_q = cu_q; p.slot_ids = slot_ids; p.items = items; p.o_raw = o_raw; p.gate = gate; p.gate_stride = gate_stride;
  p.weight = weight; p.out = out; p.out_stride = out_stride; p.norm_eps = norm_eps; p.q_scale = q_scale; p.unit_eps = unit_eps;
  p.H = H; p.share = H / G; p.D = D; p.V = V;
  cudaStream_t s = (cudaStream_t)stream;
  // four columns at a time where every slot's rows start on a 16-byte boundary
  const bool four = q25_delta_walk_columns(V, D) == 128 && slot_floats % 4 == 0 && !((uintptr_t)state & 15);
  if (!o_raw && !four && V > 32) return (int)cudaErrorInvalidValue;
  if (four) return D <= 64 ? delta_walk_shape<T, 4, 8>(p, n_items, s) : delta_walk_shape<T, 4, 16>(p, n_items, s);
  return delta_walk_shape<T, 1, 16>(p, n_items, s);
}
#define DELTA_WALK(SUF, TYPE)                                                                                                                             \
  Q25_EXPORT int q25_delta_walk_##SUF(const void* x, int xs, int ko, int vo, const float* gates, const float* sb, const float* rl, float* st,            \
                                      long long sf, const int* cu, const int* sl, const int* items, int n_items, float* o_raw, const void* gate, int gs, \
                                      const float* w, float ne, void* out, int os, int H, int G, int D, int V, float qsc, float ue, void* s) {          \
    return delta_walk<TYPE>(x, xs, ko, vo, gates, sb, rl, st, sf, cu, sl, items, n_items, o_raw, gate, gs, w, ne, out, os, H, G, D, V, qsc, ue, s);      \
  }
DELTA_WALK(f32, float)
DELTA_WALK(bf16, bf16)

// ---- runs on tensor cores --------------------------------------------------------------------------------------------

#define DL 64                // tokens of a chunk
#define DL_THREADS 256

// What delta_prepare_kernel leaves of a chunk and head (number ch = chunk * H + head).
struct DeltaScratch {
  bf16* y;                   // [ch][2][DL][D]: Y rounded, and what that left
  bf16* m;                   // [ch][2][DL][DL]: the scores M, the same way; above the diagonal's blocks left as they are
  float* uv;                 // [ch][DL][V]
  float* row;                // [ch][2][DL]: e^c q_scale / |q'| and e^(c_last - c) / |k'| of every token
  float* keep;               // [ch]: e^(c_last)
};

__device__ __forceinline__ void split_store(bf16* hi, bf16* lo, float a, float b) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  *reinterpret_cast<__nv_bfloat162*>(hi) = h;
  *reinterpret_cast<__nv_bfloat162*>(lo) = __floats2bfloat162_rn(a - __low2float(h), b - __high2float(h));
}

// blockIdx.x = head, blockIdx.y = chunk.
template <int D>
__global__ void __launch_bounds__(DL_THREADS, 3) delta_prepare_kernel(DeltaArgs p, const int* __restrict__ chunks, DeltaScratch out) {
  constexpr int DP = D + 8, LP = DL + 8, FP = DL + 8, KT = D / 16;
  extern __shared__ __align__(16) unsigned char dp_smem[];
  bf16* Ks = reinterpret_cast<bf16*>(dp_smem);               // [DL][DP]
  bf16* Qs = Ks + DL * DP;                                   // [DL][DP]; then the values, 64 columns at a time
  float* A = reinterpret_cast<float*>(Qs + DL * (DP > LP ? DP : LP));        // [DL][FP]
  float* Ti = A + DL * FP;                                   // [DL][FP]: (I + A)^-1
  float* W = Ti + DL * FP;                                   // [3][16][17]: products on the way to a block below the diagonal
  float* num = W + 3 * 16 * 17;                              // [5][DL]: c, beta, 1 / |k'|, q_scale / |q'|, beta e^c / |k'|
  pdl_trigger();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t2 = (lane & 3) * 2;
  const int head = blockIdx.x, begin = chunks[2 * blockIdx.y], end = chunks[2 * blockIdx.y + 1], n = end - begin;
  const float bias = p.step_bias[head], rate = p.rate_log[head];
  const bf16* x = (const bf16*)p.x;
  const bf16 *qx = x + (size_t)(head / p.share) * D, *kx = qx + p.k_off, *vx = x + p.v_off + (size_t)head * p.V;
  const size_t ch = (size_t)blockIdx.y * p.H + head;
  pdl_wait();
  for (int i = tid; i < DL * (D / 8); i += DL_THREADS) {
    const int r = i / (D / 8), c = (i % (D / 8)) * 8;
    const bool ok = r < n;
    const size_t row = (size_t)(begin + (ok ? r : 0)) * p.x_stride + c;
    cp_async16(Ks + r * DP + c, kx + row, ok);
    cp_async16(Qs + r * DP + c, qx + row, ok);
  }
  cp_async_commit();
  if (warp == 0) {                                           // two neighbouring tokens a lane; tokens past the end: no decay, no write
    float l[2], b[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = 2 * lane + e;
      const float* gt = p.gates + (size_t)(begin + min(t, n - 1)) * 2 * p.H + head;
      l[e] = t < n ? delta_log_decay(gt[0], bias, rate) : 0.f;
      b[e] = t < n ? 1.0f / (1.0f + expf(-gt[p.H])) : 0.f;
    }
    float sum = l[0] + l[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float before = __shfl_up_sync(0xffffffffu, sum, o);
      if (lane >= o) sum += before;
    }
    num[2 * lane] = sum - l[1]; num[2 * lane + 1] = sum;
    num[DL + 2 * lane] = b[0]; num[DL + 2 * lane + 1] = b[1];
  }
  for (int i = tid; i < DL * FP; i += DL_THREADS) Ti[i] = 0.f;
  cp_async_wait<0>();
  __syncthreads();
  for (int r = warp; r < DL; r += DL_THREADS / 32) {
    float kk = 0.f, qq = 0.f;
    for (int c = lane * 2; c < D; c += 64) {
      const float2 k = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(Ks + r * DP + c));
      const float2 q = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(Qs + r * DP + c));
      kk = fmaf(k.x, k.x, fmaf(k.y, k.y, kk)); qq = fmaf(q.x, q.x, fmaf(q.y, q.y, qq));
    }
    kk = warp_sum(kk); qq = warp_sum(qq);
    if (lane == 0) { num[2 * DL + r] = kk; num[3 * DL + r] = qq; }
  }
  __syncthreads();
  if (tid < DL) {
    const float ik = 1.0f / sqrtf(num[2 * DL + tid] + p.unit_eps), iq = p.q_scale / sqrtf(num[3 * DL + tid] + p.unit_eps), ec = expf(num[tid]);
    num[2 * DL + tid] = ik; num[3 * DL + tid] = iq; num[4 * DL + tid] = num[DL + tid] * ec * ik;
    out.row[ch * 2 * DL + tid] = ec * iq;
    out.row[(ch * 2 + 1) * DL + tid] = expf(num[DL - 1] - num[tid]) * ik;
    if (tid == 0) out.keep[ch] = expf(num[DL - 1]);
  }
  __syncthreads();
  // scores: 10 tiles of 16 x 16 on and below the diagonal, of K K^T (jobs 0 .. 9) and Q K^T (10 .. 19)
  for (int job = warp; job < 20; job += DL_THREADS / 32) {
    const bool is_q = job >= 10;
    int ti = 0, tj = is_q ? job - 10 : job;
    while (tj > ti) { tj -= ti + 1; ++ti; }
    float acc[2][4];
#pragma unroll
    for (int h = 0; h < 2; ++h)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[h][e] = 0.f;
    const bf16* R = is_q ? Qs : Ks;
#pragma unroll
    for (int k = 0; k < KT; ++k) {
      unsigned a[4], b[4];
      ldmatrix_x4(a, R + (ti * 16 + (lane & 15)) * DP + k * 16 + (lane >> 4) * 8);
      ldmatrix_x4(b, Ks + (tj * 16 + (lane & 7) + ((lane >> 4) << 3)) * DP + k * 16 + ((lane >> 3) & 1) * 8);
      mma_bf16(acc[0], a, b[0], b[1]);
      mma_bf16(acc[1], a, b[2], b[3]);
    }
#pragma unroll
    for (int h = 0; h < 2; ++h)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int t = ti * 16 + g + e * 8, j = tj * 16 + h * 8 + t2;
        const float left = is_q ? num[3 * DL + t] : num[DL + t] * num[2 * DL + t];
        float v[2];
#pragma unroll
        for (int w = 0; w < 2; ++w) {
          const bool in = is_q ? j + w <= t : j + w < t;
          v[w] = in ? acc[h][2 * e + w] * left * num[2 * DL + j + w] * expf(num[t] - num[j + w]) : 0.f;
        }
        if (is_q) {
          bf16* m = out.m + ch * 2 * DL * DL + (size_t)t * DL + j;
          split_store(m, m + DL * DL, v[0], v[1]);
        } else {
          *reinterpret_cast<float2*>(A + t * FP + j) = make_float2(v[0], v[1]);
        }
      }
  }
  __syncthreads();
  // the values' first columns take the queries' place
  auto fetch_v = [&](int v0) {
    for (int i = tid; i < DL * 8; i += DL_THREADS) {
      const int r = i / 8, c = v0 + (i % 8) * 8;
      const bool ok = r < n && c < p.V;
      cp_async16(Qs + r * LP + (i % 8) * 8, ok ? vx + (size_t)(begin + r) * p.x_stride + c : vx + (size_t)begin * p.x_stride, ok);
    }
    cp_async_commit();
  };
  fetch_v(0);
  // the inverse: blocks on the diagonal, a lane per column
  if (warp < 4 && lane < 16) {
    const float* a = A + warp * 16 * FP + warp * 16;
    float* ti = Ti + warp * 16 * FP + warp * 16;
    float col[16];
#pragma unroll
    for (int r = 0; r < 16; ++r) {
      float v = r == lane ? 1.f : 0.f;
#pragma unroll
      for (int i = 0; i < r; ++i) v = fmaf(-a[r * FP + i], col[i], v);
      col[r] = v;
      ti[r * FP + lane] = v;
    }
  }
  __syncthreads();
  // blocks below: T_IJ = -T_II sum_(J <= K < I) A_IK T_KJ, by distance from the diagonal
  for (int d = 1; d < 4; ++d) {
    for (int i = tid; i < (4 - d) * 256; i += DL_THREADS) {
      const int J = i >> 8, I = J + d, r = (i >> 4) & 15, c = i & 15;
      float v = 0.f;
      for (int k = J * 16; k < I * 16; k += 4) {
        const float4 a = *reinterpret_cast<const float4*>(A + (I * 16 + r) * FP + k);
        v = fmaf(a.x, Ti[k * FP + J * 16 + c], v);
        v = fmaf(a.y, Ti[(k + 1) * FP + J * 16 + c], v);
        v = fmaf(a.z, Ti[(k + 2) * FP + J * 16 + c], v);
        v = fmaf(a.w, Ti[(k + 3) * FP + J * 16 + c], v);
      }
      W[J * 16 * 17 + r * 17 + c] = v;
    }
    __syncthreads();
    for (int i = tid; i < (4 - d) * 256; i += DL_THREADS) {
      const int J = i >> 8, I = J + d, r = (i >> 4) & 15, c = i & 15;
      float v = 0.f;
#pragma unroll
      for (int k = 0; k < 16; ++k) v = fmaf(-Ti[(I * 16 + r) * FP + I * 16 + k], W[J * 16 * 17 + k * 17 + c], v);
      Ti[(I * 16 + r) * FP + J * 16 + c] = v;
    }
    __syncthreads();
  }
  // a 16 x 16 block of the inverse as an operand, its columns times factor: rounded, and what that left
  auto inverse_block = [&](int ti, int j, const float* factor, unsigned (&hi)[4], unsigned (&lo)[4]) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int r = ti * 16 + g + (e & 1) * 8, c = j * 16 + t2 + (e >> 1) * 8;
      const float2 v = *reinterpret_cast<const float2*>(Ti + r * FP + c), f = *reinterpret_cast<const float2*>(factor + c);
      const float a = v.x * f.x, b = v.y * f.y;
      const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
      hi[e] = *reinterpret_cast<const unsigned*>(&h);
      lo[e] = pack_bf16(a - __low2float(h), b - __high2float(h));
    }
  };
  cp_async_wait<0>();
  __syncthreads();
  // Y = T diag(e^c / |k'|) K': a warp has 16 tokens and half of the columns
  const int tile = warp & 3, half = warp >> 2;
  {
    constexpr int NT = D / 16;                               // 8-column tiles of a warp
    float acc[NT][4];
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
    for (int j = 0; j <= tile; ++j) {
      unsigned hi[4], lo[4];
      inverse_block(tile, j, num + 4 * DL, hi, lo);
#pragma unroll
      for (int i = 0; i < NT; ++i) {
        unsigned b[2];
        ldmatrix_x2_trans(b, Ks + (j * 16 + (lane & 15)) * DP + half * (D / 2) + i * 8);
        mma_bf16(acc[i], lo, b[0], b[1]);
        mma_bf16(acc[i], hi, b[0], b[1]);
      }
    }
    bf16* y = out.y + ch * 2 * DL * D;
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const size_t at = (size_t)(tile * 16 + g + e * 8) * D + half * (D / 2) + i * 8 + t2;
        split_store(y + at, y + (size_t)DL * D + at, acc[i][2 * e], acc[i][2 * e + 1]);
      }
  }
  // Uv = T V, 64 columns at a time
  for (int v0 = 0; v0 < p.V; v0 += 64) {
    if (v0 > 0) {
      __syncthreads();
      fetch_v(v0);
      cp_async_wait<0>();
      __syncthreads();
    }
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
    for (int j = 0; j <= tile; ++j) {
      unsigned hi[4], lo[4];
      inverse_block(tile, j, num + DL, hi, lo);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        unsigned b[2];
        ldmatrix_x2_trans(b, Qs + (j * 16 + (lane & 15)) * LP + half * 32 + i * 8);
        mma_bf16(acc[i], lo, b[0], b[1]);
        mma_bf16(acc[i], hi, b[0], b[1]);
      }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int c = v0 + half * 32 + i * 8 + t2;
        if (c < p.V) *reinterpret_cast<float2*>(out.uv + (ch * DL + tile * 16 + g + e * 8) * p.V + c) = make_float2(acc[i][2 * e], acc[i][2 * e + 1]);
      }
  }
}

// items: (first token row, end, entry, first chunk) per run.  blockIdx.x = head * column tiles + tile, blockIdx.y = run.
// Eight warps.  A chunk has two halves with a barrier each: first U = Uv - Y S and Q S (a warp has 16 tokens and half of the
// tile's columns), then o, and the new S (a warp has 16 rows of S, or part of their columns).  Y, q' and Uv of the next chunk are on
// their way during the second half, k' and M during the next first half.
template <int D, int VT>
__global__ void __launch_bounds__(DL_THREADS) delta_run_kernel(DeltaArgs p, const int* __restrict__ items, DeltaScratch in, int v_tiles) {
  constexpr int DP = D + 8, LP = DL + 8, VP = VT + 8, UP = VT + 4, KT = D / 16;
  constexpr int CG = 8 / KT, ST = VT / 8 / CG;               // warps side by side over a row tile of S; 8-column tiles a warp owns there
  constexpr int OT = VT / 16;                                // 8-column tiles of a warp's tokens
  static_assert(KT <= 8 && ST >= 1 && OT >= 1, "sizes");
  extern __shared__ __align__(16) unsigned char dr_smem[];
  bf16* Ys = reinterpret_cast<bf16*>(dr_smem);               // [2][DL][DP]
  bf16* Qs = Ys + 2 * DL * DP;                               // [DL][DP]
  bf16* Ks = Qs + DL * DP;                                   // [DL][DP]
  bf16* Ms = Ks + DL * DP;                                   // [2][DL][LP]
  bf16* Sh = Ms + 2 * DL * LP;                               // [2][D][VP]: S before the chunk, rounded, and what that left
  bf16* Uh = Sh + 2 * D * VP;                                // [2][DL][VP]
  bf16* Wh = Uh + 2 * DL * VP;                               // [2][DL][VP]: U times e^(c_last - c) / |k'|
  float* Uv = reinterpret_cast<float*>(Wh + 2 * DL * VP);    // [DL][UP]
  pdl_trigger();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t2 = (lane & 3) * 2;
  const int head = blockIdx.x / v_tiles, col0 = (blockIdx.x % v_tiles) * VT;
  const int* it = items + 4 * blockIdx.y;
  const int begin = it[0], end = it[1], first = it[3];
  const bf16* x = (const bf16*)p.x;
  const bf16 *qx = x + (size_t)(head / p.share) * D, *kx = qx + p.k_off;
  const int left = p.V - col0;
  pdl_wait();
  float* st = p.state + (size_t)p.slot_ids[it[2]] * p.slot_floats + (size_t)head * D * p.V + col0;

  auto fetch_first = [&](int chunk) {
    const size_t ch = (size_t)(first + chunk) * p.H + head;
    const int t0 = begin + chunk * DL;
    const bf16* y = in.y + ch * 2 * DL * D;
    for (int i = tid; i < 2 * DL * (D / 8); i += DL_THREADS) {
      const int r = i / (D / 8), c = (i % (D / 8)) * 8;
      cp_async16_whole(Ys + r * DP + c, y + (size_t)r * D + c);
    }
    for (int i = tid; i < DL * (D / 8); i += DL_THREADS) {
      const int r = i / (D / 8), c = (i % (D / 8)) * 8;
      const bool ok = t0 + r < end;
      cp_async16(Qs + r * DP + c, qx + (size_t)(ok ? t0 + r : begin) * p.x_stride + c, ok);
    }
    const float* uv = in.uv + ch * DL * p.V + col0;
    for (int i = tid; i < DL * (VT / 4); i += DL_THREADS) {
      const int r = i / (VT / 4), c = (i % (VT / 4)) * 4;
      const bool ok = c < left;
      cp_async16(Uv + r * UP + c, ok ? uv + (size_t)r * p.V + c : uv, ok);
    }
    cp_async_commit();
  };
  auto fetch_second = [&](int chunk) {
    const size_t ch = (size_t)(first + chunk) * p.H + head;
    const int t0 = begin + chunk * DL;
    for (int i = tid; i < DL * (D / 8); i += DL_THREADS) {
      const int r = i / (D / 8), c = (i % (D / 8)) * 8;
      const bool ok = t0 + r < end;
      cp_async16(Ks + r * DP + c, kx + (size_t)(ok ? t0 + r : begin) * p.x_stride + c, ok);
    }
    const bf16* m = in.m + ch * 2 * DL * DL;
    for (int i = tid; i < 2 * DL * (DL / 8); i += DL_THREADS) {
      const int r = i / (DL / 8), c = (i % (DL / 8)) * 8;
      if (c / 16 <= (r % DL) / 16) cp_async16_whole(Ms + r * LP + c, m + (size_t)r * DL + c);      // blocks above the diagonal are never read
    }
    cp_async_commit();
  };

  const int s_row = (warp % KT) * 16, s_col = (warp / KT) * ST * 8;
  float S[ST][4];
#pragma unroll
  for (int i = 0; i < ST; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int r = s_row + g + (e >> 1) * 8, c = s_col + i * 8 + t2 + (e & 1);
      S[i][e] = c < left ? st[(size_t)r * p.V + c] : 0.f;
    }
  auto put_s = [&]() {
#pragma unroll
    for (int i = 0; i < ST; ++i)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        bf16* at = Sh + (s_row + g + e * 8) * VP + s_col + i * 8 + t2;
        split_store(at, at + D * VP, S[i][2 * e], S[i][2 * e + 1]);
      }
  };
  // the last tokens of a chunk have the longest sums over M: their two warps are on different schedulers
  const int o_half = warp >> 2, o_tile = o_half ? 3 - (warp & 3) : (warp & 3);
  const int o_col = o_half * OT * 8;
  const int chunks = (end - begin + DL - 1) / DL;
  fetch_first(0);
  fetch_second(0);
  put_s();
  for (int chunk = 0; chunk < chunks; ++chunk) {
    const size_t ch = (size_t)(first + chunk) * p.H + head;
    const float* row = in.row + ch * 2 * DL;
    float fq[2], fw[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) { fq[e] = row[o_tile * 16 + g + e * 8]; fw[e] = row[DL + o_tile * 16 + g + e * 8]; }
    const float keep = in.keep[ch];
    if (chunk == 0) cp_async_wait<1>(); else cp_async_wait<0>();
    __syncthreads();                          // Y, q', Uv and S of the chunk are in; everybody is done with k' and M of the one before
    if (chunk > 0) fetch_second(chunk);
    // ---- U = Uv - Y S and Q S; sums of rounded operands and of the rests apart (shorter chains of dependent products)
    float u[2][OT][4], qs[2][OT][4];
#pragma unroll
    for (int a = 0; a < 2; ++a)
#pragma unroll
      for (int i = 0; i < OT; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) u[a][i][e] = qs[a][i][e] = 0.f;
#pragma unroll
    for (int k = 0; k < KT; ++k) {
      unsigned yh[4], yl[4], q[4];
      const int at = (o_tile * 16 + (lane & 15)) * DP + k * 16 + (lane >> 4) * 8;
      ldmatrix_x4(yh, Ys + at);
      ldmatrix_x4(yl, Ys + DL * DP + at);
      ldmatrix_x4(q, Qs + at);
#pragma unroll
      for (int i = 0; i < OT; ++i) {
        unsigned b[4];                        // the rounded S (two registers) and the rest (two registers) in one load
        ldmatrix_x4_trans(b, Sh + (lane >> 4) * D * VP + (k * 16 + (lane & 15)) * VP + o_col + i * 8);
        mma_bf16(u[0][i], yh, b[0], b[1]);
        mma_bf16(u[1][i], yh, b[2], b[3]);
        mma_bf16(u[1][i], yl, b[0], b[1]);
        mma_bf16(qs[0][i], q, b[0], b[1]);
        mma_bf16(qs[1][i], q, b[2], b[3]);
      }
    }
#pragma unroll
    for (int i = 0; i < OT; ++i)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int t = o_tile * 16 + g + e * 8, c = o_col + i * 8 + t2;
        const float2 uv = *reinterpret_cast<const float2*>(Uv + t * UP + c);
        const float a = uv.x - (u[0][i][2 * e] + u[1][i][2 * e]), b = uv.y - (u[0][i][2 * e + 1] + u[1][i][2 * e + 1]);
        split_store(Uh + t * VP + c, Uh + (DL + t) * VP + c, a, b);
        split_store(Wh + t * VP + c, Wh + (DL + t) * VP + c, a * fw[e], b * fw[e]);
      }
    cp_async_wait<0>();
    __syncthreads();                          // U and its weighted copy, k' and M are in; everybody is done with Y, q', Uv and S
    if (chunk + 1 < chunks) fetch_first(chunk + 1);
    // ---- outputs
    float y[2][OT][4];
#pragma unroll
    for (int a = 0; a < 2; ++a)
#pragma unroll
      for (int i = 0; i < OT; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) y[a][i][e] = 0.f;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      if (j <= o_tile) {
        unsigned mh[4], ml[4];
        ldmatrix_x4(mh, Ms + (o_tile * 16 + (lane & 15)) * LP + j * 16 + (lane >> 4) * 8);
        ldmatrix_x4(ml, Ms + (DL + o_tile * 16 + (lane & 15)) * LP + j * 16 + (lane >> 4) * 8);
#pragma unroll
        for (int i = 0; i < OT; ++i) {
          unsigned b[4];
          ldmatrix_x4_trans(b, Uh + (lane >> 4) * DL * VP + (j * 16 + (lane & 15)) * VP + o_col + i * 8);
          mma_bf16(y[0][i], mh, b[0], b[1]);
          mma_bf16(y[1][i], mh, b[2], b[3]);
          mma_bf16(y[1][i], ml, b[0], b[1]);
        }
      }
    }
    // ---- the state behind the chunk
    float add[2][ST][4];
#pragma unroll
    for (int a = 0; a < 2; ++a)
#pragma unroll
      for (int i = 0; i < ST; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) add[a][i][e] = 0.f;
#pragma unroll
    for (int k = 0; k < DL / 16; ++k) {
      unsigned a[4];
      ldmatrix_x4_trans(a, Ks + (k * 16 + (lane & 7) + (lane >> 4) * 8) * DP + s_row + ((lane >> 3) & 1) * 8);
#pragma unroll
      for (int i = 0; i < ST; ++i) {
        unsigned b[4];
        ldmatrix_x4_trans(b, Wh + (lane >> 4) * DL * VP + (k * 16 + (lane & 15)) * VP + s_col + i * 8);
        mma_bf16(add[0][i], a, b[0], b[1]);
        mma_bf16(add[1][i], a, b[2], b[3]);
      }
    }
#pragma unroll
    for (int i = 0; i < ST; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) S[i][e] = fmaf(keep, S[i][e], add[0][i][e] + add[1][i][e]);
    put_s();
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int tok = begin + chunk * DL + o_tile * 16 + g + e * 8;
      if (tok < end) {
        float* o = p.o_raw + ((size_t)tok * p.H + head) * p.V + col0;
#pragma unroll
        for (int i = 0; i < OT; ++i) {
          const int c = o_col + i * 8 + t2;
          if (c < left)
            *reinterpret_cast<float2*>(o + c) = make_float2(fmaf(fq[e], qs[0][i][2 * e] + qs[1][i][2 * e], y[0][i][2 * e] + y[1][i][2 * e]),
                                                            fmaf(fq[e], qs[0][i][2 * e + 1] + qs[1][i][2 * e + 1], y[0][i][2 * e + 1] + y[1][i][2 * e + 1]));
        }
      }
    }
  }
#pragma unroll
  for (int i = 0; i < ST; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int r = s_row + g + (e >> 1) * 8, c = s_col + i * 8 + t2 + (e & 1);
      if (c < left) st[(size_t)r * p.V + c] = S[i][e];
    }
}

// Floats of scratch memory per chunk and head.
static size_t delta_scratch_floats(int D, int V) { return (size_t)DL * D + (size_t)DL * DL + (size_t)DL * V + 2 * DL + 4; }
Q25_EXPORT long long q25_delta_scratch_floats(int n_chunks, int H, int D, int V) { return (long long)(delta_scratch_floats(D, V) * n_chunks * H); }

template <int D, int VT>
static int delta_run_shape(const DeltaArgs& p, const int* items, int n_runs, const DeltaScratch& sc, cudaStream_t s) {
  const size_t smem = (size_t)(4 * DL * (D + 8) + 2 * DL * (DL + 8) + (2 * D + 4 * DL) * (VT + 8)) * sizeof(bf16) + (size_t)DL * (VT + 4) * sizeof(float);
  const cudaError_t e = cudaFuncSetAttribute(delta_run_kernel<D, VT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return (int)e;
  const int v_tiles = (p.V + VT - 1) / VT;
  launch(delta_run_kernel<D, VT>, dim3(p.H * v_tiles, n_runs), dim3(DL_THREADS), smem, s, p, items, sc, v_tiles);
  return launch_status();
}

template <int D>
static int delta_prepare(const DeltaArgs& p, const int* chunks, int n_chunks, const DeltaScratch& sc, cudaStream_t s) {
  constexpr int DP = D + 8, LP = DL + 8, FP = DL + 8;
  const size_t smem = (size_t)(DL * DP + DL * (DP > LP ? DP : LP)) * sizeof(bf16) + (size_t)(2 * DL * FP + 3 * 16 * 17 + 5 * DL) * sizeof(float);
  const cudaError_t e = cudaFuncSetAttribute(delta_prepare_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return (int)e;
  launch(delta_prepare_kernel<D>, dim3(p.H, n_chunks), dim3(DL_THREADS), smem, s, p, chunks, sc);
  return launch_status();
}

// Runs of bfloat16 rows.  D is 32, 64 or 128; V a multiple of 8; every row and offset starts on a 16-byte boundary.  chunks:
// (first token row, end) each; runs: (first token row, end, entry, first chunk) each.
Q25_EXPORT int q25_delta_runs_bf16(const void* x, int x_stride, int k_off, int v_off, const float* gates, const float* step_bias, const float* rate_log,
                                   float* state, long long slot_floats, const int* slot_ids, const int* chunks, int n_chunks, const int* runs, int n_runs,
                                   float* scratch, float* o_raw, int H, int G, int D, int V, float q_scale, float unit_eps, void* stream) {
  if (n_runs <= 0 || n_chunks <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || V <= 0 || V % 8 || x_stride % 8 || k_off % 8 || v_off % 8 || (((uintptr_t)x | (uintptr_t)scratch) & 15) ||
      ((uintptr_t)o_raw & 7) || n_runs > 65535 || n_chunks > 65535 || !scratch || !o_raw)
    return (int)cudaErrorInvalidValue;
  DeltaArgs p = {};
  p.x = x; p.x_stride = x_stride; p.k_off = k_off; p.v_off = v_off; p.gates = gates; p.step_bias = step_bias; p.rate_log = rate_log; p.state = state;
  p.slot_floats = (size_t)slot_floats; p.slot_ids = slot_ids; p.o_raw = o_raw; p.q_scale = q_scale; p.unit_eps = unit_eps;
  p.H = H; p.share = H / G; p.D = D; p.V = V;
  const size_t n = (size_t)n_chunks * H;
  DeltaScratch sc;
  sc.y = reinterpret_cast<bf16*>(scratch);
  sc.m = sc.y + n * 2 * DL * D;
  sc.uv = reinterpret_cast<float*>(sc.m + n * 2 * DL * DL);
  sc.row = sc.uv + n * DL * V;
  sc.keep = sc.row + n * 2 * DL;
  cudaStream_t s = (cudaStream_t)stream;
  int rc = (int)cudaErrorInvalidValue;
  if (D == 32) rc = delta_prepare<32>(p, chunks, n_chunks, sc, s);
  else if (D == 64) rc = delta_prepare<64>(p, chunks, n_chunks, sc, s);
  else if (D == 128) rc = delta_prepare<128>(p, chunks, n_chunks, sc, s);
  if (rc) return rc;
  // narrower column tiles while those, too, all run at once
  const int sms = device_sm_count() > 0 ? device_sm_count() : 148;
  const long long per_sm = D == 128 ? 1 : 2;
  const bool narrow = (long long)H * ((V + 15) / 16) * n_runs <= per_sm * sms || V <= 16;
  switch (D) {
    case 32: return delta_run_shape<32, 32>(p, runs, n_runs, sc, s);
    case 64: return narrow ? delta_run_shape<64, 16>(p, runs, n_runs, sc, s) : delta_run_shape<64, 32>(p, runs, n_runs, sc, s);
    default: return narrow ? delta_run_shape<128, 16>(p, runs, n_runs, sc, s) : delta_run_shape<128, 32>(p, runs, n_runs, sc, s);
  }
}
