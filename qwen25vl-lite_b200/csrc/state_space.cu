// The state space of Mamba-2 on tensor cores, for runs of tokens in bfloat16 (Dao, Gu, "Transformers are SSMs: Generalized
// Models and Efficient Algorithms Through Structured State Space Duality").  Per head, with a step d_t = softplus(z_t +
// bias), l_t = -exp(A_log) d_t, and c_t the sum of l up to t within a chunk of SS_TOKENS tokens:
//
//   y_t   = exp(c_t) S^T q_t + sum_(j <= t) exp(c_t - c_j) d_j (q_t . k_j) v_j         S: the state before the chunk
//   S    <- exp(c_last) S + sum_j exp(c_last - c_j) d_j k_j v_j^T
//
// k and q [N] are shared by groups of consecutive heads, v [V] is the head's own.  A CTA owns a request's run, one head
// and VT columns of its state, and takes the chunks one after the other; S never leaves its registers but for a copy of
// it in shared memory, so nothing travels through memory but k, q, v and the results.
//
// All products are mma.sync with float accumulators.  k, q and v are bfloat16 as the convolution leaves them, so q . k
// is exact up to the order of its float sum.  What is float by nature -- the decayed scores, S as an operand, and
// exp(c_last - c_j) d_j v_j -- enters its product as a sum of two bfloat16 numbers (the rounded value and what the
// rounding left), two products each: 16 bits of mantissa, where one rounding would leave 8.  The steps, decays, their
// sums and exponentials and the carried S are float.
//
// Eight warps, two to each 16 tokens of a chunk.  Before a chunk's middle barrier a warp puts its part of S and of the
// weighted values into shared memory and computes its decayed scores (every second 16 x 16 tile of its tokens' row of the
// triangle), which go there too; behind it a warp adds up its tokens' outputs for its columns and updates its 16-row
// tiles of S, which are accumulators.  The next chunk's k and v are on their way (cp.async) from the chunk's first
// barrier on, its q from the middle one (by then q is in registers): what is left in shared memory lets two CTAs share
// an SM.
#include "mma.cuh"

#define SS_TOKENS 64
#define SS_THREADS 256

struct StateSpaceArgs {
  const bf16* x;            // rows: v of all heads at v_off, k and q of all groups at k_off and q_off
  int x_stride, q_off, k_off, v_off;
  const float* z;           // [tokens, H]
  const float* step_bias;   // [H]
  const float* rate_log;    // [H]
  float* state;             // slot * slot_floats + [H][N][V]
  size_t slot_floats;
  const int* slot_ids;
  const int* items;         // (first token row, end, entry) per run
  float* o;                 // [tokens, H, V]
  int H, V, share, v_tiles;
};

template <int N, int VT>
__global__ void __launch_bounds__(SS_THREADS, 2) state_space_kernel(StateSpaceArgs p) {
  constexpr int L = SS_TOKENS, NP = N + 8, VP = VT + 8, LP = L + 8;      // pitches: an odd number of 16-byte pieces
  constexpr int KT = N / 16;                                   // 16-row tiles of S, and k-steps of q . k
  constexpr int CG = 8 / KT, ST = VT / 8 / CG;                 // warps side by side over a row tile of S; 8-column tiles a warp owns there
  constexpr int OT = VT / 16;                                  // 8-column tiles of a warp's outputs
  static_assert(KT <= 8 && ST >= 1, "sizes");
  extern __shared__ __align__(16) unsigned char ss_smem[];
  bf16* Ks = reinterpret_cast<bf16*>(ss_smem);                 // [2][L][NP]
  bf16* Vs = Ks + 2 * L * NP;                                  // [2][L][VP]
  bf16* Qs = Vs + 2 * L * VP;                                  // [L][NP]
  bf16* Sh = Qs + L * NP;                                      // [2][N][VP]: S before the chunk, rounded, and what that left
  bf16* Wh = Sh + 2 * N * VP;                                  // [2][L][VP]: the weighted values, the same way
  bf16* Mh = Wh + 2 * L * VP;                                  // [2][L][LP]: the decayed scores, the same way
  float* gates = reinterpret_cast<float*>(Mh + 2 * L * LP);    // [2][4][L]: c_t, d_t, exp(c_last - c_t) d_t, exp(c_t)
  pdl_trigger();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t2 = (lane & 3) * 2;
  const int head = blockIdx.x / p.v_tiles, col0 = (blockIdx.x % p.v_tiles) * VT;
  const int* it = p.items + 3 * blockIdx.y;
  const int begin = it[0], end = it[1];
  const float bias = p.step_bias[head], rate = -expf(p.rate_log[head]);
  const bf16* kx = p.x + p.k_off + (size_t)(head / p.share) * N;
  const bf16* qx = p.x + p.q_off + (size_t)(head / p.share) * N;
  const bf16* vx = p.x + p.v_off + (size_t)head * p.V + col0;
  const int v_left = p.V - col0;                               // columns of this tile that exist
  pdl_wait();
  float* st = p.state + (size_t)p.slot_ids[it[2]] * p.slot_floats + (size_t)head * N * p.V + col0;

  auto fetch = [&](int chunk) {
    const int t0 = begin + chunk * L, buf = chunk & 1;
    for (int i = tid; i < L * (N / 8); i += SS_THREADS) {
      const int r = i / (N / 8), c = (i % (N / 8)) * 8;
      const bool ok = t0 + r < end;
      const size_t row = (size_t)(ok ? t0 + r : begin) * p.x_stride;
      cp_async16(Ks + (buf * L + r) * NP + c, kx + row + c, ok);
    }
    for (int i = tid; i < L * (VT / 8); i += SS_THREADS) {
      const int r = i / (VT / 8), c = (i % (VT / 8)) * 8;
      const bool ok = t0 + r < end && c < v_left;
      cp_async16(Vs + (buf * L + r) * VP + c, ok ? vx + (size_t)(t0 + r) * p.x_stride + c : vx + (size_t)begin * p.x_stride, ok);
    }
    cp_async_commit();
  };
  auto fetch_q = [&](int chunk) {
    const int t0 = begin + chunk * L;
    for (int i = tid; i < L * (N / 8); i += SS_THREADS) {
      const int r = i / (N / 8), c = (i % (N / 8)) * 8;
      const bool ok = t0 + r < end;
      cp_async16(Qs + r * NP + c, qx + (size_t)(ok ? t0 + r : begin) * p.x_stride + c, ok);
    }
    cp_async_commit();
  };
  // one warp: a chunk's gates from its raw steps, two consecutive tokens a lane (tokens behind the end: step 0)
  auto load_z = [&](int chunk, float (&z)[2]) {
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = begin + chunk * L + 2 * lane + e;
      z[e] = t < end ? p.z[(size_t)t * p.H + head] : 0.f;
    }
  };
  auto make_gates = [&](int chunk, const float (&z)[2]) {
    float* gt = gates + (chunk & 1) * 4 * L;
    float d[2], l[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const float a = z[e] + bias;
      d[e] = begin + chunk * L + 2 * lane + e < end ? fmaxf(a, 0.f) + log1pf(expf(-fabsf(a))) : 0.f;
      l[e] = rate * d[e];
    }
    float pair = l[0] + l[1], sum = pair;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float before = __shfl_up_sync(0xffffffffu, sum, o);
      if (lane >= o) sum += before;
    }
    const float last = __shfl_sync(0xffffffffu, sum, 31);
    const float c[2] = {sum - l[1], sum};
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = 2 * lane + e;
      gt[t] = c[e];
      gt[L + t] = d[e];
      gt[2 * L + t] = expf(last - c[e]) * d[e];
      gt[3 * L + t] = expf(c[e]);
    }
  };

  // this warp's part of S as accumulators
  const int s_row = (warp % KT) * 16, s_col = (warp / KT) * ST * 8;
  float S[ST][4];
#pragma unroll
  for (int i = 0; i < ST; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int r = s_row + g + (e >> 1) * 8, c = s_col + i * 8 + t2 + (e & 1);
      S[i][e] = c < v_left ? st[(size_t)r * p.V + c] : 0.f;
    }
  // this warp's outputs: 16 tokens, OT tiles of 8 columns; it shares the scores of those tokens with one other warp.  The
  // last tokens see the most: their warps are on different schedulers
  const int o_half = warp >> 2, o_tile = o_half ? 3 - (warp & 3) : (warp & 3);
  const int o_col = o_half * OT * 8;
  const bool gate_warp = o_tile == 0 && o_half == 1;           // has no tile of scores

  const int chunks = (end - begin + L - 1) / L;
  fetch(0);
  fetch_q(0);
  float z_next[2] = {0.f, 0.f};
  if (gate_warp) {
    load_z(0, z_next);
    make_gates(0, z_next);
    if (chunks > 1) load_z(1, z_next);
  }
  for (int chunk = 0; chunk < chunks; ++chunk) {
    const int buf = chunk & 1;
    cp_async_wait<0>();
    __syncthreads();                          // the chunk's rows and gates are in; the chunk before has been read out
    if (chunk + 1 < chunks) fetch(chunk + 1);
    const float* gt = gates + buf * 4 * L;
    const bf16 *K = Ks + buf * L * NP, *X = Vs + buf * L * VP;
    unsigned qf[KT][4];
#pragma unroll
    for (int k = 0; k < KT; ++k) ldmatrix_x4(qf[k], Qs + (o_tile * 16 + (lane & 15)) * NP + k * 16 + (lane >> 4) * 8);
#pragma unroll
    for (int i = 0; i < ST; ++i)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const float a = S[i][2 * e], b = S[i][2 * e + 1];
        const __nv_bfloat162 hi = __floats2bfloat162_rn(a, b);
        const __nv_bfloat162 lo = __floats2bfloat162_rn(a - __low2float(hi), b - __high2float(hi));
        const int at = (s_row + g + e * 8) * VP + s_col + i * 8 + t2;
        *reinterpret_cast<__nv_bfloat162*>(Sh + at) = hi;
        *reinterpret_cast<__nv_bfloat162*>(Sh + N * VP + at) = lo;
      }
    for (int i = tid; i < L * (VT / 2); i += SS_THREADS) {
      const int r = i / (VT / 2), c = (i % (VT / 2)) * 2;
      const __nv_bfloat162 v = *reinterpret_cast<const __nv_bfloat162*>(X + r * VP + c);
      const float w = gt[2 * L + r], a = w * __low2float(v), b = w * __high2float(v);
      const __nv_bfloat162 hi = __floats2bfloat162_rn(a, b);
      *reinterpret_cast<__nv_bfloat162*>(Wh + r * VP + c) = hi;
      *reinterpret_cast<__nv_bfloat162*>(Wh + (L + r) * VP + c) = __floats2bfloat162_rn(a - __low2float(hi), b - __high2float(hi));
    }
    // ---- decayed scores: tiles o_half, o_half + 2 of the row's o_tile + 1
    const float c_row[2] = {gt[o_tile * 16 + g], gt[o_tile * 16 + g + 8]};
#pragma unroll
    for (int jj = 0; jj < 2; ++jj) {
      const int j = o_half + 2 * jj;
      if (j <= o_tile) {
        float sc[2][2][4];                    // even and odd k-steps apart: shorter chains of dependent products
#pragma unroll
        for (int a = 0; a < 2; ++a)
#pragma unroll
          for (int h = 0; h < 2; ++h)
#pragma unroll
            for (int e = 0; e < 4; ++e) sc[a][h][e] = 0.f;
#pragma unroll
        for (int k = 0; k < KT; ++k) {
          unsigned b[4];
          ldmatrix_x4(b, K + (j * 16 + (lane & 7) + ((lane >> 4) << 3)) * NP + k * 16 + ((lane >> 3) & 1) * 8);
          mma_bf16(sc[k & 1][0], qf[k], b[0], b[1]);
          mma_bf16(sc[k & 1][1], qf[k], b[2], b[3]);
        }
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int jc = j * 16 + h * 8 + t2;
          const float2 cj = *reinterpret_cast<const float2*>(gt + jc), dj = *reinterpret_cast<const float2*>(gt + L + jc);
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int row = o_tile * 16 + g + e * 8;
            const float s0 = sc[0][h][2 * e] + sc[1][h][2 * e], s1 = sc[0][h][2 * e + 1] + sc[1][h][2 * e + 1];
            const float a = jc <= row ? s0 * expf(c_row[e] - cj.x) * dj.x : 0.f;
            const float b = jc + 1 <= row ? s1 * expf(c_row[e] - cj.y) * dj.y : 0.f;
            const __nv_bfloat162 hi = __floats2bfloat162_rn(a, b);
            *reinterpret_cast<__nv_bfloat162*>(Mh + row * LP + jc) = hi;
            *reinterpret_cast<__nv_bfloat162*>(Mh + (L + row) * LP + jc) = __floats2bfloat162_rn(a - __low2float(hi), b - __high2float(hi));
          }
        }
      }
    }
    if (gate_warp && chunk + 1 < chunks) {
      make_gates(chunk + 1, z_next);
      if (chunk + 2 < chunks) load_z(chunk + 2, z_next);
    }
    __syncthreads();
    if (chunk + 1 < chunks) fetch_q(chunk + 1);

    // ---- outputs
    float y[2][OT][4], ys[2][OT][4];          // the rounded operands' sums and the rests' apart
#pragma unroll
    for (int a = 0; a < 2; ++a)
#pragma unroll
      for (int i = 0; i < OT; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) y[a][i][e] = ys[a][i][e] = 0.f;
#pragma unroll
    for (int k = 0; k < KT; ++k) {
#pragma unroll
      for (int i = 0; i < OT; ++i) {
        unsigned b[4];                        // the rounded S (two registers) and the rest (two registers) in one load
        ldmatrix_x4_trans(b, Sh + (lane >> 4) * N * VP + (k * 16 + (lane & 15)) * VP + o_col + i * 8);
        mma_bf16(ys[0][i], qf[k], b[0], b[1]);
        mma_bf16(ys[1][i], qf[k], b[2], b[3]);
      }
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      if (j <= o_tile) {
        unsigned mh[4], ml[4];
        ldmatrix_x4(mh, Mh + (o_tile * 16 + (lane & 15)) * LP + j * 16 + (lane >> 4) * 8);
        ldmatrix_x4(ml, Mh + (L + o_tile * 16 + (lane & 15)) * LP + j * 16 + (lane >> 4) * 8);
#pragma unroll
        for (int i = 0; i < OT; ++i) {
          unsigned b[2];
          ldmatrix_x2_trans(b, X + (j * 16 + (lane & 15)) * VP + o_col + i * 8);
          mma_bf16(y[0][i], mh, b[0], b[1]);
          mma_bf16(y[1][i], ml, b[0], b[1]);
        }
      }
    }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = o_tile * 16 + g + e * 8, tok = begin + chunk * L + t;
      const float carry = gt[3 * L + t];
      if (tok < end) {
        float* o = p.o + ((size_t)tok * p.H + head) * p.V + col0;
#pragma unroll
        for (int i = 0; i < OT; ++i) {
          const int c = o_col + i * 8 + t2;
          if (c < v_left)
            *reinterpret_cast<float2*>(o + c) =
                make_float2(fmaf(carry, ys[0][i][2 * e] + ys[1][i][2 * e], y[0][i][2 * e] + y[1][i][2 * e]),
                            fmaf(carry, ys[0][i][2 * e + 1] + ys[1][i][2 * e + 1], y[0][i][2 * e + 1] + y[1][i][2 * e + 1]));
        }
      }
    }

    // ---- the state behind the chunk
    const float keep = gt[3 * L + L - 1];
#pragma unroll
    for (int i = 0; i < ST; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) S[i][e] *= keep;
#pragma unroll
    for (int k = 0; k < L / 16; ++k) {
      unsigned a[4];
      ldmatrix_x4_trans(a, K + (k * 16 + (lane & 7) + (lane >> 4) * 8) * NP + s_row + ((lane >> 3) & 1) * 8);
#pragma unroll
      for (int i = 0; i < ST; ++i) {
        unsigned b[4];
        ldmatrix_x4_trans(b, Wh + (lane >> 4) * L * VP + (k * 16 + (lane & 15)) * VP + s_col + i * 8);
        mma_bf16(S[i], a, b[0], b[1]);
        mma_bf16(S[i], a, b[2], b[3]);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < ST; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int r = s_row + g + (e >> 1) * 8, c = s_col + i * 8 + t2 + (e & 1);
      if (c < v_left) st[(size_t)r * p.V + c] = S[i][e];
    }
}

template <int N, int VT>
static int state_space_shape(StateSpaceArgs p, int n_items, cudaStream_t stream) {
  const size_t smem = (size_t)(3 * SS_TOKENS * (N + 8) + (2 * SS_TOKENS + 2 * N + 2 * SS_TOKENS) * (VT + 8) + 2 * SS_TOKENS * (SS_TOKENS + 8)) * sizeof(bf16) + 8 * SS_TOKENS * sizeof(float);
  const cudaError_t e = cudaFuncSetAttribute(state_space_kernel<N, VT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return (int)e;
  p.v_tiles = (p.V + VT - 1) / VT;
  launch(state_space_kernel<N, VT>, dim3(p.H * p.v_tiles, n_items), dim3(SS_THREADS), smem, stream, p);
  return launch_status();
}

// Runs (`items`, three ints each) of bfloat16 rows.  N is 32, 64 or 128; V a multiple of 8; every row and offset starts on
// a 16-byte boundary.
Q25_EXPORT int q25_state_space_bf16(const void* x, int x_stride, int q_off, int k_off, int v_off, const float* z, const float* step_bias,
                                    const float* rate_log, float* state, long long slot_floats, const int* slot_ids, const int* items, int n_items,
                                    float* o, int H, int groups, int N, int V, void* stream) {
  if (n_items <= 0) return 0;
  if (H <= 0 || groups <= 0 || H % groups || V <= 0 || V % 8 || x_stride % 8 || q_off % 8 || k_off % 8 || v_off % 8 || ((uintptr_t)x & 15) ||
      ((uintptr_t)o & 7) || n_items > 65535)
    return (int)cudaErrorInvalidValue;
  StateSpaceArgs p;
  p.x = (const bf16*)x; p.x_stride = x_stride; p.q_off = q_off; p.k_off = k_off; p.v_off = v_off; p.z = z; p.step_bias = step_bias;
  p.rate_log = rate_log; p.state = state; p.slot_floats = (size_t)slot_floats; p.slot_ids = slot_ids; p.items = items; p.o = o; p.H = H; p.V = V;
  p.share = H / groups; p.v_tiles = 0;
  cudaStream_t s = (cudaStream_t)stream;
  // narrower column tiles while those, too, all run at once (two CTAs to an SM)
  const int sms = device_sm_count() > 0 ? device_sm_count() : 148;
  const bool narrow = (long long)H * ((V + 15) / 16) * n_items <= 2ll * sms || V <= 16;
  switch (N) {
    case 32: return state_space_shape<32, 32>(p, n_items, s);
    case 64: return narrow ? state_space_shape<64, 16>(p, n_items, s) : state_space_shape<64, 32>(p, n_items, s);
    case 128: return narrow ? state_space_shape<128, 16>(p, n_items, s) : state_space_shape<128, 32>(p, n_items, s);
    default: return (int)cudaErrorInvalidValue;
  }
}
