// Kernels of the gated linear recurrent mixer (Griffin's recurrent block with a real-gated linear
// recurrent unit, RG-LRU).  Per channel c of the mixer's width W, for the tokens of one request in
// order:
//
//   u_t   = sum_j conv[c, j] * xin_(t - (taps-1) + j) + conv_b[c]        causal, zeros before the start
//   r_t   = sigmoid(Ra[b] u_t,b + ra_b),  i_t = sigmoid(Ri[b] u_t,b + ri_b)   per block b of W / blocks channels
//   log a = -gain * r_t * softplus(lam[c]),  a_t = exp(log a)
//   S_t   = a_t S_(t-1) + sqrt(1 - a_t^2) * i_t * u_t                     S_(-1) = 0
//   out_t = S_t * gelu_tanh(ybranch_t)
//
// xin and ybranch are the two halves of one projection (activation dtype T); everything from u on
// is float: the gates' products are sums over the block's channels in an order that the block's size alone decides, so
// a token's gates do not depend on the batch, and the state S is carried in float from step to step.
//
// Per-request state [slots, taps, W] float: row 0 is S, rows 1 .. taps-1 are the last taps-1 inputs
// xin of the request, oldest first (zeros at admission, which are the zeros before the start).
//
// The kernels: the convolution, which moves its inputs on (it also serves mixers that keep other state beside
// them); the two gates of all blocks as one batched product with the decay and the input term formed in its
// epilogue (float FMAs; for long steps whose gate matrices are bfloat16 numbers, tensor cores with u as a sum of
// three bfloat16 numbers); the scan in chunks over time, which moves S on.
#include "mma.cuh"

#define RG_MAX_TAPS 16

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// Both gates of every block: for block b (blockIdx.z), rows = tokens, columns = the block's
// channels; two FMA chains per element over the block's input channels in order.  Epilogue:
// a = exp(-gain * sigmoid(ga) * softplus(lam)), bx = sqrt(1 - a^2) * sigmoid(gi) * u.
template <int BM, int BN, int BK, int TM, int TN>
__global__ void __launch_bounds__((BM / TM) * (BN / TN))
rglru_gates_kernel(const float* __restrict__ u, const float* __restrict__ ra, const float* __restrict__ ra_b,
                   const float* __restrict__ ri, const float* __restrict__ ri_b, const float* __restrict__ lam,
                   float gain, float* __restrict__ a_out, float* __restrict__ bx_out, int n_tokens, int width, int bw) {
  pdl_trigger();
  pdl_wait();
  constexpr int THREADS = (BM / TM) * (BN / TN);
  __shared__ float Us[BK][BM + 4];
  __shared__ float As[BK][BN + 4];
  __shared__ float Is[BK][BN + 4];
  const int b = blockIdx.z;
  const int tx = threadIdx.x % (BN / TN), ty = threadIdx.x / (BN / TN);
  const int m0 = blockIdx.y * BM, n0 = blockIdx.x * BN;
  const float* Wa = ra + (size_t)b * bw * bw;
  const float* Wi = ri + (size_t)b * bw * bw;
  float acc_a[TM][TN], acc_i[TM][TN];
#pragma unroll
  for (int i = 0; i < TM; ++i)
#pragma unroll
    for (int j = 0; j < TN; ++j) acc_a[i][j] = acc_i[i][j] = 0.f;
  for (int k0 = 0; k0 < bw; k0 += BK) {
    for (int e = threadIdx.x; e < BM * BK; e += THREADS) {
      const int r = e / BK, c = e % BK;
      const int gm = m0 + r, gk = k0 + c;
      Us[c][r] = (gm < n_tokens && gk < bw) ? u[(size_t)gm * width + b * bw + gk] : 0.f;
    }
    for (int e = threadIdx.x; e < BN * BK; e += THREADS) {
      const int r = e / BK, c = e % BK;
      const int gn = n0 + r, gk = k0 + c;
      const bool ok = gn < bw && gk < bw;
      As[c][r] = ok ? Wa[(size_t)gn * bw + gk] : 0.f;
      Is[c][r] = ok ? Wi[(size_t)gn * bw + gk] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < BK; ++kk) {
      float uu[TM], wa[TN], wi[TN];
#pragma unroll
      for (int i = 0; i < TM; ++i) uu[i] = Us[kk][ty * TM + i];
#pragma unroll
      for (int j = 0; j < TN; ++j) { wa[j] = As[kk][tx * TN + j]; wi[j] = Is[kk][tx * TN + j]; }
#pragma unroll
      for (int i = 0; i < TM; ++i)
#pragma unroll
        for (int j = 0; j < TN; ++j) {
          acc_a[i][j] = fmaf(uu[i], wa[j], acc_a[i][j]);
          acc_i[i][j] = fmaf(uu[i], wi[j], acc_i[i][j]);
        }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < TM; ++i) {
    const int gm = m0 + ty * TM + i;
    if (gm >= n_tokens) continue;
#pragma unroll
    for (int j = 0; j < TN; ++j) {
      const int gn = n0 + tx * TN + j;
      if (gn >= bw) continue;
      const int c = b * bw + gn;
      const float r = sigmoid_f(acc_a[i][j] + ra_b[c]);
      const float g = sigmoid_f(acc_i[i][j] + ri_b[c]);
      const float log_a = -gain * r * softplus_f(lam[c]);
      const size_t at = (size_t)gm * width + c;
      a_out[at] = expf(log_a);
      bx_out[at] = sqrtf(-expm1f(2.0f * log_a)) * g * u[at];
    }
  }
}

// The same for steps of few tokens (decode): a CTA takes 16 tokens x 16 channels of one block and
// brings the whole depth of the product into shared memory at once, so that all its loads are in
// flight together instead of a chain of tiles; one thread per (token, channel), the same FMA chains
// in the same order as above.  Dynamic shared memory: 3 x bw x 17 floats.
__global__ void __launch_bounds__(256)
rglru_gates_small_kernel(const float* __restrict__ u, const float* __restrict__ ra, const float* __restrict__ ra_b,
                         const float* __restrict__ ri, const float* __restrict__ ri_b, const float* __restrict__ lam,
                         float gain, float* __restrict__ a_out, float* __restrict__ bx_out, int n_tokens, int width, int bw) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ float gates_smem[];
  float* Us = gates_smem;                  // [bw][17]
  float* As = Us + (size_t)bw * 17;
  float* Is = As + (size_t)bw * 17;
  const int b = blockIdx.z, m0 = blockIdx.y * 16, n0 = blockIdx.x * 16;
  const float* Wa = ra + (size_t)b * bw * bw;
  const float* Wi = ri + (size_t)b * bw * bw;
  for (int e = threadIdx.x; e < 16 * bw; e += 256) {
    const int r = e / bw, k = e % bw;                     // consecutive threads read consecutive k
    const int gm = m0 + r, gn = n0 + r;
    Us[k * 17 + r] = gm < n_tokens ? u[(size_t)gm * width + b * bw + k] : 0.f;
    As[k * 17 + r] = gn < bw ? Wa[(size_t)gn * bw + k] : 0.f;
    Is[k * 17 + r] = gn < bw ? Wi[(size_t)gn * bw + k] : 0.f;
  }
  __syncthreads();
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc_a = 0.f, acc_i = 0.f;
  for (int k = 0; k < bw; ++k) {
    const float uu = Us[k * 17 + ty];
    acc_a = fmaf(uu, As[k * 17 + tx], acc_a);
    acc_i = fmaf(uu, Is[k * 17 + tx], acc_i);
  }
  const int gm = m0 + ty, gn = n0 + tx;
  if (gm >= n_tokens || gn >= bw) return;
  const int c = b * bw + gn;
  const float r = sigmoid_f(acc_a + ra_b[c]);
  const float g = sigmoid_f(acc_i + ri_b[c]);
  const float log_a = -gain * r * softplus_f(lam[c]);
  const size_t at = (size_t)gm * width + c;
  a_out[at] = expf(log_a);
  bx_out[at] = sqrtf(-expm1f(2.0f * log_a)) * g * u[at];
}

// Both gates for long steps on tensor cores (mma.sync, float accumulators), for gate matrices whose entries are bfloat16
// numbers.  u is float: it enters as the sum of three bfloat16 numbers (the rounded value, what the rounding left,
// rounded, and what that left), which is u itself to 24 bits, in three products each; so the sums are float sums of
// exact products, as in the kernels above.  A CTA takes 64 tokens x 64 channels of one block; warp (m, h) 16 tokens x
// 32 channels of both gates.
#define RGM_K 64
#define RGM_P (RGM_K + 8)

__global__ void __launch_bounds__(256)
rglru_gates_mma_kernel(const float* __restrict__ u, const bf16* __restrict__ ra, const float* __restrict__ ra_b, const bf16* __restrict__ ri,
                       const float* __restrict__ ri_b, const float* __restrict__ lam, float gain, float* __restrict__ a_out,
                       float* __restrict__ bx_out, int n_tokens, int width, int bw) {
  pdl_trigger();
  __shared__ __align__(16) bf16 Us[3][64][RGM_P];
  __shared__ __align__(16) bf16 Ws[2][64][RGM_P];
  const int b = blockIdx.z, m0 = blockIdx.y * 64, n0 = blockIdx.x * 64;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, wm = (warp & 3) * 16, wn = (warp >> 2) * 32;
  float acc[2][4][4];
#pragma unroll
  for (int g = 0; g < 2; ++g)
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[g][i][e] = 0.f;
  pdl_wait();
  for (int k0 = 0; k0 < bw; k0 += RGM_K) {
    for (int i = tid; i < 2 * 64 * (RGM_K / 8); i += 256) {
      const int gate = i / (64 * (RGM_K / 8)), r = i / (RGM_K / 8) % 64, c = (i % (RGM_K / 8)) * 8;
      const bool ok = n0 + r < bw && k0 + c < bw;
      const bf16* src = (gate ? ri : ra) + (size_t)b * bw * bw;
      cp_async16(&Ws[gate][r][c], ok ? src + (size_t)(n0 + r) * bw + k0 + c : src, ok);
    }
    cp_async_commit();
    for (int i = tid; i < 64 * (RGM_K / 4); i += 256) {
      const int r = i / (RGM_K / 4), c = (i % (RGM_K / 4)) * 4;
      const bool ok = m0 + r < n_tokens && k0 + c < bw;
      float4 v = ok ? *reinterpret_cast<const float4*>(u + (size_t)(m0 + r) * width + (size_t)b * bw + k0 + c) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int part = 0; part < 3; ++part) {
        store4<bf16>(&Us[part][r][c], v);
        const float4 took = load4<bf16>(&Us[part][r][c]);
        v.x -= took.x; v.y -= took.y; v.z -= took.z; v.w -= took.w;
      }
    }
    cp_async_wait<0>();
    __syncthreads();
#pragma unroll
    for (int k = 0; k < RGM_K / 16; ++k) {
      unsigned a[3][4];
#pragma unroll
      for (int part = 0; part < 3; ++part) ldmatrix_x4(a[part], &Us[part][wm + (lane & 15)][k * 16 + (lane >> 4) * 8]);
#pragma unroll
      for (int g = 0; g < 2; ++g)
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          unsigned w[4];
          ldmatrix_x4(w, &Ws[g][wn + i * 16 + (lane & 7) + ((lane >> 4) << 3)][k * 16 + ((lane >> 3) & 1) * 8]);
#pragma unroll
          for (int part = 2; part >= 0; --part) {
            mma_bf16(acc[g][2 * i], a[part], w[0], w[1]);
            mma_bf16(acc[g][2 * i + 1], a[part], w[2], w[3]);
          }
        }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int gn = n0 + wn + i * 8 + (lane & 3) * 2;
    if (gn >= bw) continue;
    const int c = b * bw + gn;
    const float sp[2] = {softplus_f(lam[c]), softplus_f(lam[c + 1])};
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int gm = m0 + wm + (lane >> 2) + e * 8;
      if (gm >= n_tokens) continue;
      const size_t at = (size_t)gm * width + c;
      const float2 uu = *reinterpret_cast<const float2*>(u + at);
      float av[2], bv[2];
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        const float r = sigmoid_f(acc[0][i][2 * e + q] + ra_b[c + q]), g = sigmoid_f(acc[1][i][2 * e + q] + ri_b[c + q]);
        const float log_a = -gain * r * sp[q];
        av[q] = expf(log_a);
        bv[q] = sqrtf(-expm1f(2.0f * log_a)) * g * (q ? uu.y : uu.x);
      }
      *reinterpret_cast<float2*>(a_out + at) = make_float2(av[0], av[1]);
      *reinterpret_cast<float2*>(bx_out + at) = make_float2(bv[0], bv[1]);
    }
  }
}

__device__ __forceinline__ float gelu_tanh_f(float z) {
  return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

// The scan S_t = a_t S_(t-1) + bx_t over an entry's tokens, cut into chunks of RG_CHUNK tokens so
// that long prompts run in parallel over time as well as over channels.
//   rglru_chunk_kernel: one thread per (entry, chunk, channel) folds its chunk into (A, B) with
//     S_end = A S_start + B (A the product of the decays, B the chunk's own sum from zero); the
//     thread of chunk 0 also copies the request's S aside, so that the next kernel never reads the
//     place it writes.
//   rglru_scan_kernel: one thread per (entry, chunk, channel) folds the summaries of the chunks
//     before its own onto the request's S (a short chain of FMAs over values that all chunks of
//     the entry read, so they stay in cache), then runs its chunk and writes out = S * gelu_tanh(y).
//     The thread of the last chunk moves S on.
// A step whose entries all have up to RG_CHUNK tokens (every decode step) runs the second kernel
// alone: one chunk per entry, S read from the state itself.
// sums: [n_seqs, max_chunks, 2, width] (A, B), then [n_seqs, width] (the requests' S before the step).
#define RG_CHUNK 32

__global__ void rglru_chunk_kernel(const float* __restrict__ a, const float* __restrict__ bx, const float* __restrict__ state,
                                   const int* __restrict__ cu_q, const int* __restrict__ slot_ids, float* __restrict__ sums,
                                   int n_seqs, int width, int taps, int max_chunks) {
  pdl_trigger();
  pdl_wait();
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  const int seq = blockIdx.y, chunk = blockIdx.z;
  const int first = cu_q[seq], n = cu_q[seq + 1] - first;
  if (c >= width || chunk * RG_CHUNK >= n) return;
  if (chunk == 0) sums[(size_t)n_seqs * max_chunks * 2 * width + (size_t)seq * width + c] = state[(size_t)slot_ids[seq] * taps * width + c];
  const int t0 = chunk * RG_CHUNK, t1 = min(n, t0 + RG_CHUNK);
  float A = 1.f, B = 0.f;
#pragma unroll 8
  for (int t = t0; t < t1; ++t) {
    const size_t at = (size_t)(first + t) * width + c;
    const float av = a[at];
    A *= av;
    B = fmaf(av, B, bx[at]);
  }
  const size_t to = ((size_t)seq * max_chunks + chunk) * 2 * width + c;
  sums[to] = A;
  sums[to + width] = B;
}

template <typename T>
__global__ void rglru_scan_kernel(const float* __restrict__ a, const float* __restrict__ bx, const T* __restrict__ yx, int ld,
                                  int y_off, float* __restrict__ state, const int* __restrict__ cu_q,
                                  const int* __restrict__ slot_ids, T* __restrict__ out, const float* __restrict__ sums,
                                  int n_seqs, int width, int taps, int max_chunks) {
  pdl_trigger();
  pdl_wait();
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  const int seq = blockIdx.y, chunk = blockIdx.z;
  const int first = cu_q[seq], n = cu_q[seq + 1] - first;
  if (c >= width || chunk * RG_CHUNK >= n) return;
  float* st = state + (size_t)slot_ids[seq] * taps * width + c;
  float S = sums ? sums[(size_t)n_seqs * max_chunks * 2 * width + (size_t)seq * width + c] : st[0];
#pragma unroll 8
  for (int j = 0; j < chunk; ++j) {
    const size_t at = ((size_t)seq * max_chunks + j) * 2 * width + c;
    S = fmaf(sums[at], S, sums[at + width]);
  }
  const int t0 = chunk * RG_CHUNK, t1 = min(n, t0 + RG_CHUNK);
#pragma unroll 8
  for (int t = t0; t < t1; ++t) {
    const size_t at = (size_t)(first + t) * width + c;
    S = fmaf(a[at], S, bx[at]);
    out[at] = from_f32<T>(S * gelu_tanh_f(to_f32(yx[(size_t)(first + t) * ld + y_off + c])));
  }
  if (t1 < n) return;                          // the last chunk's thread moves the state on; nobody else reads it here
  st[0] = S;
}

// Floats of scratch memory the scan needs for a step whose longest entry has max_q_len tokens (0: none).
Q25_EXPORT long long q25_rglru_scan_scratch_floats(int n_seqs, int max_q_len, int width) {
  const int max_chunks = (max_q_len + RG_CHUNK - 1) / RG_CHUNK;
  return max_chunks <= 1 ? 0 : (long long)n_seqs * width * (2 * max_chunks + 1);
}

template <typename T>
static int rglru_scan(const float* a, const float* bx, const void* yx, int ld, int y_off, float* state, const int* cu_q,
                      const int* slot_ids, void* out, int n_seqs, int max_q_len, float* sums, int width, int taps, void* stream) {
  if (n_seqs <= 0) return 0;
  if (taps < 1 || taps > RG_MAX_TAPS || max_q_len < 1) return (int)cudaErrorInvalidValue;
  const int max_chunks = (max_q_len + RG_CHUNK - 1) / RG_CHUNK;
  if (max_chunks > 65535 || (max_chunks > 1 && !sums)) return (int)cudaErrorInvalidValue;
  const dim3 grid((width + 127) / 128, n_seqs, max_chunks);
  if (max_chunks > 1)
    launch(rglru_chunk_kernel, grid, dim3(128), 0, (cudaStream_t)stream, a, bx, (const float*)state, cu_q, slot_ids, sums, n_seqs, width,
           taps, max_chunks);
  launch(rglru_scan_kernel<T>, grid, dim3(128), 0, (cudaStream_t)stream, a, bx, (const T*)yx, ld, y_off, state, cu_q, slot_ids,
         (T*)out, (const float*)(max_chunks > 1 ? sums : nullptr), n_seqs, width, taps, max_chunks);
  return launch_status();
}

Q25_EXPORT int q25_rglru_gates(const float* u, const float* ra, const float* ra_b, const float* ri, const float* ri_b,
                               const float* lam, float gain, float* a_out, float* bx_out, int n_tokens, int width, int blocks,
                               void* stream) {
  if (n_tokens <= 0) return 0;
  if (blocks <= 0 || width % blocks) return (int)cudaErrorInvalidValue;
  const int bw = width / blocks;
  const size_t small_smem = (size_t)3 * bw * 17 * sizeof(float);
  if (n_tokens <= 128 && small_smem <= 160 * 1024) {
    if (small_smem > 48 * 1024) {
      const cudaError_t e = cudaFuncSetAttribute(rglru_gates_small_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)small_smem);
      if (e != cudaSuccess) return (int)e;
    }
    launch(rglru_gates_small_kernel, dim3((bw + 15) / 16, (n_tokens + 15) / 16, blocks), dim3(256), small_smem, (cudaStream_t)stream, u, ra,
           ra_b, ri, ri_b, lam, gain, a_out, bx_out, n_tokens, width, bw);
  } else if (n_tokens <= 16) {
    launch(rglru_gates_kernel<16, 64, 16, 1, 4>, dim3((bw + 63) / 64, (n_tokens + 15) / 16, blocks), dim3(256), 0, (cudaStream_t)stream,
           u, ra, ra_b, ri, ri_b, lam, gain, a_out, bx_out, n_tokens, width, bw);
  } else {
    launch(rglru_gates_kernel<64, 64, 16, 4, 4>, dim3((bw + 63) / 64, (n_tokens + 63) / 64, blocks), dim3(256), 0, (cudaStream_t)stream,
           u, ra, ra_b, ri, ri_b, lam, gain, a_out, bx_out, n_tokens, width, bw);
  }
  return launch_status();
}
// The same with bfloat16 gate matrices; the blocks' width is a multiple of 8.
Q25_EXPORT int q25_rglru_gates_mma(const float* u, const void* ra, const float* ra_b, const void* ri, const float* ri_b, const float* lam, float gain,
                                   float* a_out, float* bx_out, int n_tokens, int width, int blocks, void* stream) {
  if (n_tokens <= 0) return 0;
  if (blocks <= 0 || width % blocks || (width / blocks) % 8 || (((uintptr_t)u | (uintptr_t)ra | (uintptr_t)ri | (uintptr_t)a_out | (uintptr_t)bx_out) & 15))
    return (int)cudaErrorInvalidValue;
  const int bw = width / blocks;
  launch(rglru_gates_mma_kernel, dim3((bw + 63) / 64, (n_tokens + 63) / 64, blocks), dim3(256), 0, (cudaStream_t)stream, u, (const bf16*)ra, ra_b,
         (const bf16*)ri, ri_b, lam, gain, a_out, bx_out, n_tokens, width, bw);
  return launch_status();
}
Q25_EXPORT int q25_rglru_scan_f32(const float* a, const float* bx, const void* yx, int ld, int yo, float* st, const int* cu,
                                  const int* sl, void* out, int n_seqs, int max_q_len, float* sums, int w, int taps, void* s) {
  return rglru_scan<float>(a, bx, yx, ld, yo, st, cu, sl, out, n_seqs, max_q_len, sums, w, taps, s);
}
Q25_EXPORT int q25_rglru_scan_bf16(const float* a, const float* bx, const void* yx, int ld, int yo, float* st, const int* cu,
                                   const int* sl, void* out, int n_seqs, int max_q_len, float* sums, int w, int taps, void* s) {
  return rglru_scan<bf16>(a, bx, yx, ld, yo, st, cu, sl, out, n_seqs, max_q_len, sums, w, taps, s);
}

// ---- the causal convolution per channel ----------------------------------------------------------------
// out[n, c] = act(bias[c] + sum_j w[j, c] in_(t - (taps - 1) + j)[c]), the inputs before the step's first token from the
// request's history [taps - 1, channels] (floats at state + slot * slot_floats, oldest first; zeros at admission), which
// moves on.  A thread owns V channels of CONV_TOKENS consecutive tokens of an entry and slides a window over the inputs,
// so an input is read once (and taps - 1 of them again per piece); the piece that holds the entry's first token is the
// only reader of the history and writes the new one.  TO: the result's dtype.  WIN: taps rounded up to a built size; the window's older places
// carry weights of zero.
#define CONV_TOKENS 16
#define CONV_AHEAD 8         // inputs a thread asks for at once

template <typename T, int V> __device__ __forceinline__ void conv_load(const T* p, float (&v)[V]) {
  if constexpr (V == 4) {
    const float4 a = load4<T>(p);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
  } else {
    v[0] = to_f32(p[0]);
  }
}
template <typename T, int V> __device__ __forceinline__ void conv_store(T* p, const float (&v)[V]) {
  if constexpr (V == 4) store4<T>(p, make_float4(v[0], v[1], v[2], v[3]));
  else p[0] = from_f32<T>(v[0]);
}

template <typename T, typename TO, int WIN, int V>
__global__ void __launch_bounds__(128)
causal_conv_kernel(const T* __restrict__ in, int in_stride, const float* __restrict__ w, const float* __restrict__ bias, float* __restrict__ state,
                   size_t slot_floats, const int* __restrict__ cu_q, const int* __restrict__ slot_ids, TO* __restrict__ out, int out_stride,
                   int channels, int taps, int silu) {
  pdl_trigger();
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
  float wt[WIN][V], b[V];
  if (c < channels) {                          // weights: no kernel ever writes them
#pragma unroll
    for (int j = 0; j < WIN; ++j) {
#pragma unroll
      for (int v = 0; v < V; ++v) wt[j][v] = 0.f;
      if (j >= WIN - taps) conv_load<float, V>(w + (size_t)(j - (WIN - taps)) * channels + c, wt[j]);
    }
    conv_load<float, V>(bias + c, b);
  }
  pdl_wait();
  const int seq = blockIdx.y, piece = blockIdx.z;
  const int first = cu_q[seq], n = cu_q[seq + 1] - first;
  const int t0 = piece * CONV_TOKENS;
  if (c >= channels || t0 >= n) return;
  const int t1 = min(n, t0 + CONV_TOKENS);
  const T* x = in + (size_t)first * in_stride + c;
  TO* o = out + (size_t)first * out_stride + c;
  float* hist = state + (size_t)slot_ids[seq] * slot_floats + c;
  float win[WIN][V];                           // the last WIN inputs, the newest last
#pragma unroll
  for (int j = 0; j < WIN; ++j)
#pragma unroll
    for (int v = 0; v < V; ++v) win[j][v] = 0.f;
  // places 1 .. WIN - 1 before the first token (they move down by one when it comes in)
#pragma unroll
  for (int j = 1; j < WIN; ++j) {
    const int rel = t0 - WIN + j;
    if (j > WIN - taps) {
      if (rel >= 0) conv_load<T, V>(x + (size_t)rel * in_stride, win[j]);
      else if (piece == 0) {
#pragma unroll
        for (int v = 0; v < V; ++v) win[j][v] = hist[(size_t)(taps - 1 + rel) * channels + v];
      }
    }
  }
  if (piece == 0) {
    // the new history: the last taps - 1 of (old history, this entry's inputs).  The old rows are in the window; a row
    // is written after the rows it may come from have been read
    float keep[WIN > 1 ? WIN - 1 : 1][V];
#pragma unroll
    for (int j = 1; j < WIN; ++j) {
      const int rel = n - WIN + j;             // the input this row will hold, by its place in the entry
#pragma unroll
      for (int v = 0; v < V; ++v) keep[j - 1][v] = 0.f;
      if (j > WIN - taps) {
        if (rel >= 0) conv_load<T, V>(x + (size_t)rel * in_stride, keep[j - 1]);
        else {
#pragma unroll
          for (int i = 1; i < WIN; ++i)
            if (i == rel + WIN) {
#pragma unroll
              for (int v = 0; v < V; ++v) keep[j - 1][v] = win[i][v];
            }
        }
      }
    }
#pragma unroll
    for (int j = 1; j < WIN; ++j)
      if (j > WIN - taps) {
#pragma unroll
        for (int v = 0; v < V; ++v) hist[(size_t)(j - 1 - (WIN - taps)) * channels + v] = keep[j - 1][v];
      }
  }
  for (int t = t0; t < t1; t += CONV_AHEAD) {
    float next[CONV_AHEAD][V];
#pragma unroll
    for (int a = 0; a < CONV_AHEAD; ++a) {
      const int tt = min(t + a, t1 - 1);
      conv_load<T, V>(x + (size_t)tt * in_stride, next[a]);
    }
#pragma unroll
    for (int a = 0; a < CONV_AHEAD; ++a) {
      if (t + a < t1) {
        float r[V];
#pragma unroll
        for (int v = 0; v < V; ++v) {
#pragma unroll
          for (int j = 0; j + 1 < WIN; ++j) win[j][v] = win[j + 1][v];
          win[WIN - 1][v] = next[a][v];
          float acc = 0.f;
#pragma unroll
          for (int j = 0; j < WIN; ++j) acc = fmaf(wt[j][v], win[j][v], acc);
          acc += b[v];
          r[v] = silu ? acc / (1.0f + expf(-acc)) : acc;
        }
        conv_store<TO, V>(o + (size_t)(t + a) * out_stride, r);
      }
    }
  }
}

template <typename T, typename TO>
static int causal_conv(const void* in, int in_stride, const float* w, const float* bias, float* state, long long slot_floats, const int* cu_q,
                       const int* slot_ids, void* out, int out_stride, int n_seqs, int max_q_len, int channels, int taps, int silu, void* stream) {
  if (n_seqs <= 0 || channels <= 0) return 0;
  if (taps < 1 || taps > RG_MAX_TAPS || max_q_len < 1 || (taps > 1 && !state)) return (int)cudaErrorInvalidValue;
  const int pieces = (max_q_len + CONV_TOKENS - 1) / CONV_TOKENS;
  if (pieces > 65535 || n_seqs > 65535) return (int)cudaErrorInvalidValue;
  const bool four = channels % 4 == 0 && in_stride % 4 == 0 && out_stride % 4 == 0 && !(((uintptr_t)w | (uintptr_t)bias) & 15) && !((uintptr_t)in % (4 * sizeof(T))) && !((uintptr_t)out % (4 * sizeof(TO)));
  const int threads_c = four ? channels / 4 : channels;
  const dim3 grid((threads_c + 127) / 128, n_seqs, pieces);
  void (*kernel)(const T*, int, const float*, const float*, float*, size_t, const int*, const int*, TO*, int, int, int, int) =
      taps <= 4 ? (four ? causal_conv_kernel<T, TO, 4, 4> : causal_conv_kernel<T, TO, 4, 1>)
                : (four ? causal_conv_kernel<T, TO, RG_MAX_TAPS, 4> : causal_conv_kernel<T, TO, RG_MAX_TAPS, 1>);
  launch(kernel, grid, dim3(128), 0, (cudaStream_t)stream, (const T*)in, in_stride, w, bias, state, (size_t)slot_floats, cu_q, slot_ids, (TO*)out,
         out_stride, channels, taps, silu);
  return launch_status();
}
Q25_EXPORT int q25_rglru_causal_conv_f32(const void* in, int is, const float* w, const float* b, float* st, long long sf, const int* cu, const int* sl,
                                         void* out, int os, int n_seqs, int max_q_len, int channels, int taps, int silu, int out_f32, void* s) {
  return causal_conv<float, float>(in, is, w, b, st, sf, cu, sl, out, os, n_seqs, max_q_len, channels, taps, silu, s);
}
Q25_EXPORT int q25_rglru_causal_conv_bf16(const void* in, int is, const float* w, const float* b, float* st, long long sf, const int* cu, const int* sl,
                                          void* out, int os, int n_seqs, int max_q_len, int channels, int taps, int silu, int out_f32, void* s) {
  return out_f32 ? causal_conv<bf16, float>(in, is, w, b, st, sf, cu, sl, out, os, n_seqs, max_q_len, channels, taps, silu, s)
                 : causal_conv<bf16, bf16>(in, is, w, b, st, sf, cu, sl, out, os, n_seqs, max_q_len, channels, taps, silu, s);
}
