// Hyper-connections: a residual stream that is `streams` rows per token, x [N, S, W] in float.  A sublayer reads the
// weighted sum u = sum_s in[s] x_s of a token's rows and its result y goes back into all of them at once,
//
//   x_t <- sum_s mix[s, t] x_s + out[t] y          (mix: [from, to]).
//
// One kernel per sublayer does what follows the sublayer before and what comes ahead of the next one: the update still
// pending (y in the activation dtype, with its own mix and out) is written into the rows, the next sublayer's sum is
// taken from the new rows, and its RMS norm's result leaves in the activation dtype:
//
//   h = u / sqrt(mean(u^2) + eps) * w
//
// A token's rows are read and written once.  With `row_ids` only those tokens are produced and x is left as it is (the
// model's last norm, which the wanted places alone need).  Everything but y and h is float; every sum has a fixed order.
#include "common.cuh"

#define HC_MAX_STREAMS 16

__device__ __forceinline__ float4 fma4(float s, float4 v, float4 acc) {
  return make_float4(fmaf(s, v.x, acc.x), fmaf(s, v.y, acc.y), fmaf(s, v.z, acc.z), fmaf(s, v.w, acc.w));
}

// STREAMS: their number, or 0 for any up to HC_MAX_STREAMS (`streams` says how many).  VEC: four channels at a time.
template <typename T, int STREAMS, bool VEC>
__global__ void __launch_bounds__(512)
hyper_norm_kernel(float* __restrict__ x, const T* __restrict__ y, const float* __restrict__ mix, const float* __restrict__ out_w,
                  const float* __restrict__ in_w, const float* __restrict__ w, float eps, T* __restrict__ h,
                  const int* __restrict__ row_ids, int streams, int width) {
  constexpr int CAP = STREAMS ? STREAMS : HC_MAX_STREAMS;
  const int S = STREAMS ? STREAMS : streams;
  extern __shared__ __align__(16) float hc_row[];        // width floats: u; then mix [S * S], out [S], in [S]
  float* mix_s = hc_row + ((width + 3) & ~3);
  float* out_s = mix_s + S * S;
  float* in_s = out_s + S;
  __shared__ float scratch[32];
  pdl_trigger();
  if (y)
    for (int i = threadIdx.x; i < S * S + S; i += blockDim.x) mix_s[i] = i < S * S ? mix[i] : out_w[i - S * S];
  for (int i = threadIdx.x; i < S; i += blockDim.x) in_s[i] = in_w ? in_w[i] : 1.f;
  pdl_wait();
  __syncthreads();
  const int r = blockIdx.x;
  const size_t row = row_ids ? row_ids[r] : r;
  float* xr = x + row * S * width;
  const T* yr = y ? y + row * width : nullptr;
  float ss = 0.f;
  if (VEC) {
    for (int c = threadIdx.x * 4; c < width; c += blockDim.x * 4) {
      float4 v[CAP];
      float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int s = 0; s < CAP; ++s)
        if (s < S) v[s] = *reinterpret_cast<const float4*>(xr + (size_t)s * width + c);
      if (yr) {
        const float4 d = load4<T>(yr + c);
#pragma unroll
        for (int t = 0; t < CAP; ++t) {
          if (t < S) {
            float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int s = 0; s < CAP; ++s)
              if (s < S) a = fma4(mix_s[s * S + t], v[s], a);
            a = fma4(out_s[t], d, a);
            if (!row_ids) *reinterpret_cast<float4*>(xr + (size_t)t * width + c) = a;
            u = fma4(in_s[t], a, u);
          }
        }
      } else {
#pragma unroll
        for (int s = 0; s < CAP; ++s)
          if (s < S) u = fma4(in_s[s], v[s], u);
      }
      *reinterpret_cast<float4*>(hc_row + c) = u;
      ss = fmaf(u.x, u.x, ss); ss = fmaf(u.y, u.y, ss); ss = fmaf(u.z, u.z, ss); ss = fmaf(u.w, u.w, ss);
    }
  } else {
    for (int c = threadIdx.x; c < width; c += blockDim.x) {
      float v[CAP];
      float u = 0.f;
#pragma unroll
      for (int s = 0; s < CAP; ++s)
        if (s < S) v[s] = xr[(size_t)s * width + c];
      if (yr) {
        const float d = to_f32(yr[c]);
#pragma unroll
        for (int t = 0; t < CAP; ++t) {
          if (t < S) {
            float a = 0.f;
#pragma unroll
            for (int s = 0; s < CAP; ++s)
              if (s < S) a = fmaf(mix_s[s * S + t], v[s], a);
            a = fmaf(out_s[t], d, a);
            if (!row_ids) xr[(size_t)t * width + c] = a;
            u = fmaf(in_s[t], a, u);
          }
        }
      } else {
#pragma unroll
        for (int s = 0; s < CAP; ++s)
          if (s < S) u = fmaf(in_s[s], v[s], u);
      }
      hc_row[c] = u;
      ss = fmaf(u, u, ss);
    }
  }
  const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)width + eps);
  T* o = h + (size_t)r * width;
  if (VEC) {
    for (int c = threadIdx.x * 4; c < width; c += blockDim.x * 4) {
      const float4 u = *reinterpret_cast<const float4*>(hc_row + c), ww = *reinterpret_cast<const float4*>(w + c);
      store4<T>(o + c, make_float4(u.x * inv * ww.x, u.y * inv * ww.y, u.z * inv * ww.z, u.w * inv * ww.w));
    }
  } else {
    for (int c = threadIdx.x; c < width; c += blockDim.x) o[c] = from_f32<T>(hc_row[c] * inv * w[c]);
  }
}

template <typename T, int STREAMS>
static int hyper_norm_shape(float* x, const void* y, const float* mix, const float* out_w, const float* in_w, const float* w, float eps, void* h,
                            const int* row_ids, int n_out, int streams, int width, void* stream) {
  const size_t smem = (size_t)(((width + 3) & ~3) + streams * streams + 2 * streams) * sizeof(float);
  if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
  const bool vec = width % 4 == 0 && !(((uintptr_t)x | (uintptr_t)w) & 15) && !(((uintptr_t)y | (uintptr_t)h) & (4 * sizeof(T) - 1));
  void (*kernel)(float*, const T*, const float*, const float*, const float*, const float*, float, T*, const int*, int, int) =
      vec ? hyper_norm_kernel<T, STREAMS, true> : hyper_norm_kernel<T, STREAMS, false>;
  if (smem > 48 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  // a few rows finish sooner with more threads to a row; many share the SMs better with fewer
  const int threads = width >= 2048 && n_out <= 256 ? 512 : width >= 1024 ? 256 : 128;
  launch(kernel, dim3(n_out), dim3(threads), smem, (cudaStream_t)stream, x, (const T*)y, mix, out_w, in_w, w, eps, (T*)h, row_ids,
         streams, width);
  return launch_status();
}

template <typename T>
static int hyper_norm(float* x, const void* y, const float* mix, const float* out_w, const float* in_w, const float* w, float eps, void* h,
                      const int* row_ids, int n_out, int streams, int width, void* stream) {
  if (n_out <= 0) return 0;
  if (streams < 1 || streams > HC_MAX_STREAMS || width <= 0 || !w || !h || (y && (!mix || !out_w))) return (int)cudaErrorInvalidValue;
  switch (streams) {
    case 1: return hyper_norm_shape<T, 1>(x, y, mix, out_w, in_w, w, eps, h, row_ids, n_out, streams, width, stream);
    case 2: return hyper_norm_shape<T, 2>(x, y, mix, out_w, in_w, w, eps, h, row_ids, n_out, streams, width, stream);
    case 3: return hyper_norm_shape<T, 3>(x, y, mix, out_w, in_w, w, eps, h, row_ids, n_out, streams, width, stream);
    case 4: return hyper_norm_shape<T, 4>(x, y, mix, out_w, in_w, w, eps, h, row_ids, n_out, streams, width, stream);
    default: return hyper_norm_shape<T, 0>(x, y, mix, out_w, in_w, w, eps, h, row_ids, n_out, streams, width, stream);
  }
}
Q25_EXPORT int q25_hyper_norm_f32(float* x, const void* y, const float* mix, const float* ow, const float* iw, const float* w, float eps, void* h,
                                  const int* rows, int n, int streams, int width, void* s) {
  return hyper_norm<float>(x, y, mix, ow, iw, w, eps, h, rows, n, streams, width, s);
}
Q25_EXPORT int q25_hyper_norm_bf16(float* x, const void* y, const float* mix, const float* ow, const float* iw, const float* w, float eps, void* h,
                                   const int* rows, int n, int streams, int width, void* s) {
  return hyper_norm<bf16>(x, y, mix, ow, iw, w, eps, h, rows, n, streams, width, s);
}

// The stream's start: x[n, s, :] = E[token n] + P[row], the same for every s.  row is the last one of P (index `buckets`)
// for a request's first token, else (previous token * mul_prev + token * mul_cur) mod buckets, the product taken in 64
// bits.  pairs == nullptr: no second table.  The token before an entry's first one comes from `last_token` (one int per
// state slot); the block of that first row then leaves the entry's last token there, so a run may be cut anywhere.
template <typename T>
__global__ void embed_pair_kernel(const T* __restrict__ table, const T* __restrict__ pairs, const int* __restrict__ ids,
                                  const int* __restrict__ token_seq, const int* __restrict__ cu_q, const int* __restrict__ q_start,
                                  const int* __restrict__ slot_ids, int* __restrict__ last_token, float* __restrict__ x, int width, int vocab,
                                  long long buckets, long long mul_prev, long long mul_cur, int streams) {
  pdl_trigger();
  pdl_wait();
  const int n = blockIdx.x;
  int id = ids[n];
  id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);      // the host validates ids; never read outside
  const T* e = table + (size_t)id * width;
  const T* p = nullptr;
  if (pairs) {
    const int seq = token_seq[n], first = cu_q[seq];
    long long row = buckets;
    if (n > first || q_start[seq] > 0) {
      const int prev = n > first ? ids[n - 1] : last_token[slot_ids[seq]];
      row = ((long long)prev * mul_prev + (long long)id * mul_cur) % buckets;
      if (row < 0) row += buckets;
    }
    p = pairs + (size_t)row * width;
    __syncthreads();                                     // every thread has read the slot before it is written
    if (n == first && threadIdx.x == 0) last_token[slot_ids[seq]] = ids[cu_q[seq + 1] - 1];
  }
  float* dst = x + (size_t)n * streams * width;
  for (int c = threadIdx.x; c < width; c += blockDim.x) {
    const float v = to_f32(e[c]) + (p ? to_f32(p[c]) : 0.f);
    for (int s = 0; s < streams; ++s) dst[(size_t)s * width + c] = v;
  }
}

template <typename T>
static int embed_pair(const void* table, const void* pairs, const int* ids, const int* token_seq, const int* cu_q, const int* q_start,
                      const int* slot_ids, int* last_token, float* x, int n, int width, int vocab, long long buckets, long long mul_prev,
                      long long mul_cur, int streams, void* stream) {
  if (n <= 0) return 0;
  if (streams < 1 || (pairs && (buckets < 1 || !last_token))) return (int)cudaErrorInvalidValue;
  launch(embed_pair_kernel<T>, dim3(n), dim3(width >= 1024 ? 256 : 128), 0, (cudaStream_t)stream, (const T*)table, (const T*)pairs, ids, token_seq,
         cu_q, q_start, slot_ids, last_token, x, width, vocab, buckets, mul_prev, mul_cur, streams);
  return launch_status();
}
Q25_EXPORT int q25_hyper_embed_f32(const void* t, const void* p, const int* ids, const int* ts, const int* cu, const int* qs, const int* sl, int* last,
                                   float* x, int n, int w, int v, long long b, long long mp, long long mc, int streams, void* s) {
  return embed_pair<float>(t, p, ids, ts, cu, qs, sl, last, x, n, w, v, b, mp, mc, streams, s);
}
Q25_EXPORT int q25_hyper_embed_bf16(const void* t, const void* p, const int* ids, const int* ts, const int* cu, const int* qs, const int* sl, int* last,
                                    float* x, int n, int w, int v, long long b, long long mp, long long mc, int streams, void* s) {
  return embed_pair<bf16>(t, p, ids, ts, cu, qs, sl, last, x, n, w, v, b, mp, mc, streams, s);
}
