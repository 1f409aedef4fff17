// Latent attention keeps one compressed row per token instead of keys and values per head: the
// latent c (RMS-normed, with a weight) followed by one rotated key part that all heads share.  This
// kernel makes that row from the down projection's output and writes it into the token's page slot.
//
//   row[0 .. C)      = x[0 .. C) / sqrt(mean(x[0 .. C)^2) + eps) * w        (statistics in float)
//   row[C .. C + R)  = rotate(x[C .. C + R))                                 (not normed)
//
// The attention kernels then read the row as the single kv head's key (C + R channels) and its first
// C channels as the value.  Where the queries come through a latent of their own, the same launch norms that too (a
// second row of CTAs).  Where the heads' results are gated, another kernel multiplies them with the sigmoid of the
// token's gate channels.
#include "rotary.cuh"

template <typename T, bool EXACT>
__global__ void latent_store_kernel(const T* __restrict__ x, int x_row, int C, int R, const float* __restrict__ w, float eps,
                                    const float* __restrict__ angles, int half, int layout, T* __restrict__ pages,
                                    const int* __restrict__ kv_slot, const T* __restrict__ q, int q_row, int Cq,
                                    const float* __restrict__ q_w, T* __restrict__ q_out) {
  pdl_trigger();
  pdl_wait();
  __shared__ float scratch[32];
  if (blockIdx.y == 1 || !pages) {            // the queries' latent
    const T* qr = q + (size_t)blockIdx.x * q_row;
    float sq = 0.f;
    for (int c = threadIdx.x; c < Cq; c += blockDim.x) {
      const float v = to_f32(qr[c]);
      sq = fmaf(v, v, sq);
    }
    const float q_total = block_sum(sq, scratch);
    const float q_inv = EXACT ? 1.0f / sqrtf(q_total / (float)Cq + eps) : rsqrtf(q_total / (float)Cq + eps);
    T* o = q_out + (size_t)blockIdx.x * Cq;
    for (int c = threadIdx.x; c < Cq; c += blockDim.x) o[c] = from_f32<T>(to_f32(qr[c]) * q_inv * q_w[c]);
    return;
  }
  const int tok = blockIdx.x;
  const T* xr = x + (size_t)tok * x_row;
  float ss = 0.f;
  for (int c = threadIdx.x; c < C; c += blockDim.x) {
    const float v = to_f32(xr[c]);
    ss = fmaf(v, v, ss);
  }
  const float total = block_sum(ss, scratch);
  const float inv = EXACT ? 1.0f / sqrtf(total / (float)C + eps) : rsqrtf(total / (float)C + eps);
  const int slot = kv_slot[tok];
  if (slot < 0) return;
  T* row = pages + (size_t)slot * (C + R);
  for (int c = threadIdx.x; c < C; c += blockDim.x) row[c] = from_f32<T>(to_f32(xr[c]) * inv * w[c]);
  const float* ang = angles ? angles + (size_t)tok * half * 2 : nullptr;
  for (int c = threadIdx.x; c < R; c += blockDim.x) row[C + c] = from_f32<T>(rotary_channel<T>(xr + C, c, half, layout, ang));
}

template <typename T, bool EXACT>
static int latent_store(const void* x, int x_row, int C, int R, const float* w, float eps, const float* angles, int half, int layout,
                        void* pages, const int* kv_slot, int n, const void* q, int q_row, int Cq, const float* q_w, void* q_out, void* stream) {
  if (n <= 0 || (!pages && !q)) return 0;
  if (C <= 0 || R < 0 || 2 * half > R || (pages && !kv_slot) || (q && (Cq <= 0 || !q_w || !q_out))) return (int)cudaErrorInvalidValue;
  launch(latent_store_kernel<T, EXACT>, dim3(n, pages && q ? 2 : 1), dim3(128), 0, (cudaStream_t)stream, (const T*)x, x_row, C, R, w, eps, angles,
         half, layout, (T*)pages, kv_slot, (const T*)q, q_row, Cq, q_w, (T*)q_out);
  return launch_status();
}
Q25_EXPORT int q25_latent_store_f32(const void* x, int xr, int C, int R, const float* w, float eps, const float* ang, int half,
                                    int layout, void* pages, const int* slot, int n, const void* q, int qr, int Cq, const float* qw, void* qo, void* s) {
  return latent_store<float, true>(x, xr, C, R, w, eps, ang, half, layout, pages, slot, n, q, qr, Cq, qw, qo, s);
}
Q25_EXPORT int q25_latent_store_bf16(const void* x, int xr, int C, int R, const float* w, float eps, const float* ang, int half,
                                     int layout, void* pages, const int* slot, int n, const void* q, int qr, int Cq, const float* qw, void* qo, void* s) {
  return latent_store<bf16, false>(x, xr, C, R, w, eps, ang, half, layout, pages, slot, n, q, qr, Cq, qw, qo, s);
}

// y[n, c] *= sigmoid(g[n, c]), in place; y contiguous, g strided rows.
template <typename T, bool VEC>
__global__ void latent_gate_kernel(T* __restrict__ y, const T* __restrict__ g, int g_row, int channels) {
  pdl_trigger();
  pdl_wait();
  const T* gr = g + (size_t)blockIdx.y * g_row;
  T* yr = y + (size_t)blockIdx.y * channels;
  if (VEC) {
    for (int c = (blockIdx.x * blockDim.x + threadIdx.x) * 4; c < channels; c += gridDim.x * blockDim.x * 4) {
      const float4 v = load4<T>(yr + c), z = load4<T>(gr + c);
      store4<T>(yr + c, make_float4(v.x / (1.0f + expf(-z.x)), v.y / (1.0f + expf(-z.y)), v.z / (1.0f + expf(-z.z)), v.w / (1.0f + expf(-z.w))));
    }
  } else {
    for (int c = blockIdx.x * blockDim.x + threadIdx.x; c < channels; c += gridDim.x * blockDim.x)
      yr[c] = from_f32<T>(to_f32(yr[c]) / (1.0f + expf(-to_f32(gr[c]))));
  }
}
template <typename T>
static int latent_gate(void* y, const void* g, int g_row, int n, int channels, void* stream) {
  if (n <= 0 || channels <= 0) return 0;
  const bool vec = channels % 4 == 0 && g_row % 4 == 0 && !(((uintptr_t)y | (uintptr_t)g) & (4 * sizeof(T) - 1));
  const dim3 block(256);
  for (int at = 0; at < n; at += 65535) {                         // the grid's second dimension ends at 65,535
    const dim3 grid((channels + 1023) / 1024, n - at < 65535 ? n - at : 65535);
    T* yy = (T*)y + (size_t)at * channels;
    const T* gg = (const T*)g + (size_t)at * g_row;
    if (vec) launch(latent_gate_kernel<T, true>, grid, block, 0, (cudaStream_t)stream, yy, gg, g_row, channels);
    else launch(latent_gate_kernel<T, false>, grid, block, 0, (cudaStream_t)stream, yy, gg, g_row, channels);
  }
  return launch_status();
}
Q25_EXPORT int q25_latent_gate_f32(void* y, const void* g, int gr, int n, int ch, void* s) { return latent_gate<float>(y, g, gr, n, ch, s); }
Q25_EXPORT int q25_latent_gate_bf16(void* y, const void* g, int gr, int n, int ch, void* s) { return latent_gate<bf16>(y, g, gr, n, ch, s); }
