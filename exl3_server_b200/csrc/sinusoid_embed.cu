// Token embedding plus a sinusoidal vector of the token's position, and the norm that follows.
//
//   v[2i] = table[id][2i] * scale + sin(p f_i),  v[2i + 1] = table[id][2i + 1] * scale + cos(p f_i)
//   h     = v / sqrt(mean(v^2) + eps) * w        (without a weight: h = v)
//   x     = h in bfloat16, when asked for (what the first layer's projections read)
//
// Angles, the sum and the norm are float32; a frequency comes as two float32 numbers (see rope_sincos).
#include "api.h"
#include "common.cuh"

namespace exl3 {

constexpr int SE_THREADS = 256;
constexpr int SE_KEEP = 8;                       // pairs a thread keeps in registers: rows of up to 4096 values

template <typename T>
__global__ void __launch_bounds__(SE_THREADS)
embed_sinusoid_kernel(const int* __restrict__ ids, const int* __restrict__ tok_pos, const T* __restrict__ table, float scale,
                      const float* __restrict__ f_hi, const float* __restrict__ f_lo, const float* __restrict__ w, float eps,
                      float* h, __nv_bfloat16* x, int H, int V) {
  __shared__ float red[32];
  pdl_wait();
  pdl_trigger();
  const int t = blockIdx.x;
  const int id = __ldcg(ids + t);
  const float p = (float)__ldcg(tok_pos + t);
  float* row = h + (int64_t)t * H;
  const bool known = id >= 0 && id < V;          // refused on the host already; never read outside
  const T* e = table + (int64_t)(known ? id : 0) * H;
  const int pairs = (H + 1) / 2;
  auto pair = [&](int i, float& a, float& b) {
    float sn, cs;
    rope_sincos(p, f_hi[i], f_lo[i], &sn, &cs);
    a = known ? Elem<T>::load(e + 2 * i) * scale + sn : 0.0f;
    b = known && 2 * i + 1 < H ? Elem<T>::load(e + 2 * i + 1) * scale + cs : 0.0f;
  };
  float ka[SE_KEEP], kb[SE_KEEP];
  float ss = 0.0f;
#pragma unroll
  for (int k = 0; k < SE_KEEP; ++k) {
    const int i = k * SE_THREADS + threadIdx.x;
    ka[k] = kb[k] = 0.0f;
    if (i < pairs) pair(i, ka[k], kb[k]);
    ss += ka[k] * ka[k] + kb[k] * kb[k];
  }
  for (int i = SE_KEEP * SE_THREADS + threadIdx.x; i < pairs; i += SE_THREADS) {
    float a, b;
    pair(i, a, b);
    ss += a * a + b * b;
  }
  float inv = 1.0f;
  if (w) inv = 1.0f / sqrtf(block_sum(ss, red) / (float)H + eps);
  auto put = [&](int c, float v) {
    if (c >= H) return;
    if (w) v *= inv * w[c];
    row[c] = v;
    if (x) x[(int64_t)t * H + c] = __float2bfloat16_rn(v);
  };
#pragma unroll
  for (int k = 0; k < SE_KEEP; ++k) {
    const int i = k * SE_THREADS + threadIdx.x;
    if (i < pairs) {
      put(2 * i, ka[k]);
      put(2 * i + 1, kb[k]);
    }
  }
  for (int i = SE_KEEP * SE_THREADS + threadIdx.x; i < pairs; i += SE_THREADS) {
    float a, b;
    pair(i, a, b);
    put(2 * i, a);
    put(2 * i + 1, b);
  }
}

}  // namespace exl3

using namespace exl3;

extern "C" int exl3_embed_sinusoid(const int* ids, const int* tok_pos, const void* table, int dtype, float scale,
                                   const float* f_hi, const float* f_lo, const float* norm_w, float eps, float* h, void* x,
                                   int T, int H, int V, cudaStream_t stream) {
  if (T == 0) return 0;
  if (T < 0 || H < 1 || V < 1 || f_hi == nullptr || f_lo == nullptr) {
    set_error("embed_sinusoid: bad sizes T=%d H=%d V=%d, or no frequencies", T, H, V);
    return ERR_BAD_ARGUMENT;
  }
  if (dtype == DT_F32)
    launch_pdl(embed_sinusoid_kernel<float>, dim3(T), dim3(SE_THREADS), 0, stream, ids, tok_pos,
               static_cast<const float*>(table), scale, f_hi, f_lo, norm_w, eps, h, static_cast<__nv_bfloat16*>(x), H, V);
  else if (dtype == DT_BF16)
    launch_pdl(embed_sinusoid_kernel<__nv_bfloat16>, dim3(T), dim3(SE_THREADS), 0, stream, ids, tok_pos,
               static_cast<const __nv_bfloat16*>(table), scale, f_hi, f_lo, norm_w, eps, h, static_cast<__nv_bfloat16*>(x), H,
               V);
  else {
    set_error("embed_sinusoid: unsupported element type %d", dtype);
    return ERR_UNSUPPORTED;
  }
  return launch_status("embed_sinusoid");
}
