// The residual's step between two layers whose sublayers run side by side on one norm, in one kernel (a block a token):
//
//   h[t] += scale * (a[t] + b[t])              the two sublayers' outputs; b may be the picks of a routed feed-forward
//                                              that have equal weights: pick_weight * sum_k picks[t, k]
//   h[t] += emb_scale * emb[ids[t]] + vec      what joins the residual ahead of a pass over a group of layers: the
//                                              embedding's row (ids null: row t of emb) and a learned vector
//   x[t]  = h[t] / sqrt(mean(h[t]^2) + eps) * w    the norm that the next layer applies
//
// Every piece is optional.  All arithmetic is float32 and the terms are added in a fixed order, so a token's result does
// not depend on the step it is in.  A thread keeps its pieces of four values in registers (rows of up to RSTEP_THREADS * 4 *
// 8 values, a multiple of 4); other widths go value by value and read the row once more for the norm.
#include "api.h"
#include "common.cuh"

namespace exl3 {

constexpr int RSTEP_THREADS = 256, RSTEP_VECS = 8, RSTEP_PICKS = 4;     // picks whose rows are asked for together

struct ResidualStepArgs {
  float* h;
  const void* a; int a_dtype;
  const void* b; int b_dtype;
  const float* picks; int top; float pick_weight;
  float scale;
  const void* emb; int emb_dtype; const int* ids; float emb_scale;
  const float* vec;
  const void* w; int w_dtype; float eps;
  void* x; int x_dtype;
  int H;
};

__device__ inline float rs_one(const void* p, int dtype, int64_t i) {
  return dtype == DT_F32 ? __ldcg(static_cast<const float*>(p) + i)
                         : __bfloat162float(__ldcg(static_cast<const __nv_bfloat16*>(p) + i));
}
__device__ inline void rs_four(const void* p, int dtype, int64_t i, float (&v)[4]) {
  if (dtype == DT_F32) {
    load_vec_cg(static_cast<const float*>(p) + i, v);
  } else {
    const uint2 r = __ldcg(reinterpret_cast<const uint2*>(static_cast<const __nv_bfloat16*>(p) + i));
    v[0] = __uint_as_float(r.x << 16); v[1] = __uint_as_float(r.x & 0xffff0000u);
    v[2] = __uint_as_float(r.y << 16); v[3] = __uint_as_float(r.y & 0xffff0000u);
  }
}

template <int VECS>
__global__ void __launch_bounds__(RSTEP_THREADS) residual_step_kernel(const ResidualStepArgs s) {
  __shared__ float red[32];
  const int t = blockIdx.x;
  const int64_t base = (int64_t)t * s.H;
  float wv[VECS][4], add[VECS][4];                 // weights do not depend on the kernel before
#pragma unroll
  for (int p = 0; p < VECS; ++p) {
    const int c = (p * blockDim.x + threadIdx.x) * 4;
#pragma unroll
    for (int e = 0; e < 4; ++e) add[p][e] = 0.0f;
    if (c < s.H) {
      if (s.w) rs_four(s.w, s.w_dtype, c, wv[p]);
      if (s.vec) load_vec_cg(s.vec + c, add[p]);
    }
  }
  pdl_wait();
  pdl_trigger();
  float hv[VECS][4], y[VECS][4];
#pragma unroll
  for (int p = 0; p < VECS; ++p) {
    const int c = (p * blockDim.x + threadIdx.x) * 4;
#pragma unroll
    for (int e = 0; e < 4; ++e) { y[p][e] = 0.0f; hv[p][e] = 0.0f; }
    if (c < s.H) {
      load_vec_cg(s.h + base + c, hv[p]);
      if (s.a) rs_four(s.a, s.a_dtype, base + c, y[p]);
    }
  }
  if (s.b) {
#pragma unroll
    for (int p = 0; p < VECS; ++p) {
      const int c = (p * blockDim.x + threadIdx.x) * 4;
      if (c < s.H) {
        float v[4];
        rs_four(s.b, s.b_dtype, base + c, v);
#pragma unroll
        for (int e = 0; e < 4; ++e) y[p][e] += v[e];
      }
    }
  }
  if (s.picks) {
    float sum[VECS][4];
#pragma unroll
    for (int p = 0; p < VECS; ++p)
#pragma unroll
      for (int e = 0; e < 4; ++e) sum[p][e] = 0.0f;
    for (int k0 = 0; k0 < s.top; k0 += RSTEP_PICKS) {
#pragma unroll
      for (int p = 0; p < VECS; ++p) {
        const int c = (p * blockDim.x + threadIdx.x) * 4;
        if (c < s.H) {
          float v[RSTEP_PICKS][4];
#pragma unroll
          for (int k = 0; k < RSTEP_PICKS; ++k) {
#pragma unroll
            for (int e = 0; e < 4; ++e) v[k][e] = 0.0f;
            if (k0 + k < s.top) load_vec_cg(s.picks + ((int64_t)t * s.top + k0 + k) * s.H + c, v[k]);
          }
#pragma unroll
          for (int k = 0; k < RSTEP_PICKS; ++k)
#pragma unroll
            for (int e = 0; e < 4; ++e) sum[p][e] += v[k][e];
        }
      }
    }
#pragma unroll
    for (int p = 0; p < VECS; ++p)
#pragma unroll
      for (int e = 0; e < 4; ++e) y[p][e] = fmaf(s.pick_weight, sum[p][e], y[p][e]);
  }
  if (s.emb) {
    const int64_t row = (int64_t)(s.ids ? __ldcg(s.ids + t) : t) * s.H;
#pragma unroll
    for (int p = 0; p < VECS; ++p) {
      const int c = (p * blockDim.x + threadIdx.x) * 4;
      if (c < s.H) {
        float v[4];
        rs_four(s.emb, s.emb_dtype, row + c, v);
#pragma unroll
        for (int e = 0; e < 4; ++e) add[p][e] = fmaf(s.emb_scale, v[e], add[p][e]);
      }
    }
  }
  float ss = 0.0f;
#pragma unroll
  for (int p = 0; p < VECS; ++p) {
    const int c = (p * blockDim.x + threadIdx.x) * 4;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      hv[p][e] = fmaf(s.scale, y[p][e], hv[p][e]) + add[p][e];
      ss += hv[p][e] * hv[p][e];                   // zeros beyond the row
    }
    if (c < s.H) store_vec(s.h + base + c, hv[p]);
  }
  if (!s.w) return;
  const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)s.H + s.eps);
#pragma unroll
  for (int p = 0; p < VECS; ++p) {
    const int c = (p * blockDim.x + threadIdx.x) * 4;
    if (c < s.H) {
      float o[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) o[e] = hv[p][e] * inv * wv[p][e];
      if (s.x_dtype == DT_F32) {
        store_vec(static_cast<float*>(s.x) + base + c, o);
      } else {
        __nv_bfloat162 lo = __floats2bfloat162_rn(o[0], o[1]), hi = __floats2bfloat162_rn(o[2], o[3]);
        uint2 r;
        r.x = *reinterpret_cast<uint32_t*>(&lo);
        r.y = *reinterpret_cast<uint32_t*>(&hi);
        *reinterpret_cast<uint2*>(static_cast<__nv_bfloat16*>(s.x) + base + c) = r;
      }
    }
  }
}

// Any width, a value at a time.
__global__ void __launch_bounds__(RSTEP_THREADS) residual_step_any_kernel(const ResidualStepArgs s) {
  __shared__ float red[32];
  pdl_wait();
  pdl_trigger();
  const int t = blockIdx.x;
  const int64_t base = (int64_t)t * s.H;
  const int64_t row = s.emb ? (int64_t)(s.ids ? __ldcg(s.ids + t) : t) * s.H : 0;
  float ss = 0.0f;
  for (int c = threadIdx.x; c < s.H; c += blockDim.x) {
    float y = s.a ? rs_one(s.a, s.a_dtype, base + c) : 0.0f;
    if (s.b) y += rs_one(s.b, s.b_dtype, base + c);
    if (s.picks) {
      float sum = 0.0f;
      for (int k = 0; k < s.top; ++k) sum += __ldcg(s.picks + ((int64_t)t * s.top + k) * s.H + c);
      y = fmaf(s.pick_weight, sum, y);
    }
    float add = s.vec ? s.vec[c] : 0.0f;
    if (s.emb) add = fmaf(s.emb_scale, rs_one(s.emb, s.emb_dtype, row + c), add);
    const float v = fmaf(s.scale, y, __ldcg(s.h + base + c)) + add;
    s.h[base + c] = v;
    ss += v * v;
  }
  if (!s.w) return;
  const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)s.H + s.eps);
  for (int c = threadIdx.x; c < s.H; c += blockDim.x) {
    const float o = __ldcg(s.h + base + c) * inv * rs_one(s.w, s.w_dtype, c);       // the thread's own value
    if (s.x_dtype == DT_F32) static_cast<float*>(s.x)[base + c] = o;
    else static_cast<__nv_bfloat16*>(s.x)[base + c] = __float2bfloat16_rn(o);
  }
}

}  // namespace exl3

using namespace exl3;

extern "C" int exl3_residual_step(float* h, const void* a, int a_dtype, const void* b, int b_dtype, const float* picks,
                                  int top, float pick_weight, float scale, const void* emb, int emb_dtype, const int* ids,
                                  float emb_scale, const float* vec, const void* w, int w_dtype, float eps, void* x,
                                  int x_dtype, int T, int H, cudaStream_t stream) {
  if (T == 0) return 0;
  if (T < 0 || H < 1 || h == nullptr || (picks != nullptr && top < 1) || (w != nullptr && x == nullptr)) {
    set_error("residual_step: bad sizes rows=%d width=%d picks=%d", T, H, top);
    return ERR_BAD_ARGUMENT;
  }
  const int types[5] = {a_dtype, b_dtype, emb_dtype, w_dtype, x_dtype};
  for (int d : types)
    if (d != DT_F32 && d != DT_BF16) { set_error("residual_step: unsupported element type %d", d); return ERR_UNSUPPORTED; }
  ResidualStepArgs s;
  s.h = h; s.a = a; s.a_dtype = a_dtype; s.b = b; s.b_dtype = b_dtype; s.picks = picks; s.top = top;
  s.pick_weight = pick_weight; s.scale = scale; s.emb = emb; s.emb_dtype = emb_dtype; s.ids = ids; s.emb_scale = emb_scale;
  s.vec = vec; s.w = w; s.w_dtype = w_dtype; s.eps = eps; s.x = x; s.x_dtype = x_dtype; s.H = H;
  const bool vec4 = H % 4 == 0 && H <= RSTEP_THREADS * 4 * RSTEP_VECS && aligned16(h) && aligned16(a) && aligned16(b) &&
                    aligned16(picks) && aligned16(emb) && aligned16(vec) && aligned16(w) && aligned16(x);
  if (vec4) {
    int threads = ceil_div(H / 4, 32) * 32;
    if (threads > RSTEP_THREADS) threads = RSTEP_THREADS;
    const int need = ceil_div(H, threads * 4);
    if (need <= 1) launch_pdl(residual_step_kernel<1>, dim3(T), dim3(threads), 0, stream, s);
    else if (need <= 2) launch_pdl(residual_step_kernel<2>, dim3(T), dim3(threads), 0, stream, s);
    else if (need <= 4) launch_pdl(residual_step_kernel<4>, dim3(T), dim3(threads), 0, stream, s);
    else launch_pdl(residual_step_kernel<RSTEP_VECS>, dim3(T), dim3(threads), 0, stream, s);
  } else {
    launch_pdl(residual_step_any_kernel, dim3(T), dim3(RSTEP_THREADS), 0, stream, s);
  }
  return launch_status("residual_step");
}
