// What joins the branches of a layer whose sublayers read one norm's output and are added at once, times a constant:
//   llmi_normed_pair       y[t] (+)= c * (a[t] / rms(a[t]) * wa + b[t] / rms(b[t]) * wb) — two mixers side by side, each
//                          normed over the model width with a weight of its own, then averaged (c = 1/2)
//   llmi_stream_axpy_norm  x[t] += m * y[t], and (optionally) h[t] = norm_w * x[t] / rms(x[t]) of the new x in the same
//                          pass: the norm ahead of the next layer
//   llmi_stream_postnorm   x[t] = norm_w * v / rms(v) with v = a * x[t] + y[t]: a branch joins the stream and the norm BEHIND
//                          the sum replaces it; h[t] receives the new x in the compute type (what the next branch reads).
//                          Without y and norm_w: only the copy h = x
//   llmi_softcap_rows      v = cap * tanh(v / cap) in place (the logits)
// rms(v) = sqrt(mean(v^2) + eps).  All arithmetic fp32; a block per row, rows are treated alone.
#include <math.h>

#include "common.cuh"

namespace llmi {

__device__ __forceinline__ void store4(float* o, float a, float b, float c, float d) {
  *reinterpret_cast<float4*>(o) = make_float4(a, b, c, d);
}
__device__ __forceinline__ void store4(__nv_bfloat16* o, float a, float b, float c, float d) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
  uint2 u;
  u.x = *reinterpret_cast<const uint32_t*>(&lo);
  u.y = *reinterpret_cast<const uint32_t*>(&hi);
  *reinterpret_cast<uint2*>(o) = u;
}

__global__ void __launch_bounds__(256)
normed_pair_kernel(const float* __restrict__ a, long lda, const float* __restrict__ wa, const float* __restrict__ b, long ldb,
                   const float* __restrict__ wb, float eps, float coeff, float* __restrict__ y, long ldy, int W, int add,
                   int vec4) {
  __shared__ float scratch[32];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  const float* ar = a + (size_t)t * lda;
  const float* br = b + (size_t)t * ldb;
  float* yr = y + (size_t)t * ldy;
  float sa = 0.f, sb = 0.f;
  if (vec4) {                // rows of whole 16-byte pieces, every row starting on one
    for (int i = threadIdx.x; i < W / 4; i += blockDim.x) {
      const float4 p = reinterpret_cast<const float4*>(ar)[i], q = reinterpret_cast<const float4*>(br)[i];
      sa = fmaf(p.x, p.x, sa); sa = fmaf(p.y, p.y, sa); sa = fmaf(p.z, p.z, sa); sa = fmaf(p.w, p.w, sa);
      sb = fmaf(q.x, q.x, sb); sb = fmaf(q.y, q.y, sb); sb = fmaf(q.z, q.z, sb); sb = fmaf(q.w, q.w, sb);
    }
  } else {
    for (int i = threadIdx.x; i < W; i += blockDim.x) {
      sa = fmaf(ar[i], ar[i], sa);
      sb = fmaf(br[i], br[i], sb);
    }
  }
  sa = block_sum(sa, scratch);
  __syncthreads();
  sb = block_sum(sb, scratch);
  const float ia = 1.0f / sqrtf(sa / (float)W + eps), ib = 1.0f / sqrtf(sb / (float)W + eps);
  if (vec4) {
    for (int i = threadIdx.x; i < W / 4; i += blockDim.x) {
      const float4 p = reinterpret_cast<const float4*>(ar)[i], q = reinterpret_cast<const float4*>(br)[i];
      const float4 u = reinterpret_cast<const float4*>(wa)[i], w = reinterpret_cast<const float4*>(wb)[i];
      float4 v = make_float4(coeff * (p.x * ia * u.x + q.x * ib * w.x), coeff * (p.y * ia * u.y + q.y * ib * w.y),
                             coeff * (p.z * ia * u.z + q.z * ib * w.z), coeff * (p.w * ia * u.w + q.w * ib * w.w));
      if (add) {
        const float4 o = reinterpret_cast<const float4*>(yr)[i];
        v.x += o.x; v.y += o.y; v.z += o.z; v.w += o.w;
      }
      reinterpret_cast<float4*>(yr)[i] = v;
    }
  } else {
    for (int i = threadIdx.x; i < W; i += blockDim.x) {
      const float v = coeff * (ar[i] * ia * wa[i] + br[i] * ib * wb[i]);
      yr[i] = add ? yr[i] + v : v;
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
stream_axpy_norm_kernel(float* __restrict__ x, const float* __restrict__ y, float m, int W, const float* __restrict__ norm_w,
                        float eps, T* __restrict__ h) {
  __shared__ float scratch[32];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  float* xr = x + (size_t)t * W;
  const float* yr = y + (size_t)t * W;
  float ss = 0.f;
  if (W % 4 == 0) {          // rows of whole 16-byte pieces (x, y are contiguous: every row starts on one)
    for (int i = threadIdx.x; i < W / 4; i += blockDim.x) {
      float4 v = reinterpret_cast<const float4*>(xr)[i];
      const float4 u = reinterpret_cast<const float4*>(yr)[i];
      v.x = fmaf(m, u.x, v.x); v.y = fmaf(m, u.y, v.y); v.z = fmaf(m, u.z, v.z); v.w = fmaf(m, u.w, v.w);
      reinterpret_cast<float4*>(xr)[i] = v;
      ss = fmaf(v.x, v.x, ss); ss = fmaf(v.y, v.y, ss); ss = fmaf(v.z, v.z, ss); ss = fmaf(v.w, v.w, ss);
    }
  } else {
    for (int i = threadIdx.x; i < W; i += blockDim.x) {
      const float v = fmaf(m, yr[i], xr[i]);
      xr[i] = v;
      ss = fmaf(v, v, ss);
    }
  }
  if (!norm_w) return;
  ss = block_sum(ss, scratch);
  const float scale = 1.0f / sqrtf(ss / (float)W + eps);
  T* hr = h + (size_t)t * W;
  if (W % 4 == 0) {
    for (int i = threadIdx.x; i < W / 4; i += blockDim.x) {          // (my own writes above)
      const float4 v = reinterpret_cast<const float4*>(xr)[i], w = reinterpret_cast<const float4*>(norm_w)[i];
      store4(hr + 4 * i, w.x * (v.x * scale), w.y * (v.y * scale), w.z * (v.z * scale), w.w * (v.w * scale));
    }
  } else {
    for (int i = threadIdx.x; i < W; i += blockDim.x) hr[i] = from_f32<T>(norm_w[i] * (xr[i] * scale));
  }
}

// Each thread keeps its pieces of the row in registers (up to PN_KEEP of them; what is left is formed twice).
constexpr int PN_KEEP = 4;
template <typename T>
__global__ void __launch_bounds__(512)
stream_postnorm_kernel(float* __restrict__ x, const float* __restrict__ y, float alpha, int W, const float* __restrict__ norm_w,
                       float eps, T* __restrict__ h) {
  __shared__ float scratch[32];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  float* xr = x + (size_t)t * W;
  const float* yr = y ? y + (size_t)t * W : nullptr;
  T* hr = h ? h + (size_t)t * W : nullptr;
  if (!y) {
    for (int i = threadIdx.x; i < W; i += blockDim.x) hr[i] = from_f32<T>(xr[i]);
    return;
  }
  float ss = 0.f;
  if (W % 4 == 0) {
    auto joined = [&](int i) {
      const float4 v = reinterpret_cast<const float4*>(xr)[i], u = reinterpret_cast<const float4*>(yr)[i];
      return make_float4(fmaf(alpha, v.x, u.x), fmaf(alpha, v.y, u.y), fmaf(alpha, v.z, u.z), fmaf(alpha, v.w, u.w));
    };
    float4 keep[PN_KEEP];
#pragma unroll
    for (int k = 0; k < PN_KEEP; ++k) {
      const int i = threadIdx.x + k * blockDim.x;
      keep[k] = i < W / 4 ? joined(i) : make_float4(0.f, 0.f, 0.f, 0.f);
      ss = fmaf(keep[k].x, keep[k].x, ss); ss = fmaf(keep[k].y, keep[k].y, ss);
      ss = fmaf(keep[k].z, keep[k].z, ss); ss = fmaf(keep[k].w, keep[k].w, ss);
    }
    for (int i = threadIdx.x + PN_KEEP * blockDim.x; i < W / 4; i += blockDim.x) {
      const float4 v = joined(i);
      ss = fmaf(v.x, v.x, ss); ss = fmaf(v.y, v.y, ss); ss = fmaf(v.z, v.z, ss); ss = fmaf(v.w, v.w, ss);
    }
    const float scale = 1.0f / sqrtf(block_sum(ss, scratch) / (float)W + eps);
    auto leave = [&](int i, float4 v) {
      const float4 w = reinterpret_cast<const float4*>(norm_w)[i];
      v = make_float4(w.x * (v.x * scale), w.y * (v.y * scale), w.z * (v.z * scale), w.w * (v.w * scale));
      reinterpret_cast<float4*>(xr)[i] = v;
      if (hr) store4(hr + 4 * i, v.x, v.y, v.z, v.w);
    };
#pragma unroll
    for (int k = 0; k < PN_KEEP; ++k) {
      const int i = threadIdx.x + k * blockDim.x;
      if (i < W / 4) leave(i, keep[k]);
    }
    for (int i = threadIdx.x + PN_KEEP * blockDim.x; i < W / 4; i += blockDim.x) leave(i, joined(i));
  } else {
    for (int i = threadIdx.x; i < W; i += blockDim.x) {
      const float v = fmaf(alpha, xr[i], yr[i]);
      ss = fmaf(v, v, ss);
    }
    const float scale = 1.0f / sqrtf(block_sum(ss, scratch) / (float)W + eps);
    for (int i = threadIdx.x; i < W; i += blockDim.x) {
      const float v = norm_w[i] * (fmaf(alpha, xr[i], yr[i]) * scale);
      xr[i] = v;
      if (hr) hr[i] = from_f32<T>(v);
    }
  }
}

__global__ void __launch_bounds__(256) softcap_rows_kernel(float* __restrict__ v, size_t n, float cap) {
  pdl_launch_dependents();
  pdl_wait();
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) v[i] = cap * tanhf(v[i] / cap);
}

}  // namespace llmi

using namespace llmi;

// a, b fp32 rows [T, lda / ldb] of W entries; wa, wb fp32 [W]; y fp32 [T, ldy] receives (add == 0) or gains the result.
LLMI_EXPORT int llmi_normed_pair(const float* a, long lda, const float* wa, const float* b, long ldb, const float* wb, float eps,
                                 float coeff, float* y, long ldy, int W, int n_rows, int add, cudaStream_t stream) {
  if (n_rows <= 0 || W <= 0) return LLMI_ERR_BAD_SIZE;
  const int threads = W >= 1024 ? 256 : (W >= 256 ? 128 : 64);
  const int vec4 = W % 4 == 0 && lda % 4 == 0 && ldb % 4 == 0 && ldy % 4 == 0 && !((uintptr_t)a & 15) && !((uintptr_t)b & 15) &&
                   !((uintptr_t)y & 15) && !((uintptr_t)wa & 15) && !((uintptr_t)wb & 15);
  return launch_pdl(PDL_SMALL, normed_pair_kernel, dim3(n_rows), dim3(threads), 0, stream, a, lda, wa, b, ldb, wb, eps, coeff, y, ldy,
                    W, add, vec4);
}

// x, y fp32 [T, W] contiguous: x += m * y.  With norm_w (fp32 [W]): h [T, W] contiguous in `dtype` = the RMS norm of the
// new x with that weight (computed as the norm kernel does: weight * (x * scale), rounded once).
LLMI_EXPORT int llmi_stream_axpy_norm(float* x, const float* y, float m, int n_rows, int W, const float* norm_w, float eps,
                                      int dtype, void* h, cudaStream_t stream) {
  if (n_rows <= 0 || W <= 0 || (norm_w && !h)) return LLMI_ERR_BAD_SIZE;
  if (W % 4 == 0 && (((uintptr_t)x & 15) || ((uintptr_t)y & 15) || ((uintptr_t)norm_w & 15) || ((uintptr_t)h & 15))) return LLMI_ERR_ALIGN;
  const int threads = W >= 1024 ? 256 : (W >= 256 ? 128 : 64);
  if (!norm_w || dtype == LLMI_DTYPE_F32)
    return launch_pdl(PDL_SMALL, stream_axpy_norm_kernel<float>, dim3(n_rows), dim3(threads), 0, stream, x, y, m, W, norm_w, eps,
                      (float*)h);
  if (dtype == LLMI_DTYPE_BF16)
    return launch_pdl(PDL_SMALL, stream_axpy_norm_kernel<__nv_bfloat16>, dim3(n_rows), dim3(threads), 0, stream, x, y, m, W, norm_w,
                      eps, (__nv_bfloat16*)h);
  return LLMI_ERR_BAD_DTYPE;
}

// x, y fp32 [T, W] contiguous; norm_w fp32 [W]; h [T, W] contiguous in `dtype`, or null.  x = norm_w * v / rms(v) with
// v = alpha * x + y, and h = x; with y null only h = x.
LLMI_EXPORT int llmi_stream_postnorm(float* x, const float* y, float alpha, int n_rows, int W, const float* norm_w, float eps, int dtype,
                                     void* h, cudaStream_t stream) {
  if (n_rows <= 0 || W <= 0 || (y == nullptr) != (norm_w == nullptr) || (!y && !h)) return LLMI_ERR_BAD_SIZE;
  if (W % 4 == 0 && (((uintptr_t)x & 15) || ((uintptr_t)y & 15) || ((uintptr_t)norm_w & 15) || ((uintptr_t)h & 15))) return LLMI_ERR_ALIGN;
  // few rows: as many threads as a row gives work, for the shortest way through; many: four pieces a thread and more rows at a time
  const int few = W >= 2048 ? 512 : (W >= 1024 ? 256 : (W >= 256 ? 128 : 64));
  const int many = W >= 8192 ? 512 : (W >= 4096 ? 256 : (W >= 2048 ? 128 : 64));
  const int threads = n_rows >= 512 ? many : few;
  if (!h || dtype == LLMI_DTYPE_F32)
    return launch_pdl(PDL_SMALL, stream_postnorm_kernel<float>, dim3(n_rows), dim3(threads), 0, stream, x, y, alpha, W, norm_w, eps,
                      (float*)h);
  if (dtype == LLMI_DTYPE_BF16)
    return launch_pdl(PDL_SMALL, stream_postnorm_kernel<__nv_bfloat16>, dim3(n_rows), dim3(threads), 0, stream, x, y, alpha, W, norm_w,
                      eps, (__nv_bfloat16*)h);
  return LLMI_ERR_BAD_DTYPE;
}

// v fp32, n entries: v = cap * tanh(v / cap) in place.
LLMI_EXPORT int llmi_softcap_rows(float* v, long n, float cap, cudaStream_t stream) {
  if (n <= 0 || !(cap > 0.f)) return LLMI_ERR_BAD_SIZE;
  const long most = (long)sm_count() * 8, need = (n + 255) / 256;
  return launch_pdl(PDL_SMALL, softcap_rows_kernel, dim3((unsigned)(need < most ? need : most)), dim3(256), 0, stream, v, (size_t)n, cap);
}
