// Attention through a low-rank latent ("latent attention"): every token leaves ONE row in the cache,
//     [ c (rank C, RMS-normed) | r (R dims, rotated by position) ],
// and all heads read it.  With the key and value expansions folded into the query and the output
// (q~_h = Uk_hᵀ q_h, out_h = Uv_h Σ p c), a head's score is the plain dot of its query row [q~_h | qrot_h] with the
// cache row, and its context is the weighted sum of the rows' first C entries: multi-query attention with one
// shared head of C + R key dims whose values are the first C of them.
//
// Kernels here:
//   llmi_latent_prepare     per token: RMS norm of the query latent and of c (fp32), rotation of r, append to the cache
//   llmi_latent_prepare_direct  the same for a layer whose queries come straight from its input: per token and head the
//                           plain part of the query in the compute type and its rotated part, and the cache row
//   llmi_latent_q_rotate    the rotated part of every head's query into its row [q~ | qrot]
//   llmi_attention_latent   scores, softmax and context of every (token, head), any sizes, fp32 arithmetic; serves
//                           prompts and single tokens, both types; optionally over a window of the last positions only
// Rotation: pairs turned by the angle float(pos) * inv_freq[i], computed in fp32 with sincosf — neighbours (2i, 2i+1)
// (`pairing` 1) or entries (i, i + rot_dims/2) (`pairing` 0), cos and sin both times `amplitude`; entries beyond rot_dims
// pass unchanged.
#include <math.h>

#include "common.cuh"
#include "step_meta.cuh"

namespace llmi {

// Where pair i of a rotated part of rot_dims entries lies.
__device__ __forceinline__ void pair_places(int i, int rot_dims, int pairing, int& a, int& b) {
  a = pairing ? 2 * i : i;
  b = pairing ? 2 * i + 1 : i + rot_dims / 2;
}

// R entries of src, the first rot_dims of them turned by the position, into dst; thread `me` of `n`.
template <typename T>
__device__ __forceinline__ void rotate_part(const float* __restrict__ src, T* __restrict__ dst, int R, const float* __restrict__ inv_freq,
                                            int rot_dims, int pairing, float amplitude, int pos, int me, int n) {
  for (int i = me; i < rot_dims / 2; i += n) {
    int a, b;
    pair_places(i, rot_dims, pairing, a, b);
    float s, co;
    sincosf((float)pos * inv_freq[i], &s, &co);
    s *= amplitude;
    co *= amplitude;
    dst[a] = from_f32<T>(rot_lo(src[a], src[b], co, s));
    dst[b] = from_f32<T>(rot_hi(src[a], src[b], co, s));
  }
  for (int i = rot_dims + me; i < R; i += n) dst[i] = from_f32<T>(src[i]);
}

// n entries of src, divided by their root mean square and weighted, into dst; the whole block takes part.  A row of up to
// LN_KEEP entries per thread is read once (and its weights before the wait on the kernel ahead: `w` waits for nobody).
constexpr int LP_THREADS = 256, LN_KEEP = 6;
template <typename T>
__device__ __forceinline__ void normed_part(const float* __restrict__ src, const float* __restrict__ w, int n, float eps, T* __restrict__ dst,
                                            const float (&wv)[LN_KEEP], float* scratch) {
  const bool kept = n <= LN_KEEP * LP_THREADS;
  float v[LN_KEEP], ss = 0.f;
  if (kept) {
#pragma unroll
    for (int j = 0; j < LN_KEEP; ++j) {
      const int i = threadIdx.x + j * LP_THREADS;
      v[j] = i < n ? src[i] : 0.f;
    }
#pragma unroll
    for (int j = 0; j < LN_KEEP; ++j) ss = fmaf(v[j], v[j], ss);
  } else {
    for (int i = threadIdx.x; i < n; i += LP_THREADS) ss = fmaf(src[i], src[i], ss);
  }
  const float sc = 1.0f / sqrtf(block_sum(ss, scratch) / (float)n + eps);
  if (kept) {
#pragma unroll
    for (int j = 0; j < LN_KEEP; ++j) {
      const int i = threadIdx.x + j * LP_THREADS;
      if (i < n) dst[i] = from_f32<T>(wv[j] * (v[j] * sc));
    }
  } else {
    for (int i = threadIdx.x; i < n; i += LP_THREADS) dst[i] = from_f32<T>(w[i] * (src[i] * sc));
  }
}

// Two blocks per token: the query latent (blockIdx.y 0), and the cache row (1; only where rows are written).  down: fp32 [T,
// ld]: columns [0, Q) query latent, [Q, Q+C) key/value latent, [Q+C, Q+C+R) the shared key part.  cq (type T) [T, Q]
// receives the normed query latent; the cache row of (sequence, position) receives [normed c | rotated r].
template <typename T>
__global__ void __launch_bounds__(LP_THREADS)
latent_prepare_kernel(const float* __restrict__ down, long ld, int Q, int C, int R, const float* __restrict__ wq,
                      const float* __restrict__ wc, float eps, const float* __restrict__ inv_freq, int rot_dims,
                      const int32_t* __restrict__ tok_seq, const int32_t* __restrict__ tok_pos, PagedKV kv,
                      T* __restrict__ cache, T* __restrict__ cq, int write_kv, int pairing, float amplitude) {
  __shared__ float scratch[32];
  pdl_launch_dependents();
  const int t = blockIdx.x, seq = tok_seq[t];            // (the step's index block: there before any of its kernels)
  const bool is_row = blockIdx.y == 1;
  const int n = is_row ? C : Q;
  const float* w = is_row ? wc : wq;
  float wv[LN_KEEP];
#pragma unroll
  for (int j = 0; j < LN_KEEP; ++j) {
    const int i = threadIdx.x + j * LP_THREADS;
    wv[j] = i < n ? w[i] : 0.f;
  }
  const float* row = down + (size_t)t * ld;
  if (!is_row) {
    T* cq_row = cq + (size_t)t * Q;
    pdl_wait();
    if (seq < 0) {
      for (int i = threadIdx.x; i < Q; i += blockDim.x) cq_row[i] = from_f32<T>(0.f);
      return;
    }
    normed_part<T>(row, wq, Q, eps, cq_row, wv, scratch);
    return;
  }
  if (seq < 0) {
    pdl_wait();
    return;
  }
  const int pos = tok_pos[t];
  const float* c = row + Q;
  T* dst = cache + kv_row_offset(kv, seq, pos, 0);
  pdl_wait();
  normed_part<T>(c, wc, C, eps, dst, wv, scratch);
  rotate_part<T>(c + C, dst + C, R, inv_freq, rot_dims, pairing, amplitude, pos, threadIdx.x, blockDim.x);
}

// The same for a layer whose queries come straight from its input.  proj: fp32 [T, ld]: [ q: H * (D + R) | c: C | r: R ].
// One warp per (token, item), items 0 .. H-1 the query heads, item H the cache row: head h's plain part goes to
// qn [T, H, D], its rotated part behind the C folded entries of qa [T, H, C + R]; the cache row receives
// [normed c | rotated r].
constexpr int LP_WARPS = 4;
template <typename T>
__global__ void __launch_bounds__(LP_WARPS * 32)
latent_prepare_direct_kernel(const float* __restrict__ proj, long ld, int H, int D, int C, int R, const float* __restrict__ wc,
                             float eps, const float* __restrict__ inv_freq, int rot_dims, int pairing,
                             const int32_t* __restrict__ tok_seq, const int32_t* __restrict__ tok_pos, PagedKV kv,
                             T* __restrict__ cache, T* __restrict__ qn, T* __restrict__ qa, long ldqa, int n_tokens, int write_kv, float amplitude) {
  pdl_launch_dependents();
  pdl_wait();
  const long item = (long)blockIdx.x * LP_WARPS + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  const int t = (int)(item / (H + 1)), h = (int)(item - (long)t * (H + 1));
  if (t >= n_tokens) return;
  const int seq = tok_seq[t];
  const float* row = proj + (size_t)t * ld;
  if (h < H) {
    const float* src = row + (size_t)h * (D + R);
    T* plain = qn + ((size_t)t * H + h) * D;
    T* rot = qa + (size_t)t * ldqa + (size_t)h * (C + R) + C;
    if (seq < 0) {
      for (int i = lane; i < D; i += 32) plain[i] = from_f32<T>(0.f);
      for (int i = lane; i < R; i += 32) rot[i] = from_f32<T>(0.f);
      return;
    }
    for (int i = lane; i < D; i += 32) plain[i] = from_f32<T>(src[i]);
    rotate_part<T>(src + D, rot, R, inv_freq, rot_dims, pairing, amplitude, tok_pos[t], lane, 32);
    return;
  }
  if (seq < 0 || !write_kv) return;
  const float* c = row + (size_t)H * (D + R);
  float ss = 0.f;
  for (int i = lane; i < C; i += 32) ss = fmaf(c[i], c[i], ss);
  const float sc = 1.0f / sqrtf(warp_sum(ss) / (float)C + eps);
  const int pos = tok_pos[t];
  T* dst = cache + kv_row_offset(kv, seq, pos, 0);
  for (int i = lane; i < C; i += 32) dst[i] = from_f32<T>(wc[i] * (c[i] * sc));
  rotate_part<T>(c + C, dst + C, R, inv_freq, rot_dims, pairing, amplitude, pos, lane, 32);
}

// q (type T) [T, H, D + R] holds every head's plain part and its part to rotate; qa [T, H, C + R] receives the
// rotated part behind the C entries that the folded key expansion fills.
template <typename T>
__global__ void __launch_bounds__(256)
latent_q_rotate_kernel(const T* __restrict__ q, long ldq, int D, T* __restrict__ qa, long ldqa, int C, int R, int H,
                       const float* __restrict__ inv_freq, int rot_dims, const int32_t* __restrict__ tok_seq,
                       const int32_t* __restrict__ tok_pos, int n_tokens, int pairing, float amplitude) {
  pdl_launch_dependents();
  pdl_wait();
  const int half = rot_dims / 2 + (R - rot_dims + 1) / 2;      // the pairs that turn, then the rest two by two
  const size_t total = (size_t)n_tokens * H * half;
  for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (size_t)gridDim.x * blockDim.x) {
    const int i = (int)(idx % half);
    const int h = (int)((idx / half) % H);
    const int t = (int)(idx / ((size_t)half * H));
    const T* src = q + (size_t)t * ldq + (size_t)h * (D + R) + D;
    T* dst = qa + (size_t)t * ldqa + (size_t)h * (C + R) + C;
    int a = rot_dims + 2 * (i - rot_dims / 2), b = a + 1;
    if (i < rot_dims / 2) pair_places(i, rot_dims, pairing, a, b);
    if (tok_seq[t] < 0) {
      dst[a] = from_f32<T>(0.f);
      if (b < R) dst[b] = from_f32<T>(0.f);
      continue;
    }
    if (i < rot_dims / 2) {
      float s, co;
      sincosf((float)tok_pos[t] * inv_freq[i], &s, &co);
      s *= amplitude;
      co *= amplitude;
      const float u = to_f32(src[a]), v = to_f32(src[b]);
      dst[a] = from_f32<T>(rot_lo(u, v, co, s));
      dst[b] = from_f32<T>(rot_hi(u, v, co, s));
    } else {
      dst[a] = src[a];
      if (b < R) dst[b] = src[b];
    }
  }
}

constexpr int LAT_WARPS = 8;

// One block per (token, group of LAT_WARPS heads), one warp per head.  Keys are taken 32 at a time, in blocks anchored
// at positions 0, 32, 64, ..., staged once in shared memory (fp32) for all heads of the block: lane = key for the
// scores, lane = column for the context.  The order of every addition depends only on the key's position, so the
// result does not depend on how a prompt was cut or batched.  NJ = ceil(C / 32).
template <typename T, int NJ>
__global__ void __launch_bounds__(LAT_WARPS * 32)
attention_latent_kernel(const T* __restrict__ qa, long ldq, T* __restrict__ out, long ldo, const T* __restrict__ cache,
                        const int32_t* __restrict__ tok_seq, const int32_t* __restrict__ tok_pos, PagedKV kv, int n_heads,
                        int C, float scale, int window) {
  extern __shared__ float smem[];
  pdl_wait();
  pdl_launch_dependents();
  const int Dk = kv.head_dim;
  const int kstride = Dk | 1;                                 // odd: lanes on different keys hit different banks
  float* q_s = smem;                                          // [LAT_WARPS][Dk]
  float* k_s = smem + LAT_WARPS * Dk;                         // [32][kstride]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x, h = blockIdx.y * LAT_WARPS + warp;
  const bool head_ok = h < n_heads;
  const int seq = tok_seq[t];
  T* o = out + (size_t)t * ldo + (size_t)h * C;
  if (seq < 0) {
    if (head_ok)
      for (int d = lane; d < C; d += 32) o[d] = from_f32<T>(0.f);
    return;
  }
  const int pos = tok_pos[t];
  if (head_ok) {
    const T* qp = qa + (size_t)t * ldq + (size_t)h * Dk;
    for (int d = lane; d < Dk; d += 32) q_s[warp * Dk + d] = to_f32(qp[d]);
  }
  float m = -INFINITY, l = 0.f;
  float acc[NJ];
#pragma unroll
  for (int j = 0; j < NJ; ++j) acc[j] = 0.f;

  const int lo = first_visible(pos, window, 0);
  for (int c0 = lo / 32 * 32; c0 <= pos; c0 += 32) {
    __syncthreads();                                          // the block before is read out (and q_s is written)
    const int n_rows = (pos - c0 + 1 < 32) ? pos - c0 + 1 : 32;
    for (int r = warp; r < n_rows; r += LAT_WARPS) {
      if (c0 + r < lo) {                                      // (before the window: its page may be gone)
        for (int d = lane; d < Dk; d += 32) k_s[r * kstride + d] = 0.f;
        continue;
      }
      const T* kr = cache + kv_row_offset(kv, seq, c0 + r, 0);
      for (int d = lane; d < Dk; d += 32) k_s[r * kstride + d] = to_f32(kr[d]);
    }
    __syncthreads();
    if (!head_ok) continue;
    const bool valid = lane < n_rows && c0 + lane >= lo;
    float score = -INFINITY;
    if (valid) {
      const float* kq = k_s + lane * kstride;
      const float* qq = q_s + warp * Dk;
      float a = 0.f;
      for (int d = 0; d < Dk; ++d) a = fmaf(qq[d], kq[d], a);
      score = a * scale;
    }
    const float m_new = fmaxf(m, warp_max(score));
    const float p = valid ? expf(score - m_new) : 0.f;
    const float corr = expf(m - m_new);                       // first block: exp(-inf) = 0
    l = l * corr + warp_sum(p);
#pragma unroll
    for (int j = 0; j < NJ; ++j) acc[j] *= corr;
    for (int kk = 0; kk < n_rows; ++kk) {
      const float pk = __shfl_sync(0xffffffffu, p, kk);
      const float* vr = k_s + kk * kstride;
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        const int d = lane + 32 * j;
        if (d < C) acc[j] = fmaf(pk, vr[d], acc[j]);
      }
    }
    m = m_new;
  }
  if (!head_ok) return;
  const float inv = 1.0f / l;
#pragma unroll
  for (int j = 0; j < NJ; ++j) {
    const int d = lane + 32 * j;
    if (d < C) o[d] = from_f32<T>(acc[j] * inv);
  }
}

template <typename T, int NJ>
int launch_attention_latent_nj(const void* qa, long ldq, void* out, long ldo, const void* cache, const int32_t* tok_seq,
                               const int32_t* tok_pos, PagedKV kv, int n_tokens, int n_heads, int C, float scale,
                               int window, cudaStream_t stream) {
  const size_t smem = ((size_t)LAT_WARPS * kv.head_dim + 32 * (size_t)(kv.head_dim | 1)) * sizeof(float);
  static PerDevice<size_t> allowed;
  if (smem > 48 * 1024 && allowed.here() < smem) {
    if (cudaFuncSetAttribute(attention_latent_kernel<T, NJ>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
      return LLMI_ERR_BAD_SIZE;
    allowed.here() = smem;
  }
  dim3 grid(n_tokens, (n_heads + LAT_WARPS - 1) / LAT_WARPS);
  return launch_pdl(PDL_ATTENTION, attention_latent_kernel<T, NJ>, grid, dim3(LAT_WARPS * 32), smem, stream, (const T*)qa, ldq,
                    (T*)out, ldo, (const T*)cache, tok_seq, tok_pos, kv, n_heads, C, scale, window);
}

template <typename T>
int launch_attention_latent(const void* qa, long ldq, void* out, long ldo, const void* cache, const int32_t* tok_seq,
                            const int32_t* tok_pos, PagedKV kv, int n_tokens, int n_heads, int C, float scale,
                            int window, cudaStream_t stream) {
  const int nj = (C + 31) / 32;
#define LLMI_LAT(NJ) \
  return launch_attention_latent_nj<T, NJ>(qa, ldq, out, ldo, cache, tok_seq, tok_pos, kv, n_tokens, n_heads, C, scale, window, stream)
  if (nj <= 1) LLMI_LAT(1);
  if (nj <= 2) LLMI_LAT(2);
  if (nj <= 4) LLMI_LAT(4);
  if (nj <= 8) LLMI_LAT(8);
  if (nj <= 16) LLMI_LAT(16);
  if (nj <= 32) LLMI_LAT(32);
#undef LLMI_LAT
  return LLMI_ERR_BAD_SIZE;
}

}  // namespace llmi

using namespace llmi;

LLMI_EXPORT int llmi_latent_prepare(int dtype, const float* down, long ld, int Q, int C, int R, const float* wq,
                                    const float* wc, float eps, const float* inv_freq, int rot_dims,
                                    const int32_t* tok_seq, const int32_t* tok_pos, const int32_t* seq_pages,
                                    int pages_stride, int page_size, void* cache, void* cq, int n_tokens, int write_kv,
                                    int pairing, float amplitude, cudaStream_t stream) {
  if (n_tokens <= 0 || Q <= 0 || C <= 0 || R < 0 || rot_dims < 0 || rot_dims > R || (rot_dims & 1)) return LLMI_ERR_BAD_SIZE;
  PagedKV kv{seq_pages, pages_stride, page_size, 1, C + R};
  if (dtype == LLMI_DTYPE_F32)
    return launch_pdl(PDL_ROPE, latent_prepare_kernel<float>, dim3(n_tokens, write_kv ? 2 : 1), dim3(LP_THREADS), 0, stream, down, ld, Q, C, R, wq, wc, eps, inv_freq,
                      rot_dims, tok_seq, tok_pos, kv, (float*)cache, (float*)cq, write_kv, pairing, amplitude);
  if (dtype == LLMI_DTYPE_BF16)
    return launch_pdl(PDL_ROPE, latent_prepare_kernel<__nv_bfloat16>, dim3(n_tokens, write_kv ? 2 : 1), dim3(LP_THREADS), 0, stream, down, ld, Q, C, R, wq, wc, eps,
                      inv_freq, rot_dims, tok_seq, tok_pos, kv, (__nv_bfloat16*)cache, (__nv_bfloat16*)cq, write_kv, pairing, amplitude);
  return LLMI_ERR_BAD_DTYPE;
}

// proj fp32 [T, ld] = [ q: H * (D + R) | c: C | r: R ]; qn [T, H * D] contiguous, qa [T, H * (C + R)] (row pitch ldqa): the
// C leading entries of every head's row are left to the folded key expansion.
LLMI_EXPORT int llmi_latent_prepare_direct(int dtype, const float* proj, long ld, int H, int D, int C, int R, const float* wc,
                                           float eps, const float* inv_freq, int rot_dims, int pairing, const int32_t* tok_seq,
                                           const int32_t* tok_pos, const int32_t* seq_pages, int pages_stride, int page_size,
                                           void* cache, void* qn, void* qa, long ldqa, int n_tokens, int write_kv, float amplitude,
                                           cudaStream_t stream) {
  if (n_tokens <= 0 || H <= 0 || D <= 0 || C <= 0 || R < 0 || rot_dims < 0 || rot_dims > R || (rot_dims & 1) || page_size <= 0)
    return LLMI_ERR_BAD_SIZE;
  PagedKV kv{seq_pages, pages_stride, page_size, 1, C + R};
  const long blocks = ((long)n_tokens * (H + 1) + LP_WARPS - 1) / LP_WARPS;
  if (blocks > 0x7fffffffL) return LLMI_ERR_BAD_SIZE;
  if (dtype == LLMI_DTYPE_F32)
    return launch_pdl(PDL_ROPE, latent_prepare_direct_kernel<float>, dim3((unsigned)blocks), dim3(LP_WARPS * 32), 0, stream, proj, ld, H, D,
                      C, R, wc, eps, inv_freq, rot_dims, pairing, tok_seq, tok_pos, kv, (float*)cache, (float*)qn, (float*)qa, ldqa,
                      n_tokens, write_kv, amplitude);
  if (dtype == LLMI_DTYPE_BF16)
    return launch_pdl(PDL_ROPE, latent_prepare_direct_kernel<__nv_bfloat16>, dim3((unsigned)blocks), dim3(LP_WARPS * 32), 0, stream, proj,
                      ld, H, D, C, R, wc, eps, inv_freq, rot_dims, pairing, tok_seq, tok_pos, kv, (__nv_bfloat16*)cache,
                      (__nv_bfloat16*)qn, (__nv_bfloat16*)qa, ldqa, n_tokens, write_kv, amplitude);
  return LLMI_ERR_BAD_DTYPE;
}

LLMI_EXPORT int llmi_latent_q_rotate(int dtype, const void* q, long ldq, int D, void* qa, long ldqa, int C, int R, int H,
                                     const float* inv_freq, int rot_dims, const int32_t* tok_seq, const int32_t* tok_pos,
                                     int n_tokens, int pairing, float amplitude, cudaStream_t stream) {
  if (n_tokens <= 0 || H <= 0 || D < 0 || C <= 0 || R < 0 || rot_dims > R || (rot_dims & 1)) return LLMI_ERR_BAD_SIZE;
  if (R == 0) return LLMI_OK;
  const size_t total = (size_t)n_tokens * H * (rot_dims / 2 + (R - rot_dims + 1) / 2);
  const size_t most = (size_t)sm_count() * 16, need = (total + 255) / 256;
  const int blocks = (int)(need < most ? need : most);
  if (dtype == LLMI_DTYPE_F32)
    return launch_pdl(PDL_SMALL, latent_q_rotate_kernel<float>, blocks, 256, 0, stream, (const float*)q, ldq, D, (float*)qa, ldqa, C,
                      R, H, inv_freq, rot_dims, tok_seq, tok_pos, n_tokens, pairing, amplitude);
  if (dtype == LLMI_DTYPE_BF16)
    return launch_pdl(PDL_SMALL, latent_q_rotate_kernel<__nv_bfloat16>, blocks, 256, 0, stream, (const __nv_bfloat16*)q, ldq, D,
                      (__nv_bfloat16*)qa, ldqa, C, R, H, inv_freq, rot_dims, tok_seq, tok_pos, n_tokens, pairing, amplitude);
  return LLMI_ERR_BAD_DTYPE;
}

// window > 0: the query at position p sees the last `window` positions only (p - window + 1 .. p).
// qa [T, H, C + R] (row pitch ldq), out [T, H, C] (row pitch ldo), cache: the layer's pages [page][1][page_size][C + R].
LLMI_EXPORT int llmi_attention_latent(int dtype, const void* qa, long ldq, void* out, long ldo, const void* cache,
                                      const int32_t* tok_seq, const int32_t* tok_pos, const int32_t* seq_pages,
                                      int pages_stride, int page_size, int n_tokens, int n_heads, int C, int R, float scale,
                                      int window, cudaStream_t stream) {
  if (n_tokens <= 0 || n_heads <= 0 || C <= 0 || R < 0 || page_size <= 0 || window < 0) return LLMI_ERR_BAD_SIZE;
  if (n_tokens > 0x7fffffff || (n_heads + LAT_WARPS - 1) / LAT_WARPS > 65535) return LLMI_ERR_BAD_SIZE;
  PagedKV kv{seq_pages, pages_stride, page_size, 1, C + R};
  if (dtype == LLMI_DTYPE_F32)
    return launch_attention_latent<float>(qa, ldq, out, ldo, cache, tok_seq, tok_pos, kv, n_tokens, n_heads, C, scale, window, stream);
  if (dtype == LLMI_DTYPE_BF16)
    return launch_attention_latent<__nv_bfloat16>(qa, ldq, out, ldo, cache, tok_seq, tok_pos, kv, n_tokens, n_heads, C, scale, window, stream);
  return LLMI_ERR_BAD_DTYPE;
}
