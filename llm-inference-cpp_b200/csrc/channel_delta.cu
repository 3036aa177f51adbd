// The gated delta rule with a decay per key channel, for steps in which every sequence brings ONE token:
//     S <- g S (row d by its own factor g[d]);   u = beta (v - Sᵀ k);   S <- S + k uᵀ;   o = Sᵀ q
// with the conventions of delta_rule.cu (layout of a sequence's state, of a projected row, of a prepared row).  Two kernels
// between the layer's two products:
//   llmi_channel_token_prepare  everything that a token's row needs, as blocks of three kinds in one grid:
//                               a warp per (token, head of q or k) or 128 channels of v: short convolution from the carried
//                               inputs, silu, unit norm, and the carried inputs moved on by one (nobody else reads them);
//                               a warp per token for the write strengths;
//                               a block per 64 outputs of the two low-rank products (decay, output gate) for up to 16 tokens:
//                               fp32 arithmetic, every weight read once per 16 tokens, the decays finished on the spot
//   llmi_channel_token_step     a cluster per (token, head), a block per 32 columns of S: the state is asked for before the
//                               wait on the kernel before; update and read-out in registers; the blocks of a cluster
//                               exchange their sums of squares, then o / rms(o) * w * logistic(gate) leaves in the compute type
// Prompts run the general kernels of delta_rule.cu on the same state.
#include <math.h>

#include "common.cuh"
#include "sm100.cuh"

namespace llmi {

constexpr int CT_THREADS = 256, CT_WARPS = CT_THREADS / 32;
constexpr int CT_V_PIECE = 128;                          // channels of v a warp takes
constexpr int CT_TILE = 64;                              // outputs of a low-rank product a block takes
constexpr int CT_MAX_TAPS = 16;

__device__ __forceinline__ float ct_silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float ct_softplus(float z) { return z > 20.f ? z : log1pf(expf(z)); }

struct ChannelTokenArgs {
  const float* proj;             // [T, ld]: [ q (Hk*D) | k (Hk*D) | v (H*Dv) | b (H) | low ... ]
  long ld;
  int H, Hk, D, Dv, taps;
  int low_a, rank_a, low_g, rank_g;      // where the two low-rank vectors begin in a row, and their sizes
  const float* conv_w;           // [channels, taps]
  const float* a_log;            // [H]
  const float* dt_bias;          // [H*D]
  float* state;                  // [slots, state_floats]
  long state_floats;
  const int32_t *tok_seq, *seq_slot;
  float* prep;                   // [T, ldp]: [ q^ | k^ | v | decay (H*D) | beta (H) ]
  long ldp;
  float* gate;                   // [T, ldg]: the output gate before its logistic function (H*Dv)
  long ldg;
  int n_tokens, write_state;
  int row_blocks;                // blocks of the first two kinds
  int tiles_a, tiles_g;          // 64-wide tiles of the two products
};

// One channel: the convolution over the carried inputs and the current one; the carried inputs move on.
__device__ __forceinline__ float ct_conv(const ChannelTokenArgs& a, const float* row, float* carry, int ch, int Nc) {
  const int K = a.taps;
  const float cur = row[ch];
  const float* w = a.conv_w + (size_t)ch * K;
  float acc = 0.f;
  for (int j = 0; j < K - 1; ++j) {                      // oldest first
    const float x = carry[(size_t)j * Nc + ch];
    acc = fmaf(x, w[j], acc);
    if (a.write_state && j > 0) carry[(size_t)(j - 1) * Nc + ch] = x;
  }
  if (a.write_state && K > 1) carry[(size_t)(K - 2) * Nc + ch] = cur;
  return ct_silu(fmaf(cur, w[K - 1], acc));
}

__device__ __forceinline__ void ct_rows(const ChannelTokenArgs& a, int warp_item, int lane) {
  const int Nc = 2 * a.Hk * a.D + a.H * a.Dv, n_v = a.H * a.Dv;
  const int v_items = (n_v + CT_V_PIECE - 1) / CT_V_PIECE, per = 2 * a.Hk + v_items + 1;
  const int t = warp_item / per, it = warp_item - t * per;
  if (t >= a.n_tokens) return;
  const int seq = a.tok_seq[t];
  if (seq < 0) return;
  const int slot = a.seq_slot[seq];
  if (slot < 0) return;
  const float* row = a.proj + (size_t)t * a.ld;
  float* carry = a.state + (size_t)slot * a.state_floats + (size_t)a.H * a.D * a.Dv;
  float* out = a.prep + (size_t)t * a.ldp;
  if (it < 2 * a.Hk) {
    const int base = it * a.D;
    float ss = 0.f;
    for (int d = lane; d < a.D; d += 32) {
      const float y = ct_conv(a, row, carry, base + d, Nc);
      out[base + d] = y;                                 // (kept here until the scale is known; the same lane comes back)
      ss = fmaf(y, y, ss);
    }
    ss = warp_sum(ss);
    float sc = 1.0f / sqrtf(ss + 1e-6f);
    if (it < a.Hk) sc *= 1.0f / sqrtf((float)a.D);
    for (int d = lane; d < a.D; d += 32) out[base + d] *= sc;
  } else if (it < 2 * a.Hk + v_items) {
    const int c0 = (it - 2 * a.Hk) * CT_V_PIECE, off = 2 * a.Hk * a.D;
    for (int c = c0 + lane; c < min(n_v, c0 + CT_V_PIECE); c += 32) out[off + c] = ct_conv(a, row, carry, off + c, Nc);
  } else {
    for (int h = lane; h < a.H; h += 32) out[Nc + a.H * a.D + h] = 1.0f / (1.0f + expf(-row[Nc + h]));
  }
}

__device__ __forceinline__ float2 ct_pair(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 ct_pair(const __nv_bfloat16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); }

// TG: tokens of a group.  w_a [rank_a, tiles_a * 64], w_g [rank_g, tiles_g * 64]: the second matrices of the two paths,
// transposed, their outputs padded with zeros to whole tiles.
template <typename T, int TG>
__global__ void __launch_bounds__(CT_THREADS)
channel_token_prepare_kernel(const ChannelTokenArgs a, const T* __restrict__ w_a, const T* __restrict__ w_g) {
  extern __shared__ float ct_smem[];
  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if ((int)blockIdx.x < a.row_blocks) {
    pdl_wait();
    ct_rows(a, blockIdx.x * CT_WARPS + warp, lane);
    return;
  }
  // ---- a tile of a low-rank product: warp w takes an eighth of the inner size, a lane two outputs of all tokens
  const int per_group = a.tiles_a + a.tiles_g;
  const int b = blockIdx.x - a.row_blocks, group = b / per_group, tile = b - group * per_group;
  const bool is_gate = tile >= a.tiles_a;
  const int n0 = (is_gate ? tile - a.tiles_a : tile) * CT_TILE;
  const int R = is_gate ? a.rank_g : a.rank_a, at = is_gate ? a.low_g : a.low_a;
  const T* w = is_gate ? w_g : w_a;
  const long ldw = (long)(is_gate ? a.tiles_g : a.tiles_a) * CT_TILE;
  const int t0 = group * TG;
  float* low = ct_smem;                                  // [R][TG]
  float* part = ct_smem + (size_t)R * TG;                // [warps][64][TG + 1]
  const int span = (R + CT_WARPS - 1) / CT_WARPS, r_lo = warp * span, r_hi = min(R, r_lo + span);
  float2 wv[8];                                          // weights wait for nobody: the first eight rows are asked for now
#pragma unroll
  for (int j = 0; j < 8; ++j) wv[j] = r_lo + j < r_hi ? ct_pair(w + (size_t)(r_lo + j) * ldw + n0 + 2 * lane) : make_float2(0.f, 0.f);
  pdl_wait();
  for (int i = threadIdx.x; i < R * TG; i += CT_THREADS) {
    const int tt = i / R, r = i - tt * R;                // neighbouring threads read neighbouring columns
    low[r * TG + tt] = t0 + tt < a.n_tokens ? a.proj[(size_t)(t0 + tt) * a.ld + at + r] : 0.f;
  }
  __syncthreads();
  float2 acc[TG];
#pragma unroll
  for (int t = 0; t < TG; ++t) acc[t] = make_float2(0.f, 0.f);
  for (int r = r_lo; r < r_hi; r += 8) {
    float2 nxt[8];
#pragma unroll
    for (int j = 0; j < 8; ++j)
      nxt[j] = r + 8 + j < r_hi ? ct_pair(w + (size_t)(r + 8 + j) * ldw + n0 + 2 * lane) : make_float2(0.f, 0.f);
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      if (r + j >= r_hi) break;
#pragma unroll
      for (int t = 0; t < TG; ++t) {
        const float l = low[(r + j) * TG + t];
        acc[t].x = fmaf(wv[j].x, l, acc[t].x);
        acc[t].y = fmaf(wv[j].y, l, acc[t].y);
      }
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) wv[j] = nxt[j];
  }
  float* mine = part + (size_t)warp * CT_TILE * (TG + 1);
#pragma unroll
  for (int t = 0; t < TG; ++t) {
    mine[(2 * lane) * (TG + 1) + t] = acc[t].x;
    mine[(2 * lane + 1) * (TG + 1) + t] = acc[t].y;
  }
  __syncthreads();
  const int N = is_gate ? a.H * a.Dv : a.H * a.D, decay_at = 2 * a.Hk * a.D + a.H * a.Dv;
  for (int i = threadIdx.x; i < CT_TILE * TG; i += CT_THREADS) {
    const int t = i / CT_TILE, c = i - t * CT_TILE, n = n0 + c;
    if (t0 + t >= a.n_tokens || n >= N) continue;
    float v = 0.f;
#pragma unroll
    for (int q = 0; q < CT_WARPS; ++q) v += part[((size_t)q * CT_TILE + c) * (TG + 1) + t];      // warps in order
    if (is_gate) a.gate[(size_t)(t0 + t) * a.ldg + n] = v;
    else a.prep[(size_t)(t0 + t) * a.ldp + decay_at + n] = expf(-expf(a.a_log[n / a.D]) * ct_softplus(v + a.dt_bias[n]));
  }
}

template <typename T, int TG>
int launch_channel_prepare(const ChannelTokenArgs& a, const void* w_a, const void* w_g, cudaStream_t stream) {
  const int rank = a.rank_a > a.rank_g ? a.rank_a : a.rank_g;
  const size_t smem = ((size_t)rank * TG + (size_t)CT_WARPS * CT_TILE * (TG + 1)) * sizeof(float);
  static PerDevice<size_t> allowed;
  if (smem > 200 * 1024) return LLMI_ERR_BAD_SIZE;
  if (smem > 48 * 1024 && allowed.here() < smem) {
    if (cudaFuncSetAttribute(channel_token_prepare_kernel<T, TG>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
      return LLMI_ERR_BAD_SIZE;
    allowed.here() = smem;
  }
  const long blocks = a.row_blocks + (long)((a.n_tokens + TG - 1) / TG) * (a.tiles_a + a.tiles_g);
  if (blocks > 0x7fffffffL) return LLMI_ERR_BAD_SIZE;
  return launch_pdl(PDL_SMALL, channel_token_prepare_kernel<T, TG>, dim3((unsigned)blocks), dim3(CT_THREADS), smem, stream, a,
                    (const T*)w_a, (const T*)w_g);
}

// ------------------------------------------------------------------------------------------------

constexpr int CS_COLS = 32;                              // columns of S a block takes

struct ChannelStepArgs {
  const float* prep;             // [T, ldp]: [ q^ | k^ | v | decay (H*D) | beta (H) ]
  long ldp;
  int H, Hk, D, Dv;
  float* state;
  long state_floats;
  const int32_t *tok_seq, *seq_slot;
  const float* gate;             // [T, ldg]
  long ldg;
  const float* w;                // [Dv]
  float eps;
  long ld_out;
  int slices;                    // blocks of a cluster: ceil(Dv / 32)
  int write_state;
};

// LPC lanes share a column (four entries each, NCH times: entries 4 LPC i + 4 sub + 0..3); a pass covers 256 / LPC columns.
template <typename T, int LPC, int NCH>
__global__ void __launch_bounds__(CT_THREADS)
channel_token_step_kernel(const ChannelStepArgs a, T* __restrict__ out) {
  constexpr int CPP = CT_THREADS / LPC, PASSES = CS_COLS / CPP;
  __shared__ float o_s[CS_COLS];
  __shared__ float part_s[8];
  pdl_launch_dependents();
  const int slice = blockIdx.x % a.slices, h = blockIdx.x / a.slices, t = blockIdx.y;
  const int D = a.D, Dv = a.Dv;
  const int seq = a.tok_seq[t];                          // (the step's index block: there before any of its kernels)
  const int slot = seq >= 0 ? a.seq_slot[seq] : -1;
  T* dst = out + (size_t)t * a.ld_out + (size_t)h * Dv + slice * CS_COLS;
  const int n_cols = min(CS_COLS, Dv - slice * CS_COLS);
  if (slot < 0) {                                        // (the same answer in every block of the cluster)
    pdl_wait();
    if ((int)threadIdx.x < n_cols) dst[threadIdx.x] = from_f32<T>(0.f);
    return;
  }
  const int sub = threadIdx.x % LPC, cg = threadIdx.x / LPC;
  float* S_g = a.state + (size_t)slot * a.state_floats + ((size_t)h * Dv + slice * CS_COLS) * D;
  float4 S[PASSES][NCH];
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int p = 0; p < PASSES; ++p)
#pragma unroll
    for (int i = 0; i < NCH; ++i) {
      const int d = 4 * LPC * i + 4 * sub, c = p * CPP + cg;
      S[p][i] = (d < D && c < n_cols) ? *reinterpret_cast<const float4*>(S_g + (size_t)c * D + d) : zero;
    }
  pdl_wait();
  const float* row = a.prep + (size_t)t * a.ldp;
  const int kh = h / (a.H / a.Hk), Nc = 2 * a.Hk * D + a.H * Dv;
  const float* q_r = row + (size_t)kh * D;
  const float* k_r = row + (size_t)a.Hk * D + (size_t)kh * D;
  const float* v_r = row + (size_t)2 * a.Hk * D + (size_t)h * Dv + slice * CS_COLS;
  const float* g_r = row + Nc + (size_t)h * D;
  const float beta = row[Nc + a.H * D + h];
  float4 k[NCH], q[NCH];
#pragma unroll
  for (int i = 0; i < NCH; ++i) {
    const int d = 4 * LPC * i + 4 * sub;
    k[i] = d < D ? *reinterpret_cast<const float4*>(k_r + d) : zero;
    q[i] = d < D ? *reinterpret_cast<const float4*>(q_r + d) : zero;
    const float4 g = d < D ? *reinterpret_cast<const float4*>(g_r + d) : zero;
#pragma unroll
    for (int p = 0; p < PASSES; ++p) {
      S[p][i].x *= g.x; S[p][i].y *= g.y; S[p][i].z *= g.z; S[p][i].w *= g.w;
    }
  }
  float sk[PASSES], o[PASSES];
#pragma unroll
  for (int p = 0; p < PASSES; ++p) {
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < NCH; ++i)
      s = fmaf(S[p][i].x, k[i].x, fmaf(S[p][i].y, k[i].y, fmaf(S[p][i].z, k[i].z, fmaf(S[p][i].w, k[i].w, s))));
    sk[p] = s;
  }
#pragma unroll
  for (int x = 1; x < LPC; x <<= 1)
#pragma unroll
    for (int p = 0; p < PASSES; ++p) sk[p] += __shfl_xor_sync(0xffffffffu, sk[p], x);
#pragma unroll
  for (int p = 0; p < PASSES; ++p) {
    const int c = p * CPP + cg;
    const float u = c < n_cols ? beta * (v_r[c] - sk[p]) : 0.f;
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < NCH; ++i) {
      float4& z = S[p][i];
      z.x = fmaf(k[i].x, u, z.x);
      z.y = fmaf(k[i].y, u, z.y);
      z.z = fmaf(k[i].z, u, z.z);
      z.w = fmaf(k[i].w, u, z.w);
      s = fmaf(z.x, q[i].x, fmaf(z.y, q[i].y, fmaf(z.z, q[i].z, fmaf(z.w, q[i].w, s))));
      const int d = 4 * LPC * i + 4 * sub;
      if (a.write_state && d < D && c < n_cols) *reinterpret_cast<float4*>(S_g + (size_t)c * D + d) = z;
    }
    o[p] = s;
  }
#pragma unroll
  for (int x = 1; x < LPC; x <<= 1)
#pragma unroll
    for (int p = 0; p < PASSES; ++p) o[p] += __shfl_xor_sync(0xffffffffu, o[p], x);
  if (sub == 0) {
#pragma unroll
    for (int p = 0; p < PASSES; ++p) o_s[p * CPP + cg] = o[p];          // (columns beyond the head's hold zeros)
  }
  __syncthreads();
  float ss = 0.f, mine = 0.f;
  if (threadIdx.x < 32) {
    mine = o_s[threadIdx.x];
    ss = warp_sum(mine * mine);
  }
  if (a.slices > 1) {
    // every block leaves its sum with every block of the cluster; all are there behind the barrier, and nobody touches
    // another block's memory after it
    if ((int)threadIdx.x < a.slices) st_cluster_f32(map_to_rank(smem_u32(&part_s[slice]), threadIdx.x), ss);
    cluster_sync_all();
    ss = 0.f;
    for (int r = 0; r < a.slices; ++r) ss += part_s[r];
  }
  if ((int)threadIdx.x < n_cols) {
    const float sc = 1.0f / sqrtf(ss / (float)Dv + a.eps);
    const int c = slice * CS_COLS + threadIdx.x;
    const float z = a.gate[(size_t)t * a.ldg + (size_t)h * Dv + c];
    dst[threadIdx.x] = from_f32<T>(a.w[c] * (mine * sc) * (1.0f / (1.0f + expf(-z))));
  }
}

template <typename T, int LPC, int NCH>
int launch_channel_step(const ChannelStepArgs& a, void* out, int n_tokens, cudaStream_t stream) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3((unsigned)(a.H * a.slices), (unsigned)n_tokens);
  cfg.blockDim = dim3(CT_THREADS);
  cfg.stream = stream;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = pdl_enabled(PDL_ATTENTION) ? 1 : 0;
  attr[1].id = cudaLaunchAttributeClusterDimension;
  attr[1].val.clusterDim.x = (unsigned)a.slices;
  attr[1].val.clusterDim.y = 1;
  attr[1].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = a.slices > 1 ? 2 : 1;
  pairs_may_start_early = false;
  return cudaLaunchKernelEx(&cfg, channel_token_step_kernel<T, LPC, NCH>, a, (T*)out) == cudaSuccess ? LLMI_OK : LLMI_ERR_LAUNCH;
}

template <typename T>
int launch_channel_step_sizes(const ChannelStepArgs& a, void* out, int n_tokens, cudaStream_t stream) {
  if (a.D <= 32) return launch_channel_step<T, 8, 1>(a, out, n_tokens, stream);
  if (a.D <= 64) return launch_channel_step<T, 16, 1>(a, out, n_tokens, stream);
  if (a.D <= 128) return launch_channel_step<T, 32, 1>(a, out, n_tokens, stream);
  return launch_channel_step<T, 32, 2>(a, out, n_tokens, stream);
}

// rows of fp32 into the compute type, a slice of wider rows
template <typename T>
__global__ void __launch_bounds__(256)
cast_rows_kernel(const float* __restrict__ src, long lds, T* __restrict__ out, int n, size_t total) {
  pdl_launch_dependents();
  pdl_wait();
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
    const size_t t = i / n;
    out[i] = from_f32<T>(src[t * lds + (i - t * n)]);
  }
}

}  // namespace llmi

using namespace llmi;

// Sizes the single-token kernels take: 16-byte pieces of a column, one cluster of at most eight blocks per head.
LLMI_EXPORT int llmi_channel_token_supported(int H, int Hk, int D, int Dv, int taps, int rank_a, int rank_g) {
  return H > 0 && Hk > 0 && H % Hk == 0 && D > 0 && D % 4 == 0 && D <= 256 && Dv > 0 && Dv % 4 == 0 && Dv <= 256 && taps >= 1 &&
         taps <= CT_MAX_TAPS && rank_a > 0 && rank_g > 0 && rank_a <= 1024 && rank_g <= 1024;
}

// w_a [rank_a, Na], w_g [rank_g, Ng] (dtype's type), Na and Ng = H*D and H*Dv rounded up to 64, zeros behind.
LLMI_EXPORT int llmi_channel_token_prepare(int dtype, const float* proj, long ld, int H, int Hk, int D, int Dv, int taps, int low_a,
                                           int rank_a, int low_g, int rank_g, const float* conv_w, const float* a_log,
                                           const float* dt_bias, float* state, const int32_t* tok_seq, const int32_t* seq_slot,
                                           const void* w_a, const void* w_g, float* prep, long ldp, float* gate, long ldg,
                                           int n_tokens, int write_state, cudaStream_t stream) {
  if (n_tokens <= 0 || !llmi_channel_token_supported(H, Hk, D, Dv, taps, rank_a, rank_g)) return LLMI_ERR_BAD_SIZE;
  if (((uintptr_t)w_a & 7) || ((uintptr_t)w_g & 7)) return LLMI_ERR_ALIGN;
  ChannelTokenArgs a;
  a.proj = proj; a.ld = ld; a.H = H; a.Hk = Hk; a.D = D; a.Dv = Dv; a.taps = taps;
  a.low_a = low_a; a.rank_a = rank_a; a.low_g = low_g; a.rank_g = rank_g;
  a.conv_w = conv_w; a.a_log = a_log; a.dt_bias = dt_bias;
  a.state = state;
  a.state_floats = (long)H * D * Dv + (long)(taps - 1) * (2 * Hk * D + H * Dv);
  a.tok_seq = tok_seq; a.seq_slot = seq_slot; a.prep = prep; a.ldp = ldp; a.gate = gate; a.ldg = ldg;
  a.n_tokens = n_tokens; a.write_state = write_state;
  const long items = (long)n_tokens * (2 * Hk + (H * Dv + CT_V_PIECE - 1) / CT_V_PIECE + 1);
  if (items > 0x3fffffffL) return LLMI_ERR_BAD_SIZE;
  a.row_blocks = (int)((items + CT_WARPS - 1) / CT_WARPS);
  a.tiles_a = (H * D + CT_TILE - 1) / CT_TILE;
  a.tiles_g = (H * Dv + CT_TILE - 1) / CT_TILE;
  if (dtype == LLMI_DTYPE_F32) {
    if (n_tokens <= 4) return launch_channel_prepare<float, 4>(a, w_a, w_g, stream);
    if (n_tokens <= 8) return launch_channel_prepare<float, 8>(a, w_a, w_g, stream);
    return launch_channel_prepare<float, 16>(a, w_a, w_g, stream);
  }
  if (dtype == LLMI_DTYPE_BF16) {
    if (n_tokens <= 4) return launch_channel_prepare<__nv_bfloat16, 4>(a, w_a, w_g, stream);
    if (n_tokens <= 8) return launch_channel_prepare<__nv_bfloat16, 8>(a, w_a, w_g, stream);
    return launch_channel_prepare<__nv_bfloat16, 16>(a, w_a, w_g, stream);
  }
  return LLMI_ERR_BAD_DTYPE;
}

LLMI_EXPORT int llmi_channel_token_step(int dtype, const float* prep, long ldp, int H, int Hk, int D, int Dv, int taps, float* state,
                                        const int32_t* tok_seq, const int32_t* seq_slot, const float* gate, long ldg, const float* w,
                                        float eps, void* out, long ld_out, int n_tokens, int write_state, cudaStream_t stream) {
  if (n_tokens <= 0 || n_tokens > 65535 || !llmi_channel_token_supported(H, Hk, D, Dv, taps, 1, 1)) return LLMI_ERR_BAD_SIZE;
  ChannelStepArgs a;
  a.prep = prep; a.ldp = ldp; a.H = H; a.Hk = Hk; a.D = D; a.Dv = Dv; a.state = state;
  a.state_floats = (long)H * D * Dv + (long)(taps - 1) * (2 * Hk * D + H * Dv);
  if (((uintptr_t)prep & 15) || ((uintptr_t)state & 15) || ldp % 4 || a.state_floats % 4) return LLMI_ERR_ALIGN;
  a.tok_seq = tok_seq; a.seq_slot = seq_slot; a.gate = gate; a.ldg = ldg; a.w = w; a.eps = eps; a.ld_out = ld_out;
  a.slices = (Dv + CS_COLS - 1) / CS_COLS;
  a.write_state = write_state;
  if (dtype == LLMI_DTYPE_F32) return launch_channel_step_sizes<float>(a, out, n_tokens, stream);
  if (dtype == LLMI_DTYPE_BF16) return launch_channel_step_sizes<__nv_bfloat16>(a, out, n_tokens, stream);
  return LLMI_ERR_BAD_DTYPE;
}

// out [n_tokens, n] (contiguous, dtype's type) = src (fp32, row pitch lds)
LLMI_EXPORT int llmi_cast_rows(int dtype, const float* src, long lds, void* out, int n_tokens, int n, cudaStream_t stream) {
  if (n_tokens <= 0 || n <= 0) return LLMI_ERR_BAD_SIZE;
  const size_t total = (size_t)n_tokens * n, most = (size_t)sm_count() * 16, want = (total + 255) / 256;
  const int blocks = (int)(want < most ? want : most);
  if (dtype == LLMI_DTYPE_F32) return launch_pdl(PDL_SMALL, cast_rows_kernel<float>, blocks, 256, 0, stream, src, lds, (float*)out, n, total);
  if (dtype == LLMI_DTYPE_BF16)
    return launch_pdl(PDL_SMALL, cast_rows_kernel<__nv_bfloat16>, blocks, 256, 0, stream, src, lds, (__nv_bfloat16*)out, n, total);
  return LLMI_ERR_BAD_DTYPE;
}
