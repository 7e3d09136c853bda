// Latent attention: keys and values of all heads are linear images of one cached vector c per token,
//   k_h = Wk_h c,  v_h = Wv_h c,   so   q_h . k_h = (Wk_h^T q_h) . c   and   sum_j p_j v_hj = Wv_h (sum_j p_j c_j).
// The cache holds only c ([slots, rank], paged). For few query tokens the products with Wk and Wv are taken on the query
// side ("absorbed"), which turns the op into multi-query attention of H heads over one shared key = value row:
//   latent_prep       RMS norm of the down-projected row, written to the cache slot of its token; squared-relu of the
//                     feed-forward's up-projection, which sits in the same GEMM output
//   head_linear       y[t, h, :] = W[h] x[t, h, :]  (per-head GEMM: Wk^T on the query, Wv on the attended latent); optionally
//                     of tanh(x), the second half of a low-rank map with a tanh in the middle
//   attention over the paged latents, which serve as keys and as values: latent_decode_sm100.cu (split-KV partial results)
//   latent_combine    merges the splits; a per-head sink logit joins the softmax denominator here, once
//   latent_attention_plain   one warp per row, any rank, any storage type (the 32-bit mode and shapes outside the above)
// Many query tokens go through prefill_attn_sm100.cu on expanded keys and values instead.
//
// Causality: query token i of the S tokens a sequence brings attends the keys j <= kv_len - S + i.
#include "b200/attn_merge.cuh"
#include "b200/elem.cuh"
#include "b200/host.h"
#include "b200/mma_sync.cuh"

#include <cstring>
#include <type_traits>

namespace b200 {

// ------------------------------------------------------------------------------------------------ latent_prep
struct PrepParams {
  const void* latent_in;   // [T, rank] (row pitch ld); null: no latent part
  const void* gain;        // [pitch]
  void* cache;             // [slots, pitch]
  const long long* slots;  // [T], < 0 = not stored
  int rank, pitch;
  float eps;
  const void* up;          // [T, inter] (row pitch ld); null: no activation part
  void* act;               // [T, inter]
  int inter, ld;
};

// grid (T, parts): part 0 normalises the latent row, the others take 1024 columns of the activation each
template <typename T>
__global__ void __launch_bounds__(256) latent_prep_kernel(const PrepParams p) {
  __shared__ float red[8];
  const size_t t = blockIdx.x;
  const int has_latent = p.latent_in != nullptr ? 1 : 0;
  griddep_launch_dependents();
  griddep_wait();
  if (has_latent && blockIdx.y == 0) {
    const T* src = static_cast<const T*>(p.latent_in) + t * p.ld;
    float ss = 0.f;
    for (int i = threadIdx.x; i < p.rank; i += blockDim.x) {
      const float v = to_float(src[i]);
      ss += v * v;
    }
    ss = warp_sum(ss);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    float tot = 0.f;
    for (int w = 0; w < static_cast<int>(blockDim.x >> 5); ++w) tot += red[w];
    const float inv = 1.f / sqrtf(tot / p.rank + p.eps);
    const long long slot = p.slots[t];
    if (slot < 0) return;
    T* dst = static_cast<T*>(p.cache) + static_cast<size_t>(slot) * p.pitch;
    for (int i = threadIdx.x; i < p.pitch; i += blockDim.x)
      dst[i] = from_float<T>(i < p.rank ? to_float(src[i]) * inv * to_float(static_cast<const T*>(p.gain)[i]) : 0.f);
    return;
  }
  const int c = (blockIdx.y - has_latent) * 1024 + threadIdx.x * 4;
  if (p.up != nullptr && c < p.inter) {
    float4 v = load4(static_cast<const T*>(p.up) + t * p.ld + c);
    v.x = fmaxf(v.x, 0.f); v.y = fmaxf(v.y, 0.f); v.z = fmaxf(v.z, 0.f); v.w = fmaxf(v.w, 0.f);
    store4(static_cast<T*>(p.act) + t * p.inter + c, make_float4(v.x * v.x, v.y * v.y, v.z * v.z, v.w * v.w));
  }
}

// ------------------------------------------------------------------------------------------------ head_linear
struct HeadLinearParams {
  const void* x;    // x[t * ldx + h * xh + k]
  const void* w;    // [H, N, K]
  void* y;          // y[t * ldy + h * yh + n]
  int T, H, N, K;
  long long ldx, xh, ldy, yh;
};

enum HeadLinearAct : int { kActNone = 0, kActTanh = 1 };   // applied to x on its way into the product
template <bool BF16>
__device__ __forceinline__ uint32_t tanh_pair(uint32_t v) {
  const float2 f = BF16 ? unpack_bf16x2(v) : unpack_f16x2(v);
  const float x = tanh_t<__half>(f.x), y = tanh_t<__half>(f.y);   // the same for both 16-bit types
  return BF16 ? pack_bf16x2(x, y) : pack_f16x2(x, y);
}

constexpr int kHlTok = 4;  // token tiles of 8 per CTA

// 16-bit: CTA = one head, 128 / KS output rows, 8 * kHlTok tokens. A warp multiplies 16 rows of W by the tokens over its K
// slice; KS warps share the rows and add their partial sums through shared memory. Both fragments are read straight from
// global memory: a lane takes 8 consecutive k per 32-wide step (one 16-byte load per row), which permutes k inside the
// step the same way for both operands and leaves the sum over k unchanged.
template <bool BF16, int KS, int kAct>
__global__ void __launch_bounds__(256) head_linear_kernel(const HeadLinearParams p) {
  constexpr int kRows = 128 / KS;
  __shared__ float part[KS > 1 ? KS - 1 : 1][kRows / 16][32][kHlTok * 4];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, tq = lane & 3;
  const int h = blockIdx.y, rg = warp / KS, ks = warp - rg * KS;
  const int n0 = blockIdx.x * kRows + rg * 16, t0 = blockIdx.z * 8 * kHlTok;
  const int kper = ((p.K + KS - 1) / KS + 31) / 32 * 32;
  const int k_begin = ks * kper, k_end = min(p.K, k_begin + kper);
  const uint16_t* w = static_cast<const uint16_t*>(p.w) + static_cast<size_t>(h) * p.N * p.K;
  const uint16_t* x = static_cast<const uint16_t*>(p.x) + h * p.xh;
  const uint4 zero = make_uint4(0, 0, 0, 0);
  griddep_launch_dependents();
  uint4 w0[4], w1[4];
  auto load_w = [&](int kc) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int k = kc + 32 * i + 8 * tq;
      w0[i] = (k < k_end && n0 + g < p.N) ? ld_v4_nc(w + static_cast<size_t>(n0 + g) * p.K + k) : zero;
      w1[i] = (k < k_end && n0 + g + 8 < p.N) ? ld_v4_nc(w + static_cast<size_t>(n0 + g + 8) * p.K + k) : zero;
    }
  };
  load_w(k_begin);  // weights: read before the dependency wait
  griddep_wait();
  float acc[kHlTok][4] = {};
  for (int kc = k_begin; kc < k_end; kc += 128) {
    if (kc != k_begin) load_w(kc);
#pragma unroll
    for (int j = 0; j < kHlTok; ++j) {
      const int t = t0 + 8 * j + g;
      if (t0 + 8 * j >= p.T) break;
      uint4 xv[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int k = kc + 32 * i + 8 * tq;
        xv[i] = (k < k_end && t < p.T) ? *reinterpret_cast<const uint4*>(x + t * p.ldx + k) : zero;
        if (kAct == kActTanh)
          xv[i] = make_uint4(tanh_pair<BF16>(xv[i].x), tanh_pair<BF16>(xv[i].y), tanh_pair<BF16>(xv[i].z), tanh_pair<BF16>(xv[i].w));
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const uint32_t a0[4] = {w0[i].x, w1[i].x, w0[i].y, w1[i].y}, a1[4] = {w0[i].z, w1[i].z, w0[i].w, w1[i].w};
        mma16816<BF16>(acc[j], a0, xv[i].x, xv[i].y);
        mma16816<BF16>(acc[j], a1, xv[i].z, xv[i].w);
      }
    }
  }
  if (KS > 1) {
    if (ks > 0) {
#pragma unroll
      for (int j = 0; j < kHlTok; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) part[ks - 1][rg][lane][j * 4 + e] = acc[j][e];
    }
    __syncthreads();
    if (ks > 0) return;
#pragma unroll
    for (int s = 0; s < KS - 1; ++s)
#pragma unroll
      for (int j = 0; j < kHlTok; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[j][e] += part[s][rg][lane][j * 4 + e];
  }
  using T = typename std::conditional<BF16, __nv_bfloat16, __half>::type;
  T* y = static_cast<T*>(p.y) + h * p.yh;
#pragma unroll
  for (int j = 0; j < kHlTok; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {  // accumulator element e: row g + 8 * (e / 2), token 2 tq + (e & 1)
      const int n = n0 + g + 8 * (e >> 1), t = t0 + 8 * j + 2 * tq + (e & 1);
      if (n < p.N && t < p.T) y[t * p.ldy + n] = from_float<T>(acc[j][e]);
    }
}

// fp32: one output per thread, the input row in shared memory
template <int kAct>
__global__ void __launch_bounds__(128) head_linear_f32_kernel(const HeadLinearParams p) {
  extern __shared__ float xs[];
  const int t = blockIdx.x, h = blockIdx.y;
  griddep_launch_dependents();
  griddep_wait();
  const float* x = static_cast<const float*>(p.x) + t * p.ldx + h * p.xh;
  for (int k = threadIdx.x; k < p.K; k += blockDim.x) xs[k] = kAct == kActTanh ? tanhf(x[k]) : x[k];
  __syncthreads();
  const float* w = static_cast<const float*>(p.w) + static_cast<size_t>(h) * p.N * p.K;
  for (int n = threadIdx.x; n < p.N; n += blockDim.x) {
    float acc = 0.f;
    for (int k = 0; k < p.K; ++k) acc = fmaf(w[static_cast<size_t>(n) * p.K + k], xs[k], acc);
    static_cast<float*>(p.y)[t * p.ldy + h * p.yh + n] = acc;
  }
}

// ------------------------------------------------------------------------------------------------ attention
struct LatentParams {
  const void* q;           // absorbed queries [B * S * H, pitch]
  const void* cache;       // [blocks, page, pitch]
  const int* block_table;  // [B, bt_stride]
  const int* kv_lens;      // [B] keys in the cache, the S new ones included
  const float* sink;       // [H] or null
  void* out;               // [B * S * H, pitch]
  int bt_stride, page, H, S, pitch;
  float scale;
};

// grid (ceil(pitch / 128), rows): merge of the splits. The sink is one more term exp(sink) of the denominator without a
// value: the merged row is scaled by exp(lse) / (exp(lse) + exp(sink)).
template <typename T>
__global__ void __launch_bounds__(128) latent_combine_kernel(const float* o_part, const float* lse_part, const float* sink, int H,
                                                             int splits, int pitch, T* out) {
  const size_t row = blockIdx.y;
  const int c = blockIdx.x * 128 + threadIdx.x;
  griddep_launch_dependents();
  const float sk = sink != nullptr ? __ldg(sink + row % H) : -CUDART_INF_F;
  griddep_wait();
  if (c >= pitch) return;
  float o, lse;
  merge_splits(lse_part + row * splits, 1, o_part + row * splits * pitch + c, pitch, splits, o, lse);
  out[row * pitch + c] = from_float<T>(o / (1.f + expf(sk - lse)));
}

// One warp per row, keys in groups of 32: a lane scores one key, then the lanes share the columns of the values. The query
// row and the running output live in shared memory, so the rank is limited by shared memory only.
template <typename T>
__global__ void __launch_bounds__(128) latent_attention_plain_kernel(const LatentParams p) {
  extern __shared__ __align__(16) float fsm[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* q = fsm + warp * 2 * p.pitch;
  float* o = q + p.pitch;
  const int b = blockIdx.y, n_rows = p.S * p.H, r = blockIdx.x * 4 + warp;
  griddep_launch_dependents();
  griddep_wait();
  if (r >= n_rows) return;
  const size_t row = static_cast<size_t>(b) * n_rows + r;
  for (int i = lane; i < p.pitch; i += 32) {
    q[i] = to_float(static_cast<const T*>(p.q)[row * p.pitch + i]);
    o[i] = 0.f;
  }
  __syncwarp();
  const int n_keys = min(p.kv_lens[b], p.kv_lens[b] - p.S + r / p.H + 1);
  const int* table = p.block_table + static_cast<size_t>(b) * p.bt_stride;
  const T* cache = static_cast<const T*>(p.cache);
  float m = -INFINITY, l = 0.f;
  for (int j0 = 0; j0 < n_keys; j0 += 32) {
    const int j = j0 + lane;
    const bool in = j < n_keys;
    const T* c = cache + (in ? (static_cast<size_t>(table[j / p.page]) * p.page + j % p.page) : 0) * p.pitch;
    float s = 0.f;
    if (in)
      for (int i = 0; i < p.pitch; i += 4) {
        const float4 v = load4(c + i);
        s = fmaf(v.x, q[i], s); s = fmaf(v.y, q[i + 1], s); s = fmaf(v.z, q[i + 2], s); s = fmaf(v.w, q[i + 3], s);
      }
    s = in ? s * p.scale : -INFINITY;
    const float m_new = fmaxf(m, warp_max(s));
    const float pr = in ? expf(s - m_new) : 0.f;
    const float corr = expf(m - m_new);
    l = l * corr + warp_sum(pr);
    m = m_new;
    const int n = min(32, n_keys - j0);
    for (int i0 = 0; i0 < p.pitch; i0 += 32) {  // uniform over the warp: every lane takes part in the shuffles
      const int i = i0 + lane;
      float acc = i < p.pitch ? o[i] * corr : 0.f;
      for (int k = 0; k < n; ++k) {
        const float w = __shfl_sync(0xffffffffu, pr, k);
        const int jj = j0 + k;
        if (i < p.pitch)
          acc = fmaf(w, to_float(cache[(static_cast<size_t>(table[jj / p.page]) * p.page + jj % p.page) * p.pitch + i]), acc);
      }
      if (i < p.pitch) o[i] = acc;
    }
    __syncwarp();
  }
  if (p.sink != nullptr && n_keys > 0) l += expf(p.sink[r % p.H] - m);
  const float inv = l > 0.f ? 1.f / l : 0.f;
  for (int i = lane; i < p.pitch; i += 32) static_cast<T*>(p.out)[row * p.pitch + i] = from_float<T>(o[i] * inv);
}

}  // namespace b200

using namespace b200;

// latent_in / up: columns of one GEMM output with row pitch ld. Either may be null (that part is left out).
B200_API int b200_latent_prep(const void* latent_in, const void* gain, void* cache, const long long* slots, int rank, int pitch,
                              float eps, const void* up, void* act, int inter, int ld, int rows, int dtype, void* stream) {
  if (rows <= 0 || (latent_in == nullptr && up == nullptr)) return kOk;
  B200_REQUIRE(latent_in == nullptr || (gain && cache && slots && rank >= 1 && pitch >= rank), "latent part: missing arguments");
  B200_REQUIRE(up == nullptr || (act && inter % 4 == 0 && ld % 4 == 0), "activation part: inter (%d) and ld (%d) must be multiples of 4", inter, ld);
  PrepParams p{latent_in, gain, cache, slots, rank, pitch, eps, up, act, inter, ld};
  const dim3 grid(rows, (latent_in ? 1 : 0) + (up ? (inter + 1023) / 1024 : 0));
  B200_DISPATCH_FLOAT(dtype, B200_CHECK_CUDA(launch_pdl(latent_prep_kernel<T>, grid, dim3(256), 0, static_cast<cudaStream_t>(stream), p));
                      return kOk;);
}

template <int kAct>
static int launch_head_linear(const HeadLinearParams& p, int dtype, cudaStream_t s) {
  if (dtype == kF32) {
    B200_REQUIRE(p.K <= 8192, "head_linear: K (%d) is limited to 8192 in fp32", p.K);
    B200_CHECK_CUDA(launch_pdl(head_linear_f32_kernel<kAct>, dim3(p.T, p.H), dim3(128), static_cast<size_t>(p.K) * 4, s, p));
    return kOk;
  }
  B200_REQUIRE(dtype == kBF16 || dtype == kF16, "head_linear supports bf16 / f16 / f32");
  B200_REQUIRE(p.K % 8 == 0 && p.ldx % 8 == 0 && p.xh % 8 == 0, "head_linear: K (%d) and the input strides must be multiples of 8", p.K);
  const int tz = (p.T + 8 * kHlTok - 1) / (8 * kHlTok);
  B200_REQUIRE(tz <= 65535, "head_linear: too many tokens (%d)", p.T);
  const int ks = p.K > 256 ? 4 : p.K > 128 ? 2 : 1;
  const dim3 grid((p.N + 128 / ks - 1) / (128 / ks), p.H, tz);
#define B200_HL(BF)                                                                                             \
  if (ks == 4) B200_CHECK_CUDA(launch_pdl(head_linear_kernel<BF, 4, kAct>, grid, dim3(256), 0, s, p));           \
  else if (ks == 2) B200_CHECK_CUDA(launch_pdl(head_linear_kernel<BF, 2, kAct>, grid, dim3(256), 0, s, p));      \
  else B200_CHECK_CUDA(launch_pdl(head_linear_kernel<BF, 1, kAct>, grid, dim3(256), 0, s, p))
  if (dtype == kBF16) { B200_HL(true); } else { B200_HL(false); }
#undef B200_HL
  return kOk;
}

// y[t * ldy + h * yh + n] = sum_k W[h, n, k] act(x[t * ldx + h * xh + k]), act 0 = none, 1 = tanh. 16-bit: K, strides in
// multiples of 8 elements.
B200_API int b200_head_linear(const void* x, const void* w, void* y, int T, int H, int N, int K, long long ldx, long long xh,
                              long long ldy, long long yh, int act, int dtype, void* stream) {
  if (T <= 0) return kOk;
  B200_REQUIRE(H >= 1 && N >= 1 && K >= 1 && H <= 65535, "bad head_linear shape");
  B200_REQUIRE(act == kActNone || act == kActTanh, "head_linear: unknown activation %d", act);
  const HeadLinearParams p{x, w, y, T, H, N, K, ldx, xh, ldy, yh};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return act == kActTanh ? launch_head_linear<kActTanh>(p, dtype, s) : launch_head_linear<kActNone>(p, dtype, s);
}

static int fill_latent(LatentParams& p, const void* q, const void* cache, const int* block_table, int bt_stride, const int* kv_lens,
                       int B, int S, int H, int pitch, int page, float scale) {
  B200_REQUIRE(B >= 1 && S >= 1 && H >= 1 && page >= 1 && B <= 65535, "bad latent attention shape");
  B200_REQUIRE(pitch % 8 == 0, "the latent row (%d elements) must be a multiple of 8", pitch);
  memset(&p, 0, sizeof(p));
  p.q = q; p.cache = cache; p.block_table = block_table; p.kv_lens = kv_lens; p.bt_stride = bt_stride; p.page = page;
  p.H = H; p.S = S; p.pitch = pitch; p.scale = scale;
  return kOk;
}

// Merges partial results o_part fp32 [rows, splits, pitch] with log-sum-exps lse_part fp32 [rows, splits]; row % H is the head.
B200_API int b200_latent_combine(const float* o_part, const float* lse_part, const float* sink, int rows, int H, int splits, int pitch,
                                 void* out, int dtype, void* stream) {
  if (rows <= 0) return kOk;
  B200_REQUIRE(rows <= 65535, "latent_combine: too many rows (%d)", rows);
  const dim3 grid((pitch + 127) / 128, rows);
  B200_DISPATCH_FLOAT(dtype, B200_CHECK_CUDA(launch_pdl(latent_combine_kernel<T>, grid, dim3(128), 0, static_cast<cudaStream_t>(stream),
                                                        o_part, lse_part, sink, H, splits, pitch, static_cast<T*>(out)));
                      return kOk;);
}

B200_API int b200_latent_attention_plain(const void* q, const void* cache, const int* block_table, int bt_stride, const int* kv_lens,
                                         int B, int S, int H, int pitch, int page, float scale, const float* sink, void* out,
                                         int dtype, void* stream) {
  LatentParams p;
  int rc = fill_latent(p, q, cache, block_table, bt_stride, kv_lens, B, S, H, pitch, page, scale);
  if (rc != kOk) return rc;
  p.sink = sink; p.out = out;
  const int smem = 4 * 2 * pitch * 4;
  B200_REQUIRE(smem <= 200 * 1024, "latent rank %d does not fit in shared memory", pitch);
  const dim3 grid((S * H + 3) / 4, B);
  B200_DISPATCH_FLOAT(dtype,
                      B200_CHECK_CUDA(cudaFuncSetAttribute(latent_attention_plain_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
                      B200_CHECK_CUDA(launch_pdl(latent_attention_plain_kernel<T>, grid, dim3(128), smem, static_cast<cudaStream_t>(stream), p));
                      return kOk;);
}
