// Latent attention: keys and values of all heads are linear images of one cached vector c per token,
//   k_h = Wk_h c,  v_h = Wv_h c,   so   q_h . k_h = (Wk_h^T q_h) . c   and   sum_j p_j v_hj = Wv_h (sum_j p_j c_j).
// The cache holds only c ([slots, rank], paged). For few query tokens the products with Wk and Wv are taken on the query
// side ("absorbed"), which turns the op into multi-query attention of H heads over one shared key = value row:
//   latent_prep       RMS norm of the down-projected row, written to the cache slot of its token; squared-relu of the
//                     feed-forward's up-projection, which sits in the same GEMM output
//   head_linear       y[t, h, :] = W[h] x[t, h, :]  (per-head GEMM: Wk^T on the query, Wv on the attended latent)
//   latent_attention  split-KV attention over the paged latents. One CTA owns 16 or 32 rows (query token x head) of a
//                     sequence and a range of 64-token tiles; a tile is loaded into shared memory once and serves as keys
//                     (scores) and as values. The M side is a handful of heads, so it uses warp-level m16n8k16 products.
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

constexpr int kHlTok = 4;  // token tiles of 8 per CTA

// 16-bit: CTA = one head, 128 / KS output rows, 8 * kHlTok tokens. A warp multiplies 16 rows of W by the tokens over its K
// slice; KS warps share the rows and add their partial sums through shared memory. Both fragments are read straight from
// global memory: a lane takes 8 consecutive k per 32-wide step (one 16-byte load per row), which permutes k inside the
// step the same way for both operands and leaves the sum over k unchanged.
template <bool BF16, int KS>
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
__global__ void __launch_bounds__(128) head_linear_f32_kernel(const HeadLinearParams p) {
  extern __shared__ float xs[];
  const int t = blockIdx.x, h = blockIdx.y;
  griddep_launch_dependents();
  griddep_wait();
  const float* x = static_cast<const float*>(p.x) + t * p.ldx + h * p.xh;
  for (int k = threadIdx.x; k < p.K; k += blockDim.x) xs[k] = x[k];
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
  float* o_part;           // [B * S * H, splits, pitch]
  float* lse_part;         // [B * S * H, splits] natural log
  const float* sink;       // [H] or null (latent_attention_plain)
  void* out;               // [B * S * H, pitch]  (latent_attention_plain)
  int bt_stride, page, H, S, pitch, splits;
  float scale, scale_log2e;
};

constexpr int kLtKeys = 64;                 // keys per tile; the page size is a multiple of it
constexpr int kLtScorePitch = kLtKeys + 4;  // floats
constexpr int kLtProbPitch = kLtKeys + 8;   // 16-bit elements

template <int RM, int RK>
constexpr int latent_smem_bytes() {
  return (16 * RM + 2 * kLtKeys) * (RK + 8) * 2 + 16 * RM * (kLtScorePitch * 4 + kLtProbPitch * 2 + 8);
}

// RM: 16-row tiles per CTA (1 or 2); RK: rank rounded up to a multiple of 128 (the padding columns are zero in shared
// memory). 8 warps. Scores: a warp owns 16 keys x one row tile (RM = 2) or 8 keys (RM = 1). Values: a warp owns RK / 8
// columns of all rows. A row stride of RK + 8 elements puts the eight rows of an ldmatrix into different banks.
template <bool BF16, int RM, int RK>
__global__ void __launch_bounds__(256, 1) latent_attention_kernel(const LatentParams p) {
  constexpr int kRows = 16 * RM, kPitch = RK + 8, kNP = RK / 128;
  extern __shared__ __align__(16) uint8_t smem[];
  uint16_t* sq = reinterpret_cast<uint16_t*>(smem);
  uint16_t* sc = sq + kRows * kPitch;                                  // [2][64][kPitch]
  float* ss = reinterpret_cast<float*>(sc + 2 * kLtKeys * kPitch);     // [kRows][68]
  uint16_t* sp = reinterpret_cast<uint16_t*>(ss + kRows * kLtScorePitch);  // [kRows][72]
  float* corr = reinterpret_cast<float*>(sp + kRows * kLtProbPitch);   // [kRows]
  float* inv_l = corr + kRows;                                         // [kRows]

  const int split = blockIdx.x, b = blockIdx.z, r0 = blockIdx.y * kRows;
  const int n_rows = p.S * p.H;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  griddep_launch_dependents();
  griddep_wait();
  const int kv_len = p.kv_lens[b];
  const int first_key_limit = kv_len - p.S;  // last key of token 0; token i adds i
  // keys any row of this block attends, cut into `splits` ranges of whole tiles
  const int last_tok = (min(r0 + kRows, n_rows) - 1) / p.H;
  const int n_keys = max(0, min(kv_len, first_key_limit + last_tok + 1));
  const int n_tiles = (n_keys + kLtKeys - 1) / kLtKeys;
  const int per = (n_tiles + p.splits - 1) / p.splits;
  const int tile0 = min(n_tiles, split * per), tile1 = min(n_tiles, tile0 + per);
  const size_t row_base = static_cast<size_t>(b) * n_rows;
  if (tile0 >= tile1) {
    for (int r = threadIdx.x; r < kRows; r += blockDim.x)
      if (r0 + r < n_rows) p.lse_part[(row_base + r0 + r) * p.splits + split] = -INFINITY;
    return;
  }
  const uint16_t* q = static_cast<const uint16_t*>(p.q);
  const uint16_t* cache = static_cast<const uint16_t*>(p.cache);
  const int* table = p.block_table + static_cast<size_t>(b) * p.bt_stride;

  auto load_tile = [&](int tile, int stage) {
    const int j0 = tile * kLtKeys;
    const size_t base = static_cast<size_t>(table[j0 / p.page]) * p.page + j0 % p.page;
    for (int i = threadIdx.x; i < kLtKeys * (RK / 8); i += 256) {
      const int key = i / (RK / 8), c = (i - key * (RK / 8)) * 8;
      const bool in = j0 + key < n_keys && c < p.pitch;
      cp_async_16(static_cast<uint32_t>(__cvta_generic_to_shared(sc + (stage * kLtKeys + key) * kPitch + c)),
                  in ? cache + (base + key) * p.pitch + c : cache, in ? 16 : 0);
    }
    cp_async_commit();
  };
  for (int i = threadIdx.x; i < kRows * (RK / 8); i += 256) {
    const int r = i / (RK / 8), c = (i - r * (RK / 8)) * 8;
    const bool in = r0 + r < n_rows && c < p.pitch;
    cp_async_16(static_cast<uint32_t>(__cvta_generic_to_shared(sq + r * kPitch + c)), in ? q + (row_base + r0 + r) * p.pitch + c : q,
                in ? 16 : 0);
  }
  load_tile(tile0, 0);  // one group with the query rows

  constexpr int kRowsPerWarp = kRows / 8;
  float m_run[kRowsPerWarp], l_run[kRowsPerWarp];
#pragma unroll
  for (int i = 0; i < kRowsPerWarp; ++i) m_run[i] = -INFINITY, l_run[i] = 0.f;
  float acc[RM][2 * kNP][4] = {};
  const int g = lane >> 2, tq = lane & 3;
  const int col0 = warp * (RK / 8);

  for (int tile = tile0; tile < tile1; ++tile) {
    const int stage = (tile - tile0) & 1;
    cp_async_wait<0>();
    __syncthreads();  // this tile has landed for every thread, and the other stage is no longer being read
    if (tile + 1 < tile1) load_tile(tile + 1, stage ^ 1);
    const uint16_t* ct = sc + stage * kLtKeys * kPitch;
    // ---- scores
    {
      const int mt = RM == 2 ? warp >> 2 : 0;
      const uint32_t qa = static_cast<uint32_t>(__cvta_generic_to_shared(
          sq + (mt * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * kPitch + (lane >> 4) * 8));
      if (RM == 2) {
        const int kg = (warp & 3) * 16;
        const uint32_t ka = static_cast<uint32_t>(__cvta_generic_to_shared(
            ct + (kg + (lane & 7) + ((lane >> 4) & 1) * 8) * kPitch + ((lane >> 3) & 1) * 8));
        float s[2][4] = {};
#pragma unroll 8
        for (int kk = 0; kk < RK / 16; ++kk) {
          uint32_t a[4], b0, b1, b2, b3;
          ldmatrix_x4(qa + kk * 32, a[0], a[1], a[2], a[3]);
          ldmatrix_x4(ka + kk * 32, b0, b1, b2, b3);
          mma16816<BF16>(s[0], a, b0, b1);
          mma16816<BF16>(s[1], a, b2, b3);
        }
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          float* dst = ss + (mt * 16 + g) * kLtScorePitch + kg + n * 8 + 2 * tq;
          dst[0] = s[n][0]; dst[1] = s[n][1];
          dst[8 * kLtScorePitch] = s[n][2]; dst[8 * kLtScorePitch + 1] = s[n][3];
        }
      } else {
        const int kg = warp * 8;
        const uint32_t ka = static_cast<uint32_t>(__cvta_generic_to_shared(ct + (kg + (lane & 7)) * kPitch + (lane >> 3) * 8));
        float s[2][4] = {};
#pragma unroll 4
        for (int kk = 0; kk < RK / 32; ++kk) {
          uint32_t a[4], b0, b1, b2, b3;
          ldmatrix_x4(ka + kk * 64, b0, b1, b2, b3);
          ldmatrix_x4(qa + kk * 64, a[0], a[1], a[2], a[3]);
          mma16816<BF16>(s[0], a, b0, b1);
          ldmatrix_x4(qa + kk * 64 + 32, a[0], a[1], a[2], a[3]);
          mma16816<BF16>(s[1], a, b2, b3);
        }
        float* dst = ss + g * kLtScorePitch + kg + 2 * tq;
        dst[0] = s[0][0] + s[1][0]; dst[1] = s[0][1] + s[1][1];
        dst[8 * kLtScorePitch] = s[0][2] + s[1][2]; dst[8 * kLtScorePitch + 1] = s[0][3] + s[1][3];
      }
    }
    __syncthreads();
    // ---- online softmax, one row per warp at a time
#pragma unroll
    for (int i = 0; i < kRowsPerWarp; ++i) {
      const int r = warp * kRowsPerWarp + i;
      const int limit = r0 + r < n_rows ? first_key_limit + (r0 + r) / p.H - tile * kLtKeys : -1;  // last visible key of the tile
      const float s0 = lane <= limit ? ss[r * kLtScorePitch + lane] * p.scale_log2e : -INFINITY;
      const float s1 = lane + 32 <= limit ? ss[r * kLtScorePitch + lane + 32] * p.scale_log2e : -INFINITY;
      const float m_new = fmaxf(m_run[i], warp_max(fmaxf(s0, s1)));
      const float base = m_new == -INFINITY ? 0.f : m_new;
      const float p0 = exp2f(s0 - base), p1 = exp2f(s1 - base), c = exp2f(m_run[i] - base);
      l_run[i] = l_run[i] * c + warp_sum(p0 + p1);
      m_run[i] = m_new;
      const uint32_t packed = BF16 ? pack_bf16x2(p0, p1) : pack_f16x2(p0, p1);
      sp[r * kLtProbPitch + lane] = static_cast<uint16_t>(packed & 0xffffu);
      sp[r * kLtProbPitch + lane + 32] = static_cast<uint16_t>(packed >> 16);
      if (lane == 0) corr[r] = c;
    }
    __syncthreads();
    // ---- values
#pragma unroll
    for (int mt = 0; mt < RM; ++mt) {
      const float c0 = corr[mt * 16 + g], c1 = corr[mt * 16 + g + 8];
#pragma unroll
      for (int n = 0; n < 2 * kNP; ++n) {
        acc[mt][n][0] *= c0; acc[mt][n][1] *= c0;
        acc[mt][n][2] *= c1; acc[mt][n][3] *= c1;
      }
    }
#pragma unroll
    for (int kk = 0; kk < kLtKeys / 16; ++kk) {
      uint32_t a[RM][4];
#pragma unroll
      for (int mt = 0; mt < RM; ++mt)
        ldmatrix_x4(static_cast<uint32_t>(__cvta_generic_to_shared(
                        sp + (mt * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * kLtProbPitch + kk * 16 + (lane >> 4) * 8)),
                    a[mt][0], a[mt][1], a[mt][2], a[mt][3]);
#pragma unroll
      for (int n = 0; n < kNP; ++n) {
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4_trans(static_cast<uint32_t>(__cvta_generic_to_shared(
                              ct + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * kPitch + col0 + n * 16 + (lane >> 4) * 8)),
                          b0, b1, b2, b3);
#pragma unroll
        for (int mt = 0; mt < RM; ++mt) {
          mma16816<BF16>(acc[mt][2 * n], a[mt], b0, b1);
          mma16816<BF16>(acc[mt][2 * n + 1], a[mt], b2, b3);
        }
      }
    }
  }
  // ---- normalised partial result and log-sum-exp of this split
#pragma unroll
  for (int i = 0; i < kRowsPerWarp; ++i) {
    const int r = warp * kRowsPerWarp + i;
    if (lane == 0) {
      inv_l[r] = l_run[i] > 0.f ? 1.f / l_run[i] : 0.f;
      if (r0 + r < n_rows)
        p.lse_part[(row_base + r0 + r) * p.splits + split] =
            l_run[i] > 0.f ? (m_run[i] + log2f(l_run[i])) * 0.6931471805599453f : -INFINITY;
    }
  }
  __syncthreads();
#pragma unroll
  for (int mt = 0; mt < RM; ++mt)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int r = mt * 16 + g + 8 * half;
      if (r0 + r >= n_rows) continue;
      const float il = inv_l[r];
      float* dst = p.o_part + ((row_base + r0 + r) * p.splits + split) * p.pitch;
#pragma unroll
      for (int n = 0; n < 2 * kNP; ++n) {
        const int c = col0 + n * 8 + 2 * tq;
        if (c < p.pitch)
          *reinterpret_cast<float2*>(dst + c) = make_float2(acc[mt][n][2 * half] * il, acc[mt][n][2 * half + 1] * il);
      }
    }
}

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

template <bool BF16, int RM, int RK>
static int launch_latent(const LatentParams& p, int B, cudaStream_t s) {
  constexpr int smem = latent_smem_bytes<RM, RK>();
  static bool configured[64] = {false};
  int dev = 0;
  B200_CHECK_CUDA(cudaGetDevice(&dev));
  if (!configured[dev & 63]) {
    B200_CHECK_CUDA(cudaFuncSetAttribute(latent_attention_kernel<BF16, RM, RK>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    configured[dev & 63] = true;
  }
  const dim3 grid(p.splits, (p.S * p.H + 16 * RM - 1) / (16 * RM), B);
  B200_REQUIRE(grid.y <= 65535, "too many query rows (%d) for the absorbed attention", p.S * p.H);
  B200_CHECK_CUDA(launch_pdl(latent_attention_kernel<BF16, RM, RK>, grid, dim3(256), smem, s, p));
  return kOk;
}
template <bool BF16, int RM>
static int launch_latent_rank(const LatentParams& p, int B, cudaStream_t s) {
  if (p.pitch <= 128) return launch_latent<BF16, RM, 128>(p, B, s);
  if (p.pitch <= 256) return launch_latent<BF16, RM, 256>(p, B, s);
  if (p.pitch <= 384) return launch_latent<BF16, RM, 384>(p, B, s);
  return launch_latent<BF16, RM, 512>(p, B, s);
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

// y[t * ldy + h * yh + n] = sum_k W[h, n, k] x[t * ldx + h * xh + k]. 16-bit: K, strides in multiples of 8 elements.
B200_API int b200_head_linear(const void* x, const void* w, void* y, int T, int H, int N, int K, long long ldx, long long xh,
                              long long ldy, long long yh, int dtype, void* stream) {
  if (T <= 0) return kOk;
  B200_REQUIRE(H >= 1 && N >= 1 && K >= 1 && H <= 65535, "bad head_linear shape");
  HeadLinearParams p{x, w, y, T, H, N, K, ldx, xh, ldy, yh};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == kF32) {
    B200_REQUIRE(K <= 8192, "head_linear: K (%d) is limited to 8192 in fp32", K);
    B200_CHECK_CUDA(launch_pdl(head_linear_f32_kernel, dim3(T, H), dim3(128), static_cast<size_t>(K) * 4, s, p));
    return kOk;
  }
  B200_REQUIRE(dtype == kBF16 || dtype == kF16, "head_linear supports bf16 / f16 / f32");
  B200_REQUIRE(K % 8 == 0 && ldx % 8 == 0 && xh % 8 == 0, "head_linear: K (%d) and the input strides must be multiples of 8", K);
  const int tz = (T + 8 * kHlTok - 1) / (8 * kHlTok);
  B200_REQUIRE(tz <= 65535, "head_linear: too many tokens (%d)", T);
  const int ks = K > 256 ? 4 : K > 128 ? 2 : 1;
  const dim3 grid((N + 128 / ks - 1) / (128 / ks), H, tz);
#define B200_HL(BF)                                                                                       \
  if (ks == 4) B200_CHECK_CUDA(launch_pdl(head_linear_kernel<BF, 4>, grid, dim3(256), 0, s, p));           \
  else if (ks == 2) B200_CHECK_CUDA(launch_pdl(head_linear_kernel<BF, 2>, grid, dim3(256), 0, s, p));      \
  else B200_CHECK_CUDA(launch_pdl(head_linear_kernel<BF, 1>, grid, dim3(256), 0, s, p))
  if (dtype == kBF16) { B200_HL(true); } else { B200_HL(false); }
#undef B200_HL
  return kOk;
}

static int fill_latent(LatentParams& p, const void* q, const void* cache, const int* block_table, int bt_stride, const int* kv_lens,
                       int B, int S, int H, int pitch, int page, float scale) {
  B200_REQUIRE(B >= 1 && S >= 1 && H >= 1 && page >= 1 && B <= 65535, "bad latent attention shape");
  B200_REQUIRE(pitch % 8 == 0, "the latent row (%d elements) must be a multiple of 8", pitch);
  memset(&p, 0, sizeof(p));
  p.q = q; p.cache = cache; p.block_table = block_table; p.kv_lens = kv_lens; p.bt_stride = bt_stride; p.page = page;
  p.H = H; p.S = S; p.pitch = pitch; p.scale = scale; p.scale_log2e = scale * 1.4426950408889634f;
  return kOk;
}

// Split partials: o_part fp32 [B * S * H, splits, pitch], lse_part fp32 [B * S * H, splits]; merge with b200_latent_combine.
B200_API int b200_latent_attention(const void* q, const void* cache, const int* block_table, int bt_stride, const int* kv_lens, int B,
                                   int S, int H, int pitch, int page, float scale, int splits, float* o_part, float* lse_part,
                                   int dtype, void* stream) {
  LatentParams p;
  int rc = fill_latent(p, q, cache, block_table, bt_stride, kv_lens, B, S, H, pitch, page, scale);
  if (rc != kOk) return rc;
  B200_REQUIRE(dtype == kBF16 || dtype == kF16, "latent attention supports bf16 / f16 (b200_latent_attention_plain takes fp32)");
  B200_REQUIRE(pitch <= 512, "latent attention handles ranks up to 512, got %d", pitch);
  B200_REQUIRE(page % kLtKeys == 0, "the page size (%d) must be a multiple of %d", page, kLtKeys);
  B200_REQUIRE(splits >= 1 && o_part && lse_part, "latent attention needs its partial buffers");
  p.splits = splits; p.o_part = o_part; p.lse_part = lse_part;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == kBF16) return S * H > 16 ? launch_latent_rank<true, 2>(p, B, s) : launch_latent_rank<true, 1>(p, B, s);
  return S * H > 16 ? launch_latent_rank<false, 2>(p, B, s) : launch_latent_rank<false, 1>(p, B, s);
}

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
