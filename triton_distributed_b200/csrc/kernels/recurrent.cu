// Token mixers whose memory is a matrix per head, S [key size, value size] in fp32, carried from token to token:
//
//   decayed outer products (kWkv)   o_t = S^T r_t + (r_t . (u * k_t)) v_t;            S <- diag(w_t) S + k_t v_t^T
//                                   with w_t = exp(-exp(z_t + w0)) per key channel and a bonus u for the current token
//   gated delta rule (kDelta)       a = S^T k_t;  d = beta_t (v_t - g_t a);           S <- g_t S + k_t d^T;  o_t = S^T q_t
//                                   with g_t = exp(-exp(A) softplus(a_t + dt)) and beta_t = sigmoid(b_t) per head, q and k
//                                   scaled to unit length (q also by key_size^-0.5). S^T q is read from the old state together
//                                   with S^T k: o_t = g_t S_old^T q_t + (k_t . q_t) d, so a token costs one pass over S.
// Both end in the same way: o divided by its root mean square over the head, times a gain, times silu(gate).
//
// The columns of S never mix, and all of S stays in registers for the whole call. One CTA owns one head of one sequence; a
// thread owns R rows x C columns, the threads that share columns are neighbouring lanes and reduce with shuffles. Tokens go
// through shared memory in chunks of 16; the next chunk's copies are in flight while a chunk is computed. The order of
// all sums is that of the tokens, whatever the call's length: results do not depend on how a sequence is cut.
// Heads of up to 128 x 128 run this way (`recurrent_kernel`); larger ones keep S in global memory (`recurrent_plain_kernel`).
//
// In front of them: token_mix (h + (previous h - h) * mu for several mu at once) and short_conv (causal convolution over a few
// tokens per channel, silu), both of which carry the last inputs of a sequence from call to call.
#include "b200/elem.cuh"
#include "b200/host.h"
#include "b200/mma_sync.cuh"
#include "b200/packed_f32.cuh"
#include "b200/primitives.cuh"

#include <cstring>

namespace b200 {

__device__ __forceinline__ float silu(float z) { return z / (1.f + expf(-z)); }

// ------------------------------------------------------------------------------------------------ token_mix
constexpr int kMixMax = 8;       // mixes per call
constexpr int kMixTokens = 8;    // tokens per thread

struct TokenMixParams {
  const void* h;     // [B * S, pitch]
  const void* mu;    // [G, pitch]
  void* last;        // [B, pitch] the previous token of every sequence, updated
  void* out;         // [B * S, G, pitch]
  int S, G, pitch;
};

// grid (column blocks, token blocks, B). The thread of the first token block alone reads and replaces the carried row.
template <typename T, int G>
__global__ void __launch_bounds__(128) token_mix_kernel(const TokenMixParams p) {
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * 4;
  const int t0 = blockIdx.y * kMixTokens, t1 = min(p.S, t0 + kMixTokens);
  griddep_launch_dependents();
  if (c >= p.pitch) return;
  float4 mu[G];
#pragma unroll
  for (int g = 0; g < G; ++g) mu[g] = load4(static_cast<const T*>(p.mu) + static_cast<size_t>(g) * p.pitch + c);
  griddep_wait();
  const T* h = static_cast<const T*>(p.h) + static_cast<size_t>(blockIdx.z) * p.S * p.pitch + c;
  T* last = static_cast<T*>(p.last) + static_cast<size_t>(blockIdx.z) * p.pitch + c;
  T* out = static_cast<T*>(p.out) + static_cast<size_t>(blockIdx.z) * p.S * G * p.pitch + c;
  float4 before = t0 == 0 ? load4(last) : load4(h + static_cast<size_t>(t0 - 1) * p.pitch);
  if (t0 == 0) store4(last, load4(h + static_cast<size_t>(p.S - 1) * p.pitch));
  for (int t = t0; t < t1; ++t) {
    const float4 cur = load4(h + static_cast<size_t>(t) * p.pitch);
#pragma unroll
    for (int g = 0; g < G; ++g) {
      float4 o;
      o.x = fmaf(before.x - cur.x, mu[g].x, cur.x); o.y = fmaf(before.y - cur.y, mu[g].y, cur.y);
      o.z = fmaf(before.z - cur.z, mu[g].z, cur.z); o.w = fmaf(before.w - cur.w, mu[g].w, cur.w);
      store4(out + (static_cast<size_t>(t) * G + g) * p.pitch, o);
    }
    before = cur;
  }
}

// ------------------------------------------------------------------------------------------------ short_conv
constexpr int kConvTokens = 16;  // tokens per thread

struct ShortConvParams {
  const void* x;      // [B * S, C] (row pitch ldx)
  const float* taps;  // [n, C], tap n - 1 weighs the current token
  void* last;         // [B, n - 1, C] the previous inputs of every sequence, oldest first, updated
  void* out;          // [B * S, C]
  int S, C, n, ldx;
};

// grid (channel blocks, token blocks, B), four channels per thread. kN > 0: that many taps, kept in registers.
template <typename T, int kN>
__global__ void __launch_bounds__(128) short_conv_kernel(const ShortConvParams p) {
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * 4;
  const int t0 = blockIdx.y * kConvTokens, t1 = min(p.S, t0 + kConvTokens);
  griddep_launch_dependents();
  if (c >= p.C) return;
  const int n = kN > 0 ? kN : p.n;
  float4 w[kN > 0 ? kN : 1];
  if (kN > 0) {
#pragma unroll
    for (int j = 0; j < (kN > 0 ? kN : 0); ++j) w[j] = load4(p.taps + static_cast<size_t>(j) * p.C + c);
  }
  griddep_wait();
  const T* x = static_cast<const T*>(p.x) + static_cast<size_t>(blockIdx.z) * p.S * p.ldx + c;
  T* last = static_cast<T*>(p.last) + static_cast<size_t>(blockIdx.z) * (n - 1) * p.C + c;
  T* out = static_cast<T*>(p.out) + static_cast<size_t>(blockIdx.z) * p.S * p.C + c;
  // input at position t of this call; the n - 1 positions before the call are the carried rows
  auto input = [&](int t) { return t >= 0 ? load4(x + static_cast<size_t>(t) * p.ldx) : load4(last + static_cast<size_t>(n - 1 + t) * p.C); };
  float4 win[kN > 0 ? kN : 1];   // inputs t - kN + 1 .. t
  if (kN > 0) {
#pragma unroll
    for (int j = 1; j < (kN > 0 ? kN : 1); ++j) win[j] = input(t0 - kN + j);
  }
  for (int t = t0; t < t1; ++t) {
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    auto tap = [&](const float4& wj, const float4& v) {
      acc.x = fmaf(wj.x, v.x, acc.x); acc.y = fmaf(wj.y, v.y, acc.y); acc.z = fmaf(wj.z, v.z, acc.z); acc.w = fmaf(wj.w, v.w, acc.w);
    };
    if (kN > 0) {
#pragma unroll
      for (int j = 0; j + 1 < (kN > 0 ? kN : 1); ++j) win[j] = win[j + 1];
      win[(kN > 0 ? kN : 1) - 1] = input(t);
#pragma unroll
      for (int j = 0; j < (kN > 0 ? kN : 1); ++j) tap(w[j], win[j]);
    } else {
      for (int j = 0; j < n; ++j) tap(load4(p.taps + static_cast<size_t>(j) * p.C + c), input(t - n + 1 + j));
    }
    store4(out + static_cast<size_t>(t) * p.C, make_float4(silu(acc.x), silu(acc.y), silu(acc.z), silu(acc.w)));
  }
  if (t0 == 0)  // the last n - 1 inputs up to the end of the call; slot j only needs slots behind it, so ascending is safe
    for (int j = 0; j < n - 1; ++j) store4(last + static_cast<size_t>(j) * p.C, input(p.S - (n - 1) + j));
}

// ------------------------------------------------------------------------------------------------ the recurrences
enum RecurrentKind : int { kWkv = 0, kDelta = 1 };

struct RecurrentParams {
  // row t of a sequence is row b * S + t; head h at column h * (its padded size)
  const void *q, *k, *v, *gate;   // q: the read-out vector (r of kWkv)
  const void* decay;              // kWkv: z [T, H * Dp]; kDelta: a [T, H] (pitch ld_decay)
  const void* beta;               // kDelta: b [T, H] (pitch ld_decay)
  int ldq, ldk, ldv, ldg, ld_decay;
  const float* decay_base;        // kWkv: w0 [H * Dp]; kDelta: A [H]
  const float* decay_bias;        // kDelta: dt [H]
  const float* bonus;             // kWkv: u [H * Dp]
  const float* gain;              // [Ep] (gain_stride 0) or [H * Ep] (gain_stride Ep)
  int gain_stride;
  float* state;                   // [B, H, Dp, Ep]
  void* out;                      // [T, H * Ep]
  int S, H, per;                  // tokens per sequence, heads, heads per q / k head
  int D, E, Dp, Ep;               // key and value sizes of a head, and padded to multiples of 8
  float eps;
};

__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float wkv_decay(float z, float base) { return expf(-expf(z + base)); }
__device__ __forceinline__ float delta_decay(float a, float A, float dt) { return expf(-expf(A) * softplus(a + dt)); }

// eight elements global -> shared memory without registers; zeros where !in
template <typename T>
__device__ __forceinline__ void copy8(T* dst, const void* base, size_t at, bool in) {
#pragma unroll
  for (int i = 0; i < static_cast<int>(sizeof(T) / 2); ++i)
    cp_async_16(static_cast<uint32_t>(__cvta_generic_to_shared(dst)) + 16 * i,
                static_cast<const T*>(base) + (in ? at : 0) + i * (16 / sizeof(T)), in ? 16 : 0);
}
template <typename T>
__device__ __forceinline__ void load8(const T* src, float (&f)[8]) {
  const float4 a = load4(src), b = load4(src + 4);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ void store8(float* dst, const float (&f)[8]) {
  *reinterpret_cast<float4*>(dst) = make_float4(f[0], f[1], f[2], f[3]);
  *reinterpret_cast<float4*>(dst + 4) = make_float4(f[4], f[5], f[6], f[7]);
}

constexpr int kRecTokens = 16;   // tokens per chunk
constexpr int recurrent_smem(int dp, int elem) { return (6 * kRecTokens * dp + 4 * kRecTokens + 2 * dp) * 4 + 5 * kRecTokens * dp * elem; }

// kP: padded key and value size; a thread owns R rows (groups of four: rows 4 (lane % 8) + 32 i ...) and C = 4 columns.
template <typename T, int kKind, int kP, int R>
__global__ void __launch_bounds__(kP * kP / (R * 4), kP == 128 ? 2 : 4) recurrent_kernel(const RecurrentParams p) {
  constexpr int C = 4, KG = kP / R, kThreads = kP * kP / (R * C), kWarps = kThreads / 32;
  constexpr int kItems = kRecTokens * kP / 8;   // groups of eight elements of a chunk
  static_assert(KG == 8 && kItems <= kThreads, "thread layout");
  extern __shared__ __align__(16) float smf[];
  float* sq = smf;                          // [tokens][kP]
  float* sk = sq + kRecTokens * kP;
  float* sw = sk + kRecTokens * kP;         // kWkv: decays per key channel
  float* sv = sw + kRecTokens * kP;
  float* sg = sv + kRecTokens * kP;         // silu(gate)
  float* so = sg + kRecTokens * kP;
  float* s_decay = so + kRecTokens * kP;    // kDelta: [tokens]
  float* s_beta = s_decay + kRecTokens;
  float* s_qk = s_beta + kRecTokens;        // kWkv: r . (u * k); kDelta: q . k
  float* s_base = s_qk + 2 * kRecTokens;    // kWkv: w0 and u of the head
  float* s_bonus = s_base + kP;
  T* raw = reinterpret_cast<T*>(s_bonus + kP);   // [q, k, decay, v, gate][tokens][kP] of the next chunk as it lies in memory
  const int h = blockIdx.x, b = blockIdx.y, kh = h / p.per;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, kg = lane & 7;
  const int col0 = (warp * 4 + (lane >> 3)) * C;
  float* state = p.state + (static_cast<size_t>(b) * p.H + h) * p.Dp * p.Ep;
  griddep_launch_dependents();
  // the state comes from an earlier call: it may be fetched into L2, but not read, before that call is known to be over
  for (int i = threadIdx.x * 32; i < p.Dp * p.Ep; i += kThreads * 32) asm volatile("prefetch.global.L2 [%0];" ::"l"(state + i));
  const int ic = threadIdx.x % (kP / 8) * 8, it = threadIdx.x / (kP / 8);   // this thread's elements of a chunk
  const bool has_item = threadIdx.x < kItems;
  T* mine_raw = raw + it * kP + ic;   // a thread converts the elements that it copied itself
  constexpr int kRaw = kRecTokens * kP;
  if (kKind == kWkv && threadIdx.x < kP) {
    const bool in = threadIdx.x < p.Dp;
    s_base[threadIdx.x] = in ? p.decay_base[h * p.Dp + threadIdx.x] : 0.f;
    s_bonus[threadIdx.x] = in ? p.bonus[h * p.Dp + threadIdx.x] : 0.f;
  }
  const float A = kKind == kDelta ? p.decay_base[h] : 0.f, dt = kKind == kDelta ? p.decay_bias[h] : 0.f;
  griddep_wait();

  float ra = 0.f, rb = 0.f;
  const size_t row0 = static_cast<size_t>(b) * p.S;
  auto fetch = [&](int t0) {
    if (has_item) {
      const size_t row = row0 + t0 + it;
      const bool in = t0 + it < p.S, ink = in && ic < p.Dp, inv = in && ic < p.Ep;
      copy8<T>(mine_raw, p.q, row * p.ldq + kh * p.Dp + ic, ink);
      copy8<T>(mine_raw + kRaw, p.k, row * p.ldk + kh * p.Dp + ic, ink);
      if (kKind == kWkv) copy8<T>(mine_raw + 2 * kRaw, p.decay, row * p.ld_decay + h * p.Dp + ic, ink);
      copy8<T>(mine_raw + 3 * kRaw, p.v, row * p.ldv + h * p.Ep + ic, inv);
      copy8<T>(mine_raw + 4 * kRaw, p.gate, row * p.ldg + h * p.Ep + ic, inv);
    }
    cp_async_commit();
    if (kKind == kDelta && threadIdx.x < kRecTokens && t0 + static_cast<int>(threadIdx.x) < p.S) {
      const size_t at = (row0 + t0 + threadIdx.x) * p.ld_decay + h;
      ra = to_float(static_cast<const T*>(p.decay)[at]);
      rb = to_float(static_cast<const T*>(p.beta)[at]);
    }
  };
  fetch(0);
  __syncthreads();   // s_base, s_bonus

  f32x2 s[R / 2][C];   // s[2 i + e][c] = rows 32 i + 4 kg + 2 e, + 1 of column col0 + c
#pragma unroll
  for (int i = 0; i < R / 4; ++i)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = 32 * i + 4 * kg + 2 * e;
      float4 lo = make_float4(0.f, 0.f, 0.f, 0.f), hi = lo;
      if (r < p.Dp && col0 < p.Ep) {   // Dp and Ep are multiples of 8
        lo = *reinterpret_cast<const float4*>(state + static_cast<size_t>(r) * p.Ep + col0);
        hi = *reinterpret_cast<const float4*>(state + static_cast<size_t>(r + 1) * p.Ep + col0);
      }
      s[2 * i + e][0] = pack2(lo.x, hi.x); s[2 * i + e][1] = pack2(lo.y, hi.y);
      s[2 * i + e][2] = pack2(lo.z, hi.z); s[2 * i + e][3] = pack2(lo.w, hi.w);
    }

  for (int t0 = 0; t0 < p.S; t0 += kRecTokens) {
    const int n = min(kRecTokens, p.S - t0);
    // ---- registers -> shared memory. The products r . (u * k) and q . k and the lengths need sums over the kP / 8 threads of
    // a token, which are neighbouring lanes.
    cp_async_wait<0>();
    if (has_item) {   // whole warps: kItems is a multiple of 32
      float q8[8], k8[8], f[8];
      load8(mine_raw, q8);
      load8(mine_raw + kRaw, k8);
      float x = 0.f, y = 0.f, z = 0.f;
      if (kKind == kWkv) {
#pragma unroll
        for (int i = 0; i < 8; ++i) z = fmaf(q8[i] * s_bonus[ic + i], k8[i], z);
      } else {
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          x = fmaf(q8[i], q8[i], x);
          y = fmaf(k8[i], k8[i], y);
          z = fmaf(q8[i], k8[i], z);
        }
      }
#pragma unroll
      for (int o = kP / 16; o > 0; o >>= 1) {
        if (kKind == kDelta) {
          x += __shfl_xor_sync(0xffffffffu, x, o);
          y += __shfl_xor_sync(0xffffffffu, y, o);
        }
        z += __shfl_xor_sync(0xffffffffu, z, o);
      }
      if (kKind == kDelta) {
        const float iq = 1.f / (sqrtf(x + 1e-6f) * sqrtf(static_cast<float>(p.D))), ik = 1.f / sqrtf(y + 1e-6f);
        z *= iq * ik;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          q8[i] *= iq;
          k8[i] *= ik;
        }
      }
      if (ic == 0) s_qk[it] = z;
      store8(sq + it * kP + ic, q8);
      store8(sk + it * kP + ic, k8);
      if (kKind == kWkv) {
        load8(mine_raw + 2 * kRaw, f);
#pragma unroll
        for (int i = 0; i < 8; ++i) f[i] = wkv_decay(f[i], s_base[ic + i]);
        store8(sw + it * kP + ic, f);
      }
      load8(mine_raw + 3 * kRaw, f);
      store8(sv + it * kP + ic, f);
      load8(mine_raw + 4 * kRaw, f);
#pragma unroll
      for (int i = 0; i < 8; ++i) f[i] = silu(f[i]);
      store8(sg + it * kP + ic, f);
    }
    if (kKind == kDelta && threadIdx.x < kRecTokens) {
      s_decay[threadIdx.x] = delta_decay(ra, A, dt);
      s_beta[threadIdx.x] = 1.f / (1.f + expf(-rb));
    }
    __syncthreads();
    if (t0 + kRecTokens < p.S) fetch(t0 + kRecTokens);
    // ---- the tokens of the chunk
#pragma unroll 1
    for (int t = 0; t < n; ++t) {
      // four rows of this thread out of a row vector of token t
      auto four = [&](const float* x, int i) { return *reinterpret_cast<const ulonglong2*>(x + t * kP + 32 * i + 4 * kg); };
      const float4 v4 = *reinterpret_cast<const float4*>(sv + t * kP + col0);
      const float v[4] = {v4.x, v4.y, v4.z, v4.w};
      float o[4], d[4];
      if (kKind == kDelta) {
        f32x2 oa[C], da[C], kv[R / 2];
#pragma unroll
        for (int c = 0; c < C; ++c) oa[c] = da[c] = 0ull;
#pragma unroll
        for (int i = 0; i < R / 4; ++i) {
          const ulonglong2 q2 = four(sq, i), k2 = four(sk, i);
          kv[2 * i] = k2.x;
          kv[2 * i + 1] = k2.y;
#pragma unroll
          for (int c = 0; c < C; ++c) {
            da[c] = fma2(k2.x, s[2 * i][c], da[c]);
            oa[c] = fma2(q2.x, s[2 * i][c], oa[c]);
            da[c] = fma2(k2.y, s[2 * i + 1][c], da[c]);
            oa[c] = fma2(q2.y, s[2 * i + 1][c], oa[c]);
          }
        }
#pragma unroll
        for (int c = 0; c < C; ++c) {
          d[c] = sum2(da[c]);
          o[c] = sum2(oa[c]);
        }
#pragma unroll
        for (int m = 1; m < 8; m <<= 1)
#pragma unroll
          for (int c = 0; c < C; ++c) d[c] += __shfl_xor_sync(0xffffffffu, d[c], m);
        const float g = s_decay[t], beta = s_beta[t];
        const f32x2 g2 = pack2(g, g);
#pragma unroll
        for (int c = 0; c < C; ++c) {
          d[c] = beta * (v[c] - g * d[c]);
          const f32x2 d2 = pack2(d[c], d[c]);
#pragma unroll
          for (int i = 0; i < R / 2; ++i) s[i][c] = fma2(kv[i], d2, mul2(g2, s[i][c]));
        }
      } else {
        f32x2 oa[C], v2[C];
#pragma unroll
        for (int c = 0; c < C; ++c) {
          oa[c] = 0ull;
          v2[c] = pack2(v[c], v[c]);
          d[c] = v[c];
        }
#pragma unroll
        for (int i = 0; i < R / 4; ++i) {
          const ulonglong2 q2 = four(sq, i), k2 = four(sk, i), w2 = four(sw, i);
#pragma unroll
          for (int c = 0; c < C; ++c) {
            oa[c] = fma2(q2.x, s[2 * i][c], oa[c]);
            s[2 * i][c] = fma2(w2.x, s[2 * i][c], mul2(k2.x, v2[c]));
            oa[c] = fma2(q2.y, s[2 * i + 1][c], oa[c]);
            s[2 * i + 1][c] = fma2(w2.y, s[2 * i + 1][c], mul2(k2.y, v2[c]));
          }
        }
#pragma unroll
        for (int c = 0; c < C; ++c) o[c] = sum2(oa[c]);
      }
      // ---- sum over the eight lanes of a column group; lane kg is left with column (kg >> 1) of the group (kg bit 2 picks the
      // pair, bit 1 the member)
      const bool hi2 = (kg & 4) != 0, hi1 = (kg & 2) != 0;
      float k0 = hi2 ? o[2] : o[0], k1 = hi2 ? o[3] : o[1];
      k0 += __shfl_xor_sync(0xffffffffu, hi2 ? o[0] : o[2], 4);
      k1 += __shfl_xor_sync(0xffffffffu, hi2 ? o[1] : o[3], 4);
      float r = hi1 ? k1 : k0;
      r += __shfl_xor_sync(0xffffffffu, hi1 ? k0 : k1, 2);
      r += __shfl_xor_sync(0xffffffffu, r, 1);
      const float mine = hi2 ? (hi1 ? d[3] : d[2]) : (hi1 ? d[1] : d[0]);
      if ((kg & 1) == 0) so[t * kP + col0 + (kg >> 1)] = fmaf(s_qk[t], mine, kKind == kDelta ? s_decay[t] * r : r);
    }
    __syncthreads();
    // ---- norm over the head, gain, gate: one warp per token
    for (int t = warp; t < n; t += kWarps) {
      constexpr int kCols = kP / 32;
      float o[kCols], ss = 0.f;
#pragma unroll
      for (int i = 0; i < kCols; ++i) {
        o[i] = so[t * kP + 32 * i + lane];
        ss = fmaf(o[i], o[i], ss);
      }
      const float inv = 1.f / sqrtf(warp_sum(ss) / p.E + p.eps);
#pragma unroll
      for (int i = 0; i < kCols; ++i) {
        const int c = 32 * i + lane;
        if (c < p.Ep)
          static_cast<T*>(p.out)[(row0 + t0 + t) * p.H * p.Ep + h * p.Ep + c] =
              from_float<T>(o[i] * inv * p.gain[h * p.gain_stride + c] * sg[t * kP + c]);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < R / 4; ++i)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = 32 * i + 4 * kg + 2 * e;
      if (r < p.Dp && col0 < p.Ep) {
        const float2 c0 = unpack2(s[2 * i + e][0]), c1 = unpack2(s[2 * i + e][1]), c2 = unpack2(s[2 * i + e][2]), c3 = unpack2(s[2 * i + e][3]);
        *reinterpret_cast<float4*>(state + static_cast<size_t>(r) * p.Ep + col0) = make_float4(c0.x, c1.x, c2.x, c3.x);
        *reinterpret_cast<float4*>(state + static_cast<size_t>(r + 1) * p.Ep + col0) = make_float4(c0.y, c1.y, c2.y, c3.y);
      }
    }
}

__device__ __forceinline__ float cta_sum(float v, float* red) {
  v = warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  return warp_sum((threadIdx.x & 31) < (blockDim.x >> 5) ? red[threadIdx.x & 31] : 0.f);
}

// Heads of any size: the state stays in global memory, a thread walks the rows of its columns.
template <typename T, int kKind>
__global__ void __launch_bounds__(256) recurrent_plain_kernel(const RecurrentParams p) {
  extern __shared__ __align__(16) float smf[];
  __shared__ float red[32];
  float *sq = smf, *sk = sq + p.Dp, *sw = sk + p.Dp, *so = sw + p.Dp;
  const int h = blockIdx.x, b = blockIdx.y, kh = h / p.per;
  float* state = p.state + (static_cast<size_t>(b) * p.H + h) * p.Dp * p.Ep;
  griddep_launch_dependents();
  griddep_wait();
  for (int t = 0; t < p.S; ++t) {
    const size_t row = static_cast<size_t>(b) * p.S + t;
    float x = 0.f, y = 0.f, z = 0.f;
    __syncthreads();
    for (int i = threadIdx.x; i < p.Dp; i += blockDim.x) {
      const float q = to_float(static_cast<const T*>(p.q)[row * p.ldq + kh * p.Dp + i]), k = to_float(static_cast<const T*>(p.k)[row * p.ldk + kh * p.Dp + i]);
      sq[i] = q;
      sk[i] = k;
      x = fmaf(q, q, x);
      y = fmaf(k, k, y);
      z = kKind == kWkv ? fmaf(q * p.bonus[h * p.Dp + i], k, z) : fmaf(q, k, z);
      if (kKind == kWkv) sw[i] = wkv_decay(to_float(static_cast<const T*>(p.decay)[row * p.ld_decay + h * p.Dp + i]), p.decay_base[h * p.Dp + i]);
    }
    z = cta_sum(z, red);
    float g = 1.f, beta = 1.f;
    if (kKind == kDelta) {
      const float iq = 1.f / (sqrtf(cta_sum(x, red) + 1e-6f) * sqrtf(static_cast<float>(p.D))), ik = 1.f / sqrtf(cta_sum(y, red) + 1e-6f);
      z *= iq * ik;
      for (int i = threadIdx.x; i < p.Dp; i += blockDim.x) {
        sq[i] *= iq;
        sk[i] *= ik;
      }
      g = delta_decay(to_float(static_cast<const T*>(p.decay)[row * p.ld_decay + h]), p.decay_base[h], p.decay_bias[h]);
      beta = 1.f / (1.f + expf(-to_float(static_cast<const T*>(p.beta)[row * p.ld_decay + h])));
    }
    __syncthreads();
    float ss = 0.f;
    for (int c = threadIdx.x; c < p.Ep; c += blockDim.x) {
      const float v = to_float(static_cast<const T*>(p.v)[row * p.ldv + h * p.Ep + c]);
      float o = 0.f, d = 0.f;
      for (int i = 0; i < p.Dp; ++i) {
        const float s = state[static_cast<size_t>(i) * p.Ep + c];
        o = fmaf(sq[i], s, o);
        if (kKind == kDelta) d = fmaf(sk[i], s, d);
      }
      d = kKind == kDelta ? beta * (v - g * d) : v;
      for (int i = 0; i < p.Dp; ++i) {
        float* s = state + static_cast<size_t>(i) * p.Ep + c;
        *s = fmaf(sk[i], d, (kKind == kDelta ? g : sw[i]) * *s);
      }
      o = fmaf(z, d, g * o);
      so[c] = o;
      ss = fmaf(o, o, ss);
    }
    const float inv = 1.f / sqrtf(cta_sum(ss, red) / p.E + p.eps);
    for (int c = threadIdx.x; c < p.Ep; c += blockDim.x)
      static_cast<T*>(p.out)[row * p.H * p.Ep + h * p.Ep + c] = from_float<T>(
          so[c] * inv * p.gain[h * p.gain_stride + c] * silu(to_float(static_cast<const T*>(p.gate)[row * p.ldg + h * p.Ep + c])));
  }
}

template <typename T, int kKind, int kP, int R>
static int launch_recurrent(const RecurrentParams& p, int B, cudaStream_t s) {
  static bool configured[64] = {false};
  int dev = 0;
  B200_CHECK_CUDA(cudaGetDevice(&dev));
  if (!configured[dev & 63]) {
    B200_CHECK_CUDA(cudaFuncSetAttribute(recurrent_kernel<T, kKind, kP, R>, cudaFuncAttributeMaxDynamicSharedMemorySize, recurrent_smem(kP, sizeof(T))));
    configured[dev & 63] = true;
  }
  B200_CHECK_CUDA(launch_pdl(recurrent_kernel<T, kKind, kP, R>, dim3(p.H, B), dim3(kP * kP / (R * 4)), recurrent_smem(kP, sizeof(T)), s, p));
  return kOk;
}

template <typename T, int kKind>
static int dispatch_recurrent(const RecurrentParams& p, int B, int plain, cudaStream_t s) {
  const int size = p.Dp > p.Ep ? p.Dp : p.Ep;
  if (!plain && size <= 64) return launch_recurrent<T, kKind, 64, 8>(p, B, s);
  if (!plain && size <= 128) return launch_recurrent<T, kKind, 128, 16>(p, B, s);
  const int smem = (3 * p.Dp + p.Ep) * 4;
  B200_REQUIRE(smem <= 48 * 1024, "heads of %d x %d are too large", p.Dp, p.Ep);
  B200_CHECK_CUDA(launch_pdl(recurrent_plain_kernel<T, kKind>, dim3(p.H, B), dim3(256), smem, s, p));
  return kOk;
}

template <int kKind>
static int run_recurrent(const RecurrentParams& p, int B, int Hk, int plain, int dtype, void* stream) {
  if (B <= 0 || p.S <= 0) return kOk;
  B200_REQUIRE(p.H >= 1 && Hk >= 1 && p.H % Hk == 0 && B <= 65535, "heads (%d) must be a multiple of the key heads (%d)", p.H, Hk);
  B200_REQUIRE(p.D >= 1 && p.E >= 1 && p.Dp >= p.D && p.Ep >= p.E && p.Dp % 8 == 0 && p.Ep % 8 == 0, "bad head sizes %d / %d, %d / %d", p.D,
               p.Dp, p.E, p.Ep);
  B200_REQUIRE((p.ldq | p.ldk | p.ldv | p.ldg) % 8 == 0 && (kKind == kDelta || p.ld_decay % 8 == 0), "row pitches must be multiples of 8");
  B200_DISPATCH_FLOAT(dtype, return (dispatch_recurrent<T, kKind>(p, B, plain, static_cast<cudaStream_t>(stream))););
}

}  // namespace b200

using namespace b200;

// out[t, g, :] = h[t] + (h[t - 1] - h[t]) * mu[g]; the row before the first one is last[b], which becomes the call's last row.
B200_API int b200_token_mix(const void* h, const void* mu, void* last, void* out, int B, int S, int G, int pitch, int dtype, void* stream) {
  if (B <= 0 || S <= 0) return kOk;
  B200_REQUIRE(G >= 1 && G <= kMixMax && pitch % 4 == 0 && B <= 65535, "token_mix: 1..%d mixes and a pitch in multiples of 4", kMixMax);
  const TokenMixParams p{h, mu, last, out, S, G, pitch};
  const dim3 grid((pitch / 4 + 127) / 128, (S + kMixTokens - 1) / kMixTokens, B);
  B200_REQUIRE(grid.y <= 65535, "token_mix: too many tokens");
  cudaStream_t s = static_cast<cudaStream_t>(stream);
#define B200_MIX(N) case N: B200_CHECK_CUDA(launch_pdl(token_mix_kernel<T, N>, grid, dim3(128), 0, s, p)); return kOk;
  B200_DISPATCH_FLOAT(dtype, switch (G) { B200_MIX(1) B200_MIX(2) B200_MIX(3) B200_MIX(4) B200_MIX(5) B200_MIX(6) B200_MIX(7) B200_MIX(8) });
#undef B200_MIX
  return kOk;
}

// out = silu(sum_j taps[j] * x[t - n + 1 + j]); last [B, n - 1, C] carries the inputs before the call. C and ldx: multiples of 4.
B200_API int b200_short_conv(const void* x, const float* taps, void* last, void* out, int B, int S, int C, int n, int ldx, int dtype,
                             void* stream) {
  if (B <= 0 || S <= 0) return kOk;
  B200_REQUIRE(n >= 1 && C % 4 == 0 && ldx % 4 == 0 && B <= 65535, "short_conv: channels (%d) and pitch (%d) must be multiples of 4", C, ldx);
  const ShortConvParams p{x, taps, last, out, S, C, n, ldx};
  const dim3 grid((C / 4 + 127) / 128, (S + kConvTokens - 1) / kConvTokens, B);
  B200_REQUIRE(grid.y <= 65535, "short_conv: too many tokens");
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  B200_DISPATCH_FLOAT(dtype,
                      if (n == 4) B200_CHECK_CUDA(launch_pdl(short_conv_kernel<T, 4>, grid, dim3(128), 0, s, p));
                      else if (n == 3) B200_CHECK_CUDA(launch_pdl(short_conv_kernel<T, 3>, grid, dim3(128), 0, s, p));
                      else if (n == 2) B200_CHECK_CUDA(launch_pdl(short_conv_kernel<T, 2>, grid, dim3(128), 0, s, p));
                      else B200_CHECK_CUDA(launch_pdl(short_conv_kernel<T, 0>, grid, dim3(128), 0, s, p));
                      return kOk;);
}

// Decayed outer products. r, k, z [T, H * Dp], v, gate [T, H * Ep] with their row pitches; w0, u fp32 [H * Dp]; gain fp32 [H * Ep];
// state fp32 [B, H, Dp, Ep]; out [T, H * Ep]. plain != 0 forces the kernel for any head size.
B200_API int b200_wkv(const void* r, int ldr, const void* k, int ldk, const void* v, int ldv, const void* z, int ldz, const void* gate, int ldg,
                      const float* w0, const float* u, const float* gain, float eps, float* state, void* out, int B, int S, int H, int D,
                      int Dp, int E, int Ep, int plain, int dtype, void* stream) {
  RecurrentParams p;
  memset(&p, 0, sizeof(p));
  p.q = r; p.ldq = ldr; p.k = k; p.ldk = ldk; p.v = v; p.ldv = ldv; p.decay = z; p.ld_decay = ldz; p.gate = gate; p.ldg = ldg;
  p.decay_base = w0; p.bonus = u; p.gain = gain; p.gain_stride = Ep; p.eps = eps; p.state = state; p.out = out;
  p.S = S; p.H = H; p.per = 1; p.D = D; p.Dp = Dp; p.E = E; p.Ep = Ep;
  return run_recurrent<kWkv>(p, B, H, plain, dtype, stream);
}

// Gated delta rule. q, k [T, G * Dp], v, gate [T, H * Ep], a, b [T, H] with their row pitches; A, dt fp32 [H]; gain fp32 [Ep]; state
// fp32 [B, H, Dp, Ep]; out [T, H * Ep]. Head h reads q / k head h / (H / G).
B200_API int b200_gated_delta(const void* q, int ldq, const void* k, int ldk, const void* v, int ldv, const void* a, const void* b, int lda,
                              const void* gate, int ldg, const float* A, const float* dt, const float* gain, float eps, float* state,
                              void* out, int B, int S, int H, int G, int D, int Dp, int E, int Ep, int plain, int dtype, void* stream) {
  RecurrentParams p;
  memset(&p, 0, sizeof(p));
  B200_REQUIRE(G >= 1, "gated_delta needs at least one key head");
  p.q = q; p.ldq = ldq; p.k = k; p.ldk = ldk; p.v = v; p.ldv = ldv; p.decay = a; p.beta = b; p.ld_decay = lda; p.gate = gate; p.ldg = ldg;
  p.decay_base = A; p.decay_bias = dt; p.gain = gain; p.gain_stride = 0; p.eps = eps; p.state = state; p.out = out;
  p.S = S; p.H = H; p.per = H / G; p.D = D; p.Dp = Dp; p.E = E; p.Ep = Ep;
  return run_recurrent<kDelta>(p, B, G, plain, dtype, stream);
}
