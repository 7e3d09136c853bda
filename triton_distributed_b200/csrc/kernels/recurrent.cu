// Token mixers whose memory is a matrix per head, S [key size, value size] in fp32, carried from token to token:
//
//   decayed outer products (kWkv)   o_t = S^T r_t + (r_t . (u * k_t)) v_t;            S <- diag(w_t) S + k_t v_t^T
//                                   with w_t = exp(-exp(z_t + w0)) per key channel and a bonus u for the current token
//   gated delta rule (kDelta)       a = S^T k_t;  d = beta_t (v_t - g_t a);           S <- g_t S + k_t d^T;  o_t = S^T q_t
//                                   with g_t = exp(-exp(A) softplus(a_t + dt)) and beta_t = sigmoid(b_t) per head, q and k
//                                   scaled to unit length (q also by key_size^-0.5)
// Both end in the same way: o divided by its root mean square over the head, times a gain, times silu(gate).
//
// The columns of S never mix, and all of S stays in registers for the whole call. One CTA owns one head of one sequence; a
// thread owns R rows x 4 columns, the eight threads that share columns are neighbouring lanes and reduce with shuffles. Tokens go
// through shared memory in chunks of 16; the next chunk's copies are in flight while a chunk is computed. All arithmetic is
// fp32 on the CUDA cores (two products per instruction), so the fp32 pipe is what bounds a long call. To save its instructions
// four tokens share a pass over S: what they owe each other is a 4 x 4 triangle of scalars (see the kernel).
// Heads of up to 128 x 128 run this way (`recurrent_kernel`; calls of one token `recurrent_step_kernel`); larger ones keep S in
// global memory (`recurrent_plain_kernel`).
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

// ------------------------------------------------------------------------------------------------ tanh of a column slice
template <typename T>
__global__ void __launch_bounds__(256) tanh_rows_kernel(const T* x, T* out, int rows, int cols, int ldx) {
  const int groups = cols / 4;
  const size_t at = blockIdx.x * static_cast<size_t>(blockDim.x) + threadIdx.x;
  griddep_launch_dependents();
  griddep_wait();
  if (at >= static_cast<size_t>(rows) * groups) return;
  const size_t t = at / groups;
  const int c = static_cast<int>(at - t * groups) * 4;
  const float4 v = load4(x + t * ldx + c);
  store4(out + t * cols + c, make_float4(tanh_t<T>(v.x), tanh_t<T>(v.y), tanh_t<T>(v.z), tanh_t<T>(v.w)));
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
    store4(out + static_cast<size_t>(t) * p.C, make_float4(silu<T>(acc.x), silu<T>(acc.y), silu<T>(acc.z), silu<T>(acc.w)));
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
template <typename T>
__device__ __forceinline__ float wkv_decay(float z, float base) { return exp_t<T>(-exp_t<T>(z + base)); }
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
constexpr int kRecGroup = 4;     // tokens per pass over the memory
constexpr int kRecGroups = kRecTokens / kRecGroup;
constexpr int recurrent_smem(int p, int elem) {
  return (4 * kRecTokens * p + kRecGroups * p + 3 * p + kRecTokens * 8 + kRecGroups * 32 + 4 * kRecTokens) * 4 + 5 * kRecTokens * p * elem;
}

// sums over the warp of N = 16 or 32 values; lane l is left with the sum of v[l % N]
template <int N>
__device__ __forceinline__ float warp_sums(float (&v)[N]) {
  const int lane = threadIdx.x & 31;
#pragma unroll
  for (int m = N / 2; m > 0; m >>= 1) {
    const bool hi = (lane & m) != 0;
#pragma unroll
    for (int i = 0; i < m; ++i) v[i] = (hi ? v[i + m] : v[i]) + __shfl_xor_sync(0xffffffffu, hi ? v[i] : v[i + m], m);
  }
  return N == 32 ? v[0] : v[0] + __shfl_xor_sync(0xffffffffu, v[0], 16);
}

// V consecutive elements of shared memory as floats
template <typename T, int V>
__device__ __forceinline__ void load_few(const T* src, float (&f)[V]) {
  if (V == 4) {
    const float4 x = load4(src);
    f[0] = x.x; f[1] = x.y; f[V - 2] = x.z; f[V - 1] = x.w;
  } else if (sizeof(T) == 4) {
    const float2 x = *reinterpret_cast<const float2*>(src);
    f[0] = x.x; f[1] = x.y;
  } else {
    const uint32_t x = *reinterpret_cast<const uint32_t*>(src);
    f[0] = to_float(reinterpret_cast<const T*>(&x)[0]); f[1] = to_float(reinterpret_cast<const T*>(&x)[1]);
  }
}
template <int V>
__device__ __forceinline__ void store_few(float* dst, const float (&f)[V]) {
  if (V == 4) *reinterpret_cast<float4*>(dst) = make_float4(f[0], f[1], f[V - 2], f[V - 1]);
  else *reinterpret_cast<float2*>(dst) = make_float2(f[0], f[1]);
}

// kP: padded key and value size; a thread owns R = kP / 8 rows (groups of four, eight lanes apart) and four columns.
// Four tokens are taken in one pass over S. With S the memory in front of them, tokens 0..3:
//   kWkv    o_i = S^T (r_i * prod_{l<i} w_l) + sum_{j<i} (sum_d r_i k_j prod_{j<l<i} w_l) v_j + (r_i . (u * k_i)) v_i
//           S  <- diag(prod w) S + sum_j (k_j * prod_{l>j} w_l) v_j^T
//   kDelta  with G_ij = prod_{j<l<=i} g_l, c_i = prod_{l<=i} g_l:
//           d_i = beta_i (v_i - c_i S^T k_i - sum_{j<i} G_ij (k_j . k_i) d_j),   o_i = c_i S^T q_i + sum_{j<=i} G_ij (k_j . q_i) d_j
//           S  <- c_3 S + sum_j G_3j k_j d_j^T
// The scaled vectors and the sums over key channels are prepared per chunk, one warp per four tokens. Tokens behind the end of the
// call count as w = g = 1, k = 0.
template <typename T, int kKind, int kP>
__global__ void __launch_bounds__(2 * kP, kP == 128 ? 2 : 4) recurrent_kernel(const RecurrentParams p) {
  constexpr int R = kP / 8, C = 4, kThreads = 2 * kP, kWarps = kThreads / 32, V = kP / 32;
  constexpr int kRaw = kRecTokens * kP;
  static_assert(kWarps == 4 || kWarps == 8, "one warp per group of tokens");
  extern __shared__ __align__(16) float smf[];
  float* sq = smf;                            // [tokens][kP] read-out vectors
  float* sk = sq + kRaw;                      // [tokens][kP]
  float* sv = sk + kRaw;
  float* so = sv + kRaw;
  float* sw = so + kRaw;                      // kWkv: [groups][kP] product of the decays
  float* s_base = sw + kRecGroups * kP;       // kWkv: w0 and u of the head
  float* s_bonus = s_base + kP;
  float* s_gain = s_bonus + kP;
  float* s_n = s_gain + kP;                   // [tokens][4] coefficients of o_i on v_j (kWkv) / d_j (kDelta)
  float* s_m = s_n + kRecTokens * 4;          // kDelta: [tokens][4] coefficients of d_i on d_j
  float* s_dot = s_m + kRecTokens * 4;        // [groups][32]
  float* s_c = s_dot + kRecGroups * 32;       // kDelta: c_i, G_3i, beta_i, g_i per token
  float* s_tail = s_c + kRecTokens;
  float* s_beta = s_tail + kRecTokens;
  float* s_g = s_beta + kRecTokens;
  T* raw = reinterpret_cast<T*>(s_g + kRecTokens);   // [q, k, decay, v, gate][tokens][kP] of the next chunk as it lies in memory
  const int h = blockIdx.x, b = blockIdx.y, kh = h / p.per;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, kg = lane & 7;
  const int col0 = (warp * 4 + (lane >> 3)) * C;
  float* state = p.state + (static_cast<size_t>(b) * p.H + h) * p.Dp * p.Ep;
  griddep_launch_dependents();
  // the state comes from an earlier call: it may be fetched into L2, but not read, before that call is known to be over
  for (int i = threadIdx.x * 32; i < p.Dp * p.Ep; i += kThreads * 32) asm volatile("prefetch.global.L2 [%0];" ::"l"(state + i));
  const int ic = threadIdx.x % (kP / 8) * 8, it = threadIdx.x / (kP / 8);   // this thread's eight elements of a chunk
  if (threadIdx.x < kP) s_gain[threadIdx.x] = threadIdx.x < p.Ep ? p.gain[h * p.gain_stride + threadIdx.x] : 0.f;
  if (kKind == kWkv && threadIdx.x < kP) {
    const bool in = threadIdx.x < p.Dp;
    s_base[threadIdx.x] = in ? p.decay_base[h * p.Dp + threadIdx.x] : 0.f;
    s_bonus[threadIdx.x] = in ? p.bonus[h * p.Dp + threadIdx.x] : 0.f;
  }
  const float A = kKind == kDelta ? p.decay_base[h] : 0.f, dt = kKind == kDelta ? p.decay_bias[h] : 0.f;
  griddep_wait();

  float ra = 0.f, rb = 0.f;   // kDelta: logits of token 4 * warp + lane of the next chunk
  const size_t row0 = static_cast<size_t>(b) * p.S;
  auto fetch = [&](int t0) {
    const size_t row = row0 + t0 + it;
    T* dst = raw + it * kP + ic;
    const bool in = t0 + it < p.S, ink = in && ic < p.Dp, inv = in && ic < p.Ep;
    copy8<T>(dst, p.q, row * p.ldq + kh * p.Dp + ic, ink);
    copy8<T>(dst + kRaw, p.k, row * p.ldk + kh * p.Dp + ic, ink);
    if (kKind == kWkv) copy8<T>(dst + 2 * kRaw, p.decay, row * p.ld_decay + h * p.Dp + ic, ink);
    copy8<T>(dst + 3 * kRaw, p.v, row * p.ldv + h * p.Ep + ic, inv);
    copy8<T>(dst + 4 * kRaw, p.gate, row * p.ldg + h * p.Ep + ic, inv);
    cp_async_commit();
    const int tok = t0 + warp * kRecGroup + lane;
    if (kKind == kDelta && warp < kRecGroups && lane < kRecGroup && tok < p.S) {
      const size_t at = (row0 + tok) * p.ld_decay + h;
      ra = to_float(static_cast<const T*>(p.decay)[at]);
      rb = to_float(static_cast<const T*>(p.beta)[at]);
    }
  };
  fetch(0);

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
    const int n = min(kRecTokens, p.S - t0), n_groups = (n + kRecGroup - 1) / kRecGroup;
    cp_async_wait<0>();
    __syncthreads();   // the raw chunk of all threads; the last chunk's results have been read
    // ---- prepare: every thread its own values; warp w the vectors of group w, a lane V channels
    float gate[8];   // of this thread's results
    {
      float f[8];
      load8(raw + 3 * kRaw + it * kP + ic, f);
      store8(sv + it * kP + ic, f);
      load8(raw + 4 * kRaw + it * kP + ic, gate);
    }
    if (warp < n_groups) {
      float q[kRecGroup][V], k[kRecGroup][V];
#pragma unroll
      for (int i = 0; i < kRecGroup; ++i) {
        load_few<T, V>(raw + (warp * kRecGroup + i) * kP + lane * V, q[i]);
        load_few<T, V>(raw + kRaw + (warp * kRecGroup + i) * kP + lane * V, k[i]);
      }
      if (kKind == kWkv) {
        float w[kRecGroup][V], x[16], total[V];
#pragma unroll
        for (int i = 0; i < kRecGroup; ++i) {
          load_few<T, V>(raw + 2 * kRaw + (warp * kRecGroup + i) * kP + lane * V, w[i]);
#pragma unroll
          for (int e = 0; e < V; ++e) w[i][e] = warp * kRecGroup + i < n ? wkv_decay<T>(w[i][e], s_base[lane * V + e]) : 1.f;
        }
#pragma unroll
        for (int i = 0; i < 16; ++i) x[i] = 0.f;
#pragma unroll
        for (int e = 0; e < V; ++e) {
          const float u = s_bonus[lane * V + e];
#pragma unroll
          for (int i = 0; i < kRecGroup; ++i) {
            x[4 * i + i] = fmaf(q[i][e] * u, k[i][e], x[4 * i + i]);
            float rw = q[i][e];   // r_i times the decays between the two tokens
#pragma unroll
            for (int j = i - 1; j >= 0; --j) {
              x[4 * i + j] = fmaf(rw, k[j][e], x[4 * i + j]);
              rw *= w[j][e];
            }
            q[i][e] = rw;         // now times the decays of all earlier tokens of the group
          }
          float after = 1.f;
#pragma unroll
          for (int j = kRecGroup - 1; j >= 0; --j) {
            k[j][e] *= after;
            after *= w[j][e];
          }
          total[e] = after;
        }
        store_few<V>(sw + warp * kP + lane * V, total);
        const float dot = warp_sums<16>(x);
        if (lane < 16) s_n[warp * 16 + lane] = dot;
      } else {
        float x[32];
#pragma unroll
        for (int i = 0; i < 32; ++i) x[i] = 0.f;
#pragma unroll
        for (int e = 0; e < V; ++e)
#pragma unroll
          for (int i = 0; i < kRecGroup; ++i) {
            x[16 + i] = fmaf(q[i][e], q[i][e], x[16 + i]);
            x[20 + i] = fmaf(k[i][e], k[i][e], x[20 + i]);
#pragma unroll
            for (int j = 0; j < kRecGroup; ++j) x[4 * i + j] = fmaf(j <= i ? q[i][e] : k[i][e], k[j][e], x[4 * i + j]);  // k_j . q_i, or k_i . k_j
          }
        float* dot = s_dot + warp * 32;
        const int tok = warp * kRecGroup + lane;
        dot[lane] = warp_sums<32>(x);
        if (lane < kRecGroup) {
          s_g[tok] = tok < n ? delta_decay(ra, A, dt) : 1.f;
          s_beta[tok] = tok < n ? 1.f / (1.f + expf(-rb)) : 0.f;
        }
        __syncwarp();
        const float* g = s_g + warp * kRecGroup;
        const float root = sqrtf(static_cast<float>(p.D));
        if (lane < 16) {
          const int i = lane >> 2, j = lane & 3, lo = min(i, j), hi = max(i, j);
          float G = dot[lane] / sqrtf(dot[20 + j] + 1e-6f);
          for (int l = lo + 1; l <= hi; ++l) G *= g[l];
          if (j <= i) s_n[(warp * kRecGroup + i) * 4 + j] = G / (sqrtf(dot[16 + i] + 1e-6f) * root);
          else s_m[(warp * kRecGroup + j) * 4 + i] = G / sqrtf(dot[20 + i] + 1e-6f);
        } else if (lane < 16 + kRecGroup) {
          const int i = lane - 16;
          float c = 1.f, tail = 1.f;
          for (int l = 0; l <= i; ++l) c *= g[l];
          for (int l = i + 1; l < kRecGroup; ++l) tail *= g[l];
          s_c[warp * kRecGroup + i] = c;
          s_tail[warp * kRecGroup + i] = tail;
        }
#pragma unroll
        for (int i = 0; i < kRecGroup; ++i) {
          const float iq = 1.f / (sqrtf(dot[16 + i] + 1e-6f) * root), ik = 1.f / sqrtf(dot[20 + i] + 1e-6f);
#pragma unroll
          for (int e = 0; e < V; ++e) {
            q[i][e] *= iq;
            k[i][e] *= ik;
          }
        }
      }
#pragma unroll
      for (int i = 0; i < kRecGroup; ++i) {
        store_few<V>(sq + (warp * kRecGroup + i) * kP + lane * V, q[i]);
        store_few<V>(sk + (warp * kRecGroup + i) * kP + lane * V, k[i]);
      }
    }
    __syncthreads();
    if (t0 + kRecTokens < p.S) fetch(t0 + kRecTokens);
    // ---- the tokens of the chunk
#pragma unroll 1
    for (int grp = 0; grp < n_groups; ++grp) {
      const int tok = grp * kRecGroup;
      // four rows of this thread out of a row vector
      auto four = [&](const float* x, int i) { return *reinterpret_cast<const ulonglong2*>(x + 32 * i + 4 * kg); };
      // per-token partial sums of this thread's rows with the memory
      auto products = [&](const float* x, float (&o)[kRecGroup][C]) {
        f32x2 acc[kRecGroup][C];
#pragma unroll
        for (int i = 0; i < R / 4; ++i)
#pragma unroll
          for (int t = 0; t < kRecGroup; ++t) {
            const ulonglong2 x2 = four(x + (tok + t) * kP, i);
#pragma unroll
            for (int c = 0; c < C; ++c) {
              acc[t][c] = i == 0 ? mul2(x2.x, s[0][c]) : fma2(x2.x, s[2 * i][c], acc[t][c]);
              acc[t][c] = fma2(x2.y, s[2 * i + 1][c], acc[t][c]);
            }
          }
#pragma unroll
        for (int t = 0; t < kRecGroup; ++t)
#pragma unroll
          for (int c = 0; c < C; ++c) o[t][c] = sum2(acc[t][c]);
      };
      const bool b2 = (kg & 4) != 0, b1 = (kg & 2) != 0, b0 = (kg & 1) != 0;
      if (kKind == kWkv) {
        float o[kRecGroup][C];
        products(sq, o);
        // sums over the eight lanes; lane kg is left with token kg >> 1 and a pair of columns
        float x[2][C], y[C], z[2];
#pragma unroll
        for (int t = 0; t < 2; ++t)
#pragma unroll
          for (int c = 0; c < C; ++c) x[t][c] = (b2 ? o[t + 2][c] : o[t][c]) + __shfl_xor_sync(0xffffffffu, b2 ? o[t][c] : o[t + 2][c], 4);
#pragma unroll
        for (int c = 0; c < C; ++c) y[c] = (b1 ? x[1][c] : x[0][c]) + __shfl_xor_sync(0xffffffffu, b1 ? x[0][c] : x[1][c], 2);
#pragma unroll
        for (int c = 0; c < 2; ++c) z[c] = (b0 ? y[c + 2] : y[c]) + __shfl_xor_sync(0xffffffffu, b0 ? y[c] : y[c + 2], 1);
        f32x2 v2[kRecGroup][C];
#pragma unroll
        for (int t = 0; t < kRecGroup; ++t) {
          const float4 v = *reinterpret_cast<const float4*>(sv + (tok + t) * kP + col0);
          v2[t][0] = pack2(v.x, v.x); v2[t][1] = pack2(v.y, v.y); v2[t][2] = pack2(v.z, v.z); v2[t][3] = pack2(v.w, v.w);
        }
#pragma unroll
        for (int i = 0; i < R / 4; ++i) {
          const ulonglong2 w2 = four(sw + grp * kP, i);
#pragma unroll
          for (int c = 0; c < C; ++c) {
            s[2 * i][c] = mul2(w2.x, s[2 * i][c]);
            s[2 * i + 1][c] = mul2(w2.y, s[2 * i + 1][c]);
          }
#pragma unroll
          for (int t = 0; t < kRecGroup; ++t) {
            const ulonglong2 k2 = four(sk + (tok + t) * kP, i);
#pragma unroll
            for (int c = 0; c < C; ++c) {
              s[2 * i][c] = fma2(k2.x, v2[t][c], s[2 * i][c]);
              s[2 * i + 1][c] = fma2(k2.y, v2[t][c], s[2 * i + 1][c]);
            }
          }
        }
        const int mine = tok + (kg >> 1), col = col0 + 2 * (kg & 1);
        const float4 co = *reinterpret_cast<const float4*>(s_n + mine * 4);
        const float f[kRecGroup] = {co.x, co.y, co.z, co.w};
#pragma unroll
        for (int j = 0; j < kRecGroup; ++j) {
          const float2 v = *reinterpret_cast<const float2*>(sv + (tok + j) * kP + col);
          z[0] = fmaf(f[j], v.x, z[0]);
          z[1] = fmaf(f[j], v.y, z[1]);
        }
        *reinterpret_cast<float2*>(so + mine * kP + col) = make_float2(z[0], z[1]);
      } else {
        // sums over the eight lanes; lanes kg and kg ^ 1 are left with column kg >> 1, all four tokens
        auto column_sums = [&](const float (&o)[kRecGroup][C], float (&r)[kRecGroup]) {
          float x[kRecGroup][2];
#pragma unroll
          for (int t = 0; t < kRecGroup; ++t)
#pragma unroll
            for (int c = 0; c < 2; ++c) x[t][c] = (b2 ? o[t][c + 2] : o[t][c]) + __shfl_xor_sync(0xffffffffu, b2 ? o[t][c] : o[t][c + 2], 4);
#pragma unroll
          for (int t = 0; t < kRecGroup; ++t) r[t] = (b1 ? x[t][1] : x[t][0]) + __shfl_xor_sync(0xffffffffu, b1 ? x[t][0] : x[t][1], 2);
#pragma unroll
          for (int t = 0; t < kRecGroup; ++t) r[t] += __shfl_xor_sync(0xffffffffu, r[t], 1);
        };
        float part[kRecGroup][C], a[kRecGroup], o[kRecGroup], d[kRecGroup];
        products(sk, part);
        column_sums(part, a);
        products(sq, part);
        column_sums(part, o);
        const int col = col0 + (kg >> 1);
        float c4[4], beta[4], tail[4];
        load_few<float, 4>(s_c + tok, c4);
        load_few<float, 4>(s_beta + tok, beta);
        load_few<float, 4>(s_tail + tok, tail);
#pragma unroll
        for (int i = 0; i < kRecGroup; ++i) {
          float m[4], e[4];
          load_few<float, 4>(s_m + (tok + i) * 4, m);
          load_few<float, 4>(s_n + (tok + i) * 4, e);
          float t = fmaf(-c4[i], a[i], sv[(tok + i) * kP + col]);
#pragma unroll
          for (int j = 0; j < i; ++j) t = fmaf(-m[j], d[j], t);
          d[i] = beta[i] * t;
          o[i] *= c4[i];
#pragma unroll
          for (int j = 0; j <= i; ++j) o[i] = fmaf(e[j], d[j], o[i]);
        }
        so[(tok + (b0 ? 2 : 0)) * kP + col] = b0 ? o[2] : o[0];
        so[(tok + (b0 ? 3 : 1)) * kP + col] = b0 ? o[3] : o[1];
        f32x2 d2[kRecGroup][C];   // the weighted d of the thread's four columns
#pragma unroll
        for (int t = 0; t < kRecGroup; ++t) {
          const float own = tail[t] * d[t], near = __shfl_xor_sync(0xffffffffu, own, 2);
          const float p0 = b1 ? near : own, p1 = b1 ? own : near;
          const float f0 = __shfl_xor_sync(0xffffffffu, p0, 4), f1 = __shfl_xor_sync(0xffffffffu, p1, 4);
          const float e[C] = {b2 ? f0 : p0, b2 ? f1 : p1, b2 ? p0 : f0, b2 ? p1 : f1};
#pragma unroll
          for (int c = 0; c < C; ++c) d2[t][c] = pack2(e[c], e[c]);
        }
        const f32x2 g2 = pack2(c4[kRecGroup - 1], c4[kRecGroup - 1]);
#pragma unroll
        for (int i = 0; i < R / 4; ++i) {
#pragma unroll
          for (int c = 0; c < C; ++c) {
            s[2 * i][c] = mul2(g2, s[2 * i][c]);
            s[2 * i + 1][c] = mul2(g2, s[2 * i + 1][c]);
          }
#pragma unroll
          for (int t = 0; t < kRecGroup; ++t) {
            const ulonglong2 k2 = four(sk + (tok + t) * kP, i);
#pragma unroll
            for (int c = 0; c < C; ++c) {
              s[2 * i][c] = fma2(k2.x, d2[t][c], s[2 * i][c]);
              s[2 * i + 1][c] = fma2(k2.y, d2[t][c], s[2 * i + 1][c]);
            }
          }
        }
      }
    }
    __syncthreads();
    // ---- norm over the head, gain, gate: eight columns of a token per thread
    {
      float o[8], ss = 0.f;
      load8(so + it * kP + ic, o);
#pragma unroll
      for (int i = 0; i < 8; ++i) ss = fmaf(o[i], o[i], ss);
#pragma unroll
      for (int m = kP / 16; m > 0; m >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, m);
      const float inv = inv_sqrt<T>(ss / p.E + p.eps);
      if (it < n && ic < p.Ep) {
        float f[8];
        load8(s_gain + ic, f);
#pragma unroll
        for (int i = 0; i < 8; ++i) f[i] *= o[i] * inv * silu<T>(gate[i]);
        T* dst = static_cast<T*>(p.out) + (row0 + t0 + it) * p.H * p.Ep + h * p.Ep + ic;
        store4(dst, make_float4(f[0], f[1], f[2], f[3]));
        store4(dst + 4, make_float4(f[4], f[5], f[6], f[7]));
      }
    }
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

// One token per sequence: bound by reading and writing S once. The layout of recurrent_kernel, one token at a time; q and k keep
// their length, which enters as a factor.
template <typename T, int kKind, int kP>
__global__ void __launch_bounds__(2 * kP) recurrent_step_kernel(const RecurrentParams p) {
  constexpr int R = kP / 8, kWarps = kP / 16, kThreads = 2 * kP;
  __shared__ __align__(16) float sq[kP], sk[kP], sw[kP], sv[kP], so[kP];
  __shared__ float red[3][kWarps];
  const int h = blockIdx.x, b = blockIdx.y, kh = h / p.per;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, kg = lane & 7;
  const int col0 = (warp * 4 + (lane >> 3)) * 4, ch = threadIdx.x;
  float* state = p.state + (static_cast<size_t>(b) * p.H + h) * p.Dp * p.Ep;
  griddep_launch_dependents();
  // the state comes from an earlier call: it may be fetched into L2, but not read, before that call is known to be over
  for (int i = threadIdx.x * 32; i < p.Dp * p.Ep; i += kThreads * 32) asm volatile("prefetch.global.L2 [%0];" ::"l"(state + i));
  const float base = kKind == kWkv && ch < p.Dp ? p.decay_base[h * p.Dp + ch] : 0.f, bonus = kKind == kWkv && ch < p.Dp ? p.bonus[h * p.Dp + ch] : 0.f;
  const float gain = ch < p.Ep ? p.gain[h * p.gain_stride + ch] : 0.f;
  griddep_wait();
  float q = 0.f, k = 0.f, z = 0.f, v = 0.f, gate = 0.f, g = 1.f, beta = 1.f;
  const size_t row = b;
  if (ch < p.Dp) {
    q = to_float(static_cast<const T*>(p.q)[row * p.ldq + kh * p.Dp + ch]);
    k = to_float(static_cast<const T*>(p.k)[row * p.ldk + kh * p.Dp + ch]);
    if (kKind == kWkv) z = to_float(static_cast<const T*>(p.decay)[row * p.ld_decay + h * p.Dp + ch]);
  }
  if (ch < p.Ep) {
    v = to_float(static_cast<const T*>(p.v)[row * p.ldv + h * p.Ep + ch]);
    gate = to_float(static_cast<const T*>(p.gate)[row * p.ldg + h * p.Ep + ch]);
  }
  if (kKind == kDelta) {
    g = to_float(static_cast<const T*>(p.decay)[row * p.ld_decay + h]);
    beta = to_float(static_cast<const T*>(p.beta)[row * p.ld_decay + h]);
  }
  float4 s[R];   // s[4 i + e] = row 32 i + 4 kg + e, columns col0 ...
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int r = 32 * (i >> 2) + 4 * kg + (i & 3);
    s[i] = r < p.Dp && col0 < p.Ep ? *reinterpret_cast<const float4*>(state + static_cast<size_t>(r) * p.Ep + col0) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  if (ch < kP) {
    sq[ch] = q;
    sk[ch] = k;
    sv[ch] = v;
    if (kKind == kWkv) sw[ch] = wkv_decay<T>(z, base);
  }
  // sums over the key channels
  const float x = warp_sum(kKind == kWkv ? q * bonus * k : q * k);
  const float y = kKind == kDelta ? warp_sum(q * q) : 0.f, w = kKind == kDelta ? warp_sum(k * k) : 0.f;
  if (lane == 0) {
    red[0][warp] = x;
    red[1][warp] = y;
    red[2][warp] = w;
  }
  __syncthreads();
  float qk = 0.f, qq = 0.f, kk = 0.f;
#pragma unroll
  for (int i = 0; i < kP / 32; ++i) {
    qk += red[0][i];
    if (kKind == kDelta) {
      qq += red[1][i];
      kk += red[2][i];
    }
  }
  float iq = 1.f, ik = 1.f;
  if (kKind == kDelta) {
    iq = 1.f / (sqrtf(qq + 1e-6f) * sqrtf(static_cast<float>(p.D)));
    ik = 1.f / sqrtf(kk + 1e-6f);
    g = delta_decay(g, p.decay_base[h], p.decay_bias[h]);
    beta = 1.f / (1.f + expf(-beta));
  }
  const float4 v4 = *reinterpret_cast<const float4*>(sv + col0);
  float o[4] = {0.f, 0.f, 0.f, 0.f}, d[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
  for (int i = 0; i < R / 4; ++i) {
    float qr[4], kr[4];
    load_few<float, 4>(sq + 32 * i + 4 * kg, qr);
    if (kKind == kDelta) load_few<float, 4>(sk + 32 * i + 4 * kg, kr);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float4 t = s[4 * i + e];
      o[0] = fmaf(qr[e], t.x, o[0]); o[1] = fmaf(qr[e], t.y, o[1]); o[2] = fmaf(qr[e], t.z, o[2]); o[3] = fmaf(qr[e], t.w, o[3]);
      if (kKind == kDelta) {
        d[0] = fmaf(kr[e], t.x, d[0]); d[1] = fmaf(kr[e], t.y, d[1]); d[2] = fmaf(kr[e], t.z, d[2]); d[3] = fmaf(kr[e], t.w, d[3]);
      }
    }
  }
#pragma unroll
  for (int m = 1; m < 8; m <<= 1)
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      o[c] += __shfl_xor_sync(0xffffffffu, o[c], m);
      if (kKind == kDelta) d[c] += __shfl_xor_sync(0xffffffffu, d[c], m);
    }
  const float vv[4] = {v4.x, v4.y, v4.z, v4.w};
#pragma unroll
  for (int c = 0; c < 4; ++c) {
    d[c] = kKind == kDelta ? beta * fmaf(-g * ik, d[c], vv[c]) : vv[c];
    o[c] = iq * fmaf(ik * qk, d[c], g * o[c]);
    d[c] *= ik;
  }
  if (kg == 0) *reinterpret_cast<float4*>(so + col0) = make_float4(o[0], o[1], o[2], o[3]);
#pragma unroll
  for (int i = 0; i < R / 4; ++i) {
    float kr[4], wr[4];
    load_few<float, 4>(sk + 32 * i + 4 * kg, kr);
    if (kKind == kWkv) load_few<float, 4>(sw + 32 * i + 4 * kg, wr);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int r = 32 * i + 4 * kg + e;
      const float f = kKind == kWkv ? wr[e] : g;
      const float4 t = s[4 * i + e];
      if (r < p.Dp && col0 < p.Ep)
        *reinterpret_cast<float4*>(state + static_cast<size_t>(r) * p.Ep + col0) =
            make_float4(fmaf(kr[e], d[0], f * t.x), fmaf(kr[e], d[1], f * t.y), fmaf(kr[e], d[2], f * t.z), fmaf(kr[e], d[3], f * t.w));
    }
  }
  __syncthreads();
  // ---- norm over the head, gain, gate
  const float mine = ch < kP ? so[ch] : 0.f, part = warp_sum(mine * mine);
  if (lane == 0) red[0][warp] = part;
  __syncthreads();
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < kP / 32; ++i) ss += red[0][i];
  if (ch < p.Ep)
    static_cast<T*>(p.out)[row * p.H * p.Ep + h * p.Ep + ch] = from_float<T>(mine * inv_sqrt<T>(ss / p.E + p.eps) * gain * silu<T>(gate));
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
      if (kKind == kWkv) sw[i] = wkv_decay<T>(to_float(static_cast<const T*>(p.decay)[row * p.ld_decay + h * p.Dp + i]), p.decay_base[h * p.Dp + i]);
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
          so[c] * inv * p.gain[h * p.gain_stride + c] * silu<T>(to_float(static_cast<const T*>(p.gate)[row * p.ldg + h * p.Ep + c])));
  }
}

template <typename T, int kKind, int kP>
static int launch_recurrent(const RecurrentParams& p, int B, cudaStream_t s) {
  if (p.S == 1) {
    B200_CHECK_CUDA(launch_pdl(recurrent_step_kernel<T, kKind, kP>, dim3(p.H, B), dim3(2 * kP), 0, s, p));
    return kOk;
  }
  static bool configured[64] = {false};
  int dev = 0;
  B200_CHECK_CUDA(cudaGetDevice(&dev));
  if (!configured[dev & 63]) {
    B200_CHECK_CUDA(cudaFuncSetAttribute(recurrent_kernel<T, kKind, kP>, cudaFuncAttributeMaxDynamicSharedMemorySize, recurrent_smem(kP, sizeof(T))));
    configured[dev & 63] = true;
  }
  B200_CHECK_CUDA(launch_pdl(recurrent_kernel<T, kKind, kP>, dim3(p.H, B), dim3(2 * kP), recurrent_smem(kP, sizeof(T)), s, p));
  return kOk;
}

template <typename T, int kKind>
static int dispatch_recurrent(const RecurrentParams& p, int B, int plain, cudaStream_t s) {
  const int size = p.Dp > p.Ep ? p.Dp : p.Ep;
  if (!plain && size <= 64) return launch_recurrent<T, kKind, 64>(p, B, s);
  if (!plain && size <= 128) return launch_recurrent<T, kKind, 128>(p, B, s);
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

// out [rows, cols] = tanh(x), x with row pitch ldx; cols and ldx: multiples of 4.
B200_API int b200_tanh_rows(const void* x, void* out, int rows, int cols, int ldx, int dtype, void* stream) {
  if (rows <= 0) return kOk;
  B200_REQUIRE(cols >= 4 && cols % 4 == 0 && ldx % 4 == 0, "tanh_rows: columns (%d) and pitch (%d) must be multiples of 4", cols, ldx);
  const size_t n = static_cast<size_t>(rows) * (cols / 4);
  B200_DISPATCH_FLOAT(dtype, B200_CHECK_CUDA(launch_pdl(tanh_rows_kernel<T>, dim3(static_cast<unsigned>((n + 255) / 256)), dim3(256), 0,
                                                        static_cast<cudaStream_t>(stream), static_cast<const T*>(x), static_cast<T*>(out),
                                                        rows, cols, ldx));
                      return kOk;);
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
