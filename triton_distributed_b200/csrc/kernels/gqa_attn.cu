// Grouped-query attention for head sizes and storage types outside the 128-wide kernels.
//
//   head_norm_rope    per-head RMS norm and interleaved rotary positions of q and k (on the first `rot` dimensions of a head),
//                     the score scale multiplied into q, and the write of k and v to their cache slots, in one launch. Rows may be
//                     padded: the sizes that are read and written are the padded ones, statistics use the true size.
//   gqa_attention_plain   one warp per (query token, head), keys in groups of 32, fp32 arithmetic, any head sizes and storage type:
//                     the 32-bit mode and heads that the tensor-core kernels do not take
// Large-tile work goes through prefill_attn_sm100.cu, 128-wide decode through decode_attn.cu.
#include "b200/elem.cuh"
#include "b200/host.h"

#include <cstring>

namespace b200 {

struct HeadNormRopeParams {
  const void *q, *k, *v;      // [T, H * qk_in], [T, G * qk_in], [T, G * v_in] with one row pitch ld
  const void *gain_q, *gain_k;  // [D] or null (no norm)
  const float* cos_sin;       // [positions, rot] = (cos, sin) of pair 0, of pair 1, ...
  const int* positions;       // [T]
  const long long* slots;     // [T], < 0 = not stored
  void *q_out, *k_cache, *v_cache;  // [T, H, qk_out], [slots, G, qk_out], [slots, G, v_out]
  int T, H, G, D, rot, qk_in, qk_out, v_in, v_out, ld;
  float eps, q_scale;
};

// one warp per (token, head); a lane owns pairs of dimensions
template <typename T>
__global__ void __launch_bounds__(256) head_norm_rope_kernel(const HeadNormRopeParams p) {
  const int heads = p.H + 2 * p.G, lane = threadIdx.x & 31;
  const long long w = (static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x) >> 5;
  griddep_launch_dependents();
  griddep_wait();
  if (w >= static_cast<long long>(p.T) * heads) return;
  const size_t t = w / heads;
  const int h = static_cast<int>(w - static_cast<long long>(t) * heads);
  const long long slot = p.slots != nullptr ? p.slots[t] : static_cast<long long>(t);
  if (h >= p.H && slot < 0) return;
  if (h >= p.H + p.G) {  // values: copied, zero-padded
    const int g = h - p.H - p.G;
    const T* src = static_cast<const T*>(p.v) + t * p.ld + g * p.v_in;
    T* dst = static_cast<T*>(p.v_cache) + (static_cast<size_t>(slot) * p.G + g) * p.v_out;
    for (int c = 4 * lane; c < p.v_out; c += 128) store4(dst + c, c < p.v_in ? load4(src + c) : make_float4(0.f, 0.f, 0.f, 0.f));
    return;
  }
  const bool is_q = h < p.H;
  const T* src = is_q ? static_cast<const T*>(p.q) + t * p.ld + h * p.qk_in : static_cast<const T*>(p.k) + t * p.ld + (h - p.H) * p.qk_in;
  T* dst = is_q ? static_cast<T*>(p.q_out) + (t * p.H + h) * p.qk_out
                : static_cast<T*>(p.k_cache) + (static_cast<size_t>(slot) * p.G + (h - p.H)) * p.qk_out;
  const T* gain = static_cast<const T*>(is_q ? p.gain_q : p.gain_k);
  float inv = 1.f;
  if (gain != nullptr) {
    float ss = 0.f;
    for (int c = 4 * lane; c < p.qk_in; c += 128) {  // padding is zero
      const float4 x = load4(src + c);
      ss += (x.x * x.x + x.y * x.y) + (x.z * x.z + x.w * x.w);
    }
    inv = 1.f / sqrtf(warp_sum(ss) / p.D + p.eps);
  }
  const float* table = p.cos_sin + static_cast<size_t>(p.positions[t]) * p.rot;
  for (int c = 4 * lane; c < p.qk_out; c += 128) {
    float x[4] = {0.f, 0.f, 0.f, 0.f};
    if (c < p.qk_in) {
      const float4 f = load4(src + c);
      x[0] = f.x; x[1] = f.y; x[2] = f.z; x[3] = f.w;
    }
#pragma unroll
    for (int e = 0; e < 4; ++e)
      if (gain != nullptr) x[e] = c + e < p.D ? x[e] * inv * to_float(gain[c + e]) : 0.f;
#pragma unroll
    for (int e = 0; e < 4; e += 2)
      if (c + e < p.rot) {   // rot is even
        const float cs = table[c + e], sn = table[c + e + 1], a = x[e], b = x[e + 1];
        x[e] = a * cs - b * sn;
        x[e + 1] = b * cs + a * sn;
      }
    const float m = is_q ? p.q_scale : 1.f;
    store4(dst + c, make_float4(x[0] * m, x[1] * m, x[2] * m, x[3] * m));
  }
}

struct GqaPlainParams {
  const void* q;           // [B * S, H, dk]
  const void *k, *v;       // [blocks, page, G, dk], [blocks, page, G, dv]
  const int* block_table;  // [B, bt_stride]
  const int* kv_lens;      // [B] keys in the cache, the S new ones included
  const void* gate;        // [B * S, H] (row pitch ldg) or null: the output times sigmoid(gate)
  void* out;               // [B * S, H, dv]
  int bt_stride, page, H, G, S, dk, dv, ldg;
  float scale;
};

template <typename T>
__global__ void __launch_bounds__(128) gqa_attention_plain_kernel(const GqaPlainParams p) {
  extern __shared__ __align__(16) float fsm[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* q = fsm + warp * (p.dk + p.dv);
  float* o = q + p.dk;
  const int b = blockIdx.y, n_rows = p.S * p.H, r = blockIdx.x * 4 + warp;
  griddep_launch_dependents();
  griddep_wait();
  if (r >= n_rows) return;
  const size_t row = static_cast<size_t>(b) * n_rows + r;
  const int g = (r % p.H) / (p.H / p.G);
  for (int i = lane; i < p.dk; i += 32) q[i] = to_float(static_cast<const T*>(p.q)[row * p.dk + i]);
  for (int i = lane; i < p.dv; i += 32) o[i] = 0.f;
  __syncwarp();
  const int n_keys = min(p.kv_lens[b], p.kv_lens[b] - p.S + r / p.H + 1);
  const int* table = p.block_table + static_cast<size_t>(b) * p.bt_stride;
  auto slot = [&](int j) { return static_cast<size_t>(table[j / p.page]) * p.page + j % p.page; };
  float m = -INFINITY, l = 0.f;
  for (int j0 = 0; j0 < n_keys; j0 += 32) {
    const int j = j0 + lane;
    const bool in = j < n_keys;
    float s = 0.f;
    if (in) {
      const T* k = static_cast<const T*>(p.k) + (slot(j) * p.G + g) * p.dk;
      for (int i = 0; i < p.dk; i += 4) {
        const float4 x = load4(k + i);
        s = fmaf(x.x, q[i], s); s = fmaf(x.y, q[i + 1], s); s = fmaf(x.z, q[i + 2], s); s = fmaf(x.w, q[i + 3], s);
      }
    }
    s = in ? s * p.scale : -INFINITY;
    const float m_new = fmaxf(m, warp_max(s));
    const float pr = in ? expf(s - m_new) : 0.f;
    const float corr = expf(m - m_new);
    l = l * corr + warp_sum(pr);
    m = m_new;
    const int n = min(32, n_keys - j0);
    for (int i0 = 0; i0 < p.dv; i0 += 32) {  // uniform over the warp: every lane takes part in the shuffles
      const int i = i0 + lane;
      float acc = i < p.dv ? o[i] * corr : 0.f;
      for (int kk = 0; kk < n; ++kk) {
        const float w = __shfl_sync(0xffffffffu, pr, kk);
        if (i < p.dv) acc = fmaf(w, to_float(static_cast<const T*>(p.v)[(slot(j0 + kk) * p.G + g) * p.dv + i]), acc);
      }
      if (i < p.dv) o[i] = acc;
    }
    __syncwarp();
  }
  float inv = l > 0.f ? 1.f / l : 0.f;
  if (p.gate != nullptr) inv /= 1.f + expf(-to_float(static_cast<const T*>(p.gate)[(row / p.H) * p.ldg + r % p.H]));
  for (int i = lane; i < p.dv; i += 32) static_cast<T*>(p.out)[row * p.dv + i] = from_float<T>(o[i] * inv);
}

}  // namespace b200

using namespace b200;

// q, k, v: columns of one GEMM output with row pitch ld. Heads of qk_in / v_in columns come in and leave with qk_out / v_out
// columns (zeros behind). cos_sin fp32 [positions, rot] holds (cos, sin) pairs; gains of the norm may be null. Sizes and ld: multiples of 4.
B200_API int b200_head_norm_rope(const void* q, const void* k, const void* v, int ld, const void* gain_q, const void* gain_k,
                                 const float* cos_sin, const int* positions, const long long* slots, void* q_out, void* k_cache,
                                 void* v_cache, int rows, int H, int G, int D, int rot, int qk_in, int qk_out, int v_in, int v_out, float eps,
                                 float q_scale, int dtype, void* stream) {
  if (rows <= 0) return kOk;
  B200_REQUIRE(H >= 1 && G >= 1 && D >= 1 && qk_in >= D && qk_out >= qk_in && v_out >= v_in && v_in >= 1, "bad head sizes");
  B200_REQUIRE((qk_in | qk_out | v_in | v_out | ld) % 4 == 0, "head sizes and the row pitch must be multiples of 4");
  B200_REQUIRE(rot >= 0 && rot % 2 == 0 && rot <= D, "rotary dimensions (%d) must be even and at most %d", rot, D);
  HeadNormRopeParams p{q, k, v, gain_q, gain_k, cos_sin, positions, slots, q_out, k_cache, v_cache,
                       rows, H, G, D, rot, qk_in, qk_out, v_in, v_out, ld, eps, q_scale};
  const long long blocks = (static_cast<long long>(rows) * (H + 2 * G) + 7) / 8;
  B200_REQUIRE(blocks < (1LL << 31), "head_norm_rope: too many tokens");
  B200_DISPATCH_FLOAT(dtype, B200_CHECK_CUDA(launch_pdl(head_norm_rope_kernel<T>, dim3(static_cast<unsigned>(blocks)), dim3(256), 0,
                                                        static_cast<cudaStream_t>(stream), p));
                      return kOk;);
}

// Causal attention of the last S tokens of every sequence over its paged keys. q [B * S, H, dk], out [B * S, H, dv]; gate nullable.
B200_API int b200_gqa_attention_plain(const void* q, const void* k, const void* v, const int* block_table, int bt_stride,
                                      const int* kv_lens, int B, int S, int H, int G, int dk, int dv, int page, float scale,
                                      const void* gate, int ldg, void* out, int dtype, void* stream) {
  B200_REQUIRE(B >= 1 && S >= 1 && G >= 1 && H % G == 0 && page >= 1 && B <= 65535, "bad attention shape");
  B200_REQUIRE(dk % 4 == 0 && dv % 4 == 0, "head sizes (%d, %d) must be multiples of 4", dk, dv);
  GqaPlainParams p{q, k, v, block_table, kv_lens, gate, out, bt_stride, page, H, G, S, dk, dv, ldg, scale};
  const int smem = 4 * (dk + dv) * 4;
  B200_REQUIRE(smem <= 48 * 1024, "heads of %d / %d do not fit in shared memory", dk, dv);
  const dim3 grid((S * H + 3) / 4, B);
  B200_DISPATCH_FLOAT(dtype, B200_CHECK_CUDA(launch_pdl(gqa_attention_plain_kernel<T>, grid, dim3(128), smem,
                                                        static_cast<cudaStream_t>(stream), p));
                      return kOk;);
}
