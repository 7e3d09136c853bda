// The residual stream of decoders that keep it in fp32: embedding, gated sublayer sums, a weighted average over the
// states of all earlier layers ("depth average"), and the norm whose output the next layer's GEMMs read. One CTA per
// token, one pass: everything a layer does between its last GEMM and the next layer's first one is one kernel.
//
//   embed_norm       x = table[id] * scale;  state_0 = x;  h = norm(x)
//   residual_norm    s = x + mult * (sigmoid(ga + ba) * a + sigmoid(gb + bb) * b)     (gates and b optional)
//                    state_n = s;  x = w_0 state_0 + ... + w_{n-1} state_{n-1} + w_n s (with weights; else x = s)
//                    h = norm(x)
//   residual_post    x = x + mult * (rms(a) * gain_a + rms(b) * gain_b);  h = norm(x)  (b optional): sublayers whose results are
//                    RMS-normed on their way into the stream
// norm is layer norm (mean removed, variance = mean of squared deviations), RMS norm or tanh(alpha x), with a gain and an
// optional bias; or a plain copy of x in the storage type. The stream, the states and all arithmetic are fp32; a, b, the gates and h have the model's
// storage type (bf16 / f16 / fp32). Rows are `pitch` wide: columns in [width, pitch) are padding, which carries zeros and
// is left out of the statistics.
//
// Few tokens (decode) do not fill the machine with one CTA each, and a row with many earlier states is a long chain of loads:
// then a cluster of CTAs shares a row, a slice of columns each, and exchanges (count, mean, squared deviations) of the slices
// through distributed shared memory, which merge exactly.
#include "b200/elem.cuh"
#include "b200/host.h"
#include "b200/tcgen05.cuh"

#include <cstring>

namespace b200 {

constexpr int kRnThreads = 512;

enum NormKind : int { kNormRms = 0, kNormLayer = 1, kNormTanh = 2, kNormCopy = 3 };

struct NormParams {
  int width, pitch, kind;
  float eps;          // of the statistics (rms, layer); the factor alpha of kNormTanh
  const void* gain;   // [pitch] (not read by kNormCopy)
  const void* bias;   // [pitch] or null
  void* h;            // [T, pitch]; null: no norm
};

struct ResidualParams {
  const void *a, *b;              // sublayer results [T, pitch]; b nullable
  const void *gate_a, *gate_b;    // gate logits [T, *] with row pitch ldg; null = no gate
  const void *bias_a, *bias_b;    // [pitch] or null
  int ldg;
  float mult;
  float* x;                       // [T, pitch] in / out
  float* states;                  // [*, T, pitch] states 0 .. n_prev - 1 are read; null without weights
  long long state_stride;         // elements between two states
  const float* weights;           // [n_prev + 1] or null
  int n_prev;
  int keep;                       // store the new state at index n_prev
  NormParams norm;
};

struct PostParams {
  const void *a, *b;              // sublayer results [T, pitch]; b nullable
  const void *gain_a, *gain_b;    // [pitch] gains of their RMS norms
  float eps, mult;
  float* x;                       // [T, pitch] in / out
  NormParams norm;
};

struct EmbedParams {
  const long long* ids;
  const void* table;   // [V, pitch]
  long long V;
  float scale;
  float* x;            // [T, pitch]
  float* state0;       // [T, pitch] or null
  NormParams norm;
};

__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  const int nw = blockDim.x >> 5;
  return warp_sum((threadIdx.x & 31) < nw ? red[threadIdx.x & 31] : 0.f);
}

// The slice of a row that a CTA owns: all of it, or one of kCl equal parts (in groups of four columns).
template <int kCl>
struct Slice {
  int begin, end;
  __device__ __forceinline__ explicit Slice(int pitch) {
    const int span = ((pitch / 4 + kCl - 1) / kCl) * 4;
    begin = kCl == 1 ? 0 : static_cast<int>(cluster_ctarank()) * span;
    end = min(pitch, begin + span);
  }
  // group u of this thread: columns [col(u), col(u) + 4)
  __device__ __forceinline__ int col(int u) const { return begin + 4 * (threadIdx.x + u * blockDim.x); }
};

struct RowStats {
  float mean, m2;  // mean, sum of squared deviations from it
};

// statistics of the CTA's slice; RMS norm takes the deviations from zero
template <int U, int kCl>
__device__ __forceinline__ RowStats slice_stats(const NormParams& n, const Slice<kCl>& sl, const float4 (&v)[U], int count, float* red) {
  RowStats st{0.f, 0.f};
  if (n.kind == kNormLayer) {
    float s = 0.f;
#pragma unroll
    for (int u = 0; u < U; ++u) s += (v[u].x + v[u].y) + (v[u].z + v[u].w);  // padding columns are zero
    st.mean = count > 0 ? block_sum(s, red) / count : block_sum(s, red);
  }
  float ss = 0.f;
#pragma unroll
  for (int u = 0; u < U; ++u) {
    const int c = sl.col(u);
    const float d[4] = {v[u].x - st.mean, v[u].y - st.mean, v[u].z - st.mean, v[u].w - st.mean};
#pragma unroll
    for (int e = 0; e < 4; ++e) ss += c + e < min(sl.end, n.width) ? d[e] * d[e] : 0.f;
  }
  st.m2 = block_sum(ss, red);
  return st;
}

template <typename T, int U, int kCl>
__device__ __forceinline__ void norm_row(const NormParams& n, const Slice<kCl>& sl, size_t row, const float4 (&v)[U],
                                         const float4 (&gain)[U], const float4 (&bias)[U], float* red, float4* shared_stats) {
  if (n.h == nullptr) return;  // the same for the whole cluster
  if (n.kind >= kNormTanh) {   // no statistics
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int c = sl.col(u);
      if (c >= sl.end) continue;
      float4 o = v[u];
      if (n.kind == kNormTanh) {
        o.x = tanh_t<T>(n.eps * o.x) * gain[u].x + bias[u].x;
        o.y = tanh_t<T>(n.eps * o.y) * gain[u].y + bias[u].y;
        o.z = tanh_t<T>(n.eps * o.z) * gain[u].z + bias[u].z;
        o.w = tanh_t<T>(n.eps * o.w) * gain[u].w + bias[u].w;
      }
      store4(static_cast<T*>(n.h) + row * n.pitch + c, o);
    }
    return;
  }
  const int count = max(0, min(sl.end, n.width) - sl.begin);
  RowStats st = slice_stats<U, kCl>(n, sl, v, count, red);
  if (kCl > 1) {
    const uint32_t me = cluster_ctarank();
    if (threadIdx.x < kCl) {
      const uint32_t dst = mapa_u32(shared_stats + me, threadIdx.x);
      asm volatile("st.shared::cluster.v4.f32 [%0], {%1, %2, %3, %4};" ::"r"(dst), "f"(static_cast<float>(count)), "f"(st.mean),
                   "f"(st.m2), "f"(0.f)
                   : "memory");
    }
    cluster_sync_all();
    float total = 0.f;
#pragma unroll
    for (int i = 0; i < kCl; ++i) total += shared_stats[i].x * shared_stats[i].y;
    const float mean = total / n.width;
    float m2 = 0.f;
#pragma unroll
    for (int i = 0; i < kCl; ++i) {
      const float d = shared_stats[i].y - mean;
      m2 += shared_stats[i].z + shared_stats[i].x * d * d;
    }
    st = RowStats{mean, m2};
  }
  const float inv = 1.f / sqrtf(st.m2 / n.width + n.eps);
#pragma unroll
  for (int u = 0; u < U; ++u) {
    const int c = sl.col(u);
    if (c < sl.end) {
      float4 o;
      o.x = (v[u].x - st.mean) * inv * gain[u].x + bias[u].x;
      o.y = (v[u].y - st.mean) * inv * gain[u].y + bias[u].y;
      o.z = (v[u].z - st.mean) * inv * gain[u].z + bias[u].z;
      o.w = (v[u].w - st.mean) * inv * gain[u].w + bias[u].w;
      store4(static_cast<T*>(n.h) + row * n.pitch + c, o);
    }
  }
}

// the gain and bias are weights: read before the dependency wait
template <typename T, int U, int kCl>
__device__ __forceinline__ void load_norm_weights(const NormParams& n, const Slice<kCl>& sl, float4 (&gain)[U], float4 (&bias)[U]) {
#pragma unroll
  for (int u = 0; u < U; ++u) {
    const int c = sl.col(u);
    gain[u] = bias[u] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (n.gain != nullptr && c < sl.end) {
      gain[u] = load4(static_cast<const T*>(n.gain) + c);
      if (n.bias != nullptr) bias[u] = load4(static_cast<const T*>(n.bias) + c);
    }
  }
}

template <typename T, int U, int kCl>
__global__ void __launch_bounds__(kRnThreads) embed_norm_kernel(const EmbedParams p) {
  __shared__ float red[32];
  __shared__ float4 stats[kCl];
  const size_t t = blockIdx.x / kCl;
  const int pitch = p.norm.pitch;
  const Slice<kCl> sl(pitch);
  griddep_launch_dependents();
  float4 gain[U], bias[U], v[U];
  load_norm_weights<T, U, kCl>(p.norm, sl, gain, bias);
  if (kCl > 1) cluster_sync_all();  // every CTA of the cluster runs before any writes to another's shared memory
  griddep_wait();
  const long long id = p.ids[t];
  const bool ok = id >= 0 && id < p.V;   // an id outside the table reads as a zero row
#pragma unroll
  for (int u = 0; u < U; ++u) {
    const int c = sl.col(u);
    v[u] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < sl.end) {
      if (ok) v[u] = load4(static_cast<const T*>(p.table) + static_cast<size_t>(id) * pitch + c);
      v[u].x *= p.scale; v[u].y *= p.scale; v[u].z *= p.scale; v[u].w *= p.scale;
      store4(p.x + t * pitch + c, v[u]);
      if (p.state0 != nullptr) store4(p.state0 + t * pitch + c, v[u]);
    }
  }
  norm_row<T, U, kCl>(p.norm, sl, t, v, gain, bias, red, stats);
}

__device__ __forceinline__ float sigmoid(float z) { return 1.f / (1.f + expf(-z)); }

template <typename T>
__device__ __forceinline__ float4 gated(const void* val, const void* gate, const void* bias, size_t row, int pitch, int ldg, int c) {
  float4 a = load4(static_cast<const T*>(val) + row * pitch + c);
  if (gate != nullptr) {
    float4 z = load4(static_cast<const T*>(gate) + row * ldg + c);
    if (bias != nullptr) {
      const float4 b = load4(static_cast<const T*>(bias) + c);
      z.x += b.x; z.y += b.y; z.z += b.z; z.w += b.w;
    }
    a.x *= sigmoid(z.x); a.y *= sigmoid(z.y); a.z *= sigmoid(z.z); a.w *= sigmoid(z.w);
  }
  return a;
}

template <typename T, int U, int kCl>
__global__ void __launch_bounds__(kRnThreads) residual_norm_kernel(const ResidualParams p) {
  __shared__ float red[32];
  __shared__ float4 stats[kCl];
  const size_t t = blockIdx.x / kCl;
  const int pitch = p.norm.pitch;
  const Slice<kCl> sl(pitch);
  griddep_launch_dependents();
  float4 gain[U], bias[U], x[U];
  load_norm_weights<T, U, kCl>(p.norm, sl, gain, bias);
  if (kCl > 1) cluster_sync_all();  // every CTA of the cluster runs before any writes to another's shared memory
  griddep_wait();
#pragma unroll
  for (int u = 0; u < U; ++u) {
    const int c = sl.col(u);
    x[u] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c >= sl.end) continue;
    const size_t at = t * pitch + c;
    // the average over the earlier states first: its loads do not depend on anything else of the row
    float4 avg = make_float4(0.f, 0.f, 0.f, 0.f);
    float wn = 1.f;
    if (p.weights != nullptr) {
      const float* st = p.states + at;
      wn = __ldg(p.weights + p.n_prev);
#pragma unroll 8
      for (int j = 0; j < p.n_prev; ++j) {
        const float w = __ldg(p.weights + j);
        const float4 o = load4(st + j * p.state_stride);
        avg.x = fmaf(w, o.x, avg.x); avg.y = fmaf(w, o.y, avg.y); avg.z = fmaf(w, o.z, avg.z); avg.w = fmaf(w, o.w, avg.w);
      }
    }
    float4 r = load4(p.x + at);
    float4 s = gated<T>(p.a, p.gate_a, p.bias_a, t, pitch, p.ldg, c);
    if (p.b != nullptr) {
      const float4 b = gated<T>(p.b, p.gate_b, p.bias_b, t, pitch, p.ldg, c);
      s.x += b.x; s.y += b.y; s.z += b.z; s.w += b.w;
    }
    r.x = fmaf(p.mult, s.x, r.x); r.y = fmaf(p.mult, s.y, r.y); r.z = fmaf(p.mult, s.z, r.z); r.w = fmaf(p.mult, s.w, r.w);
    if (p.weights != nullptr) {
      if (p.keep) store4(p.states + p.n_prev * p.state_stride + at, r);
      r.x = fmaf(wn, r.x, avg.x); r.y = fmaf(wn, r.y, avg.y); r.z = fmaf(wn, r.z, avg.z); r.w = fmaf(wn, r.w, avg.w);
    }
    x[u] = r;
    store4(p.x + at, r);
  }
  norm_row<T, U, kCl>(p.norm, sl, t, x, gain, bias, red, stats);
}

// sums over the row of the squares of `v` and `w`, for the whole cluster
template <int U, int kCl>
__device__ __forceinline__ float2 row_squares(const float4 (&v)[U], const float4 (&w)[U], float2* red, float2* shared_sums) {
  float2 s = make_float2(0.f, 0.f);
#pragma unroll
  for (int u = 0; u < U; ++u) {  // padding columns are zero
    s.x += (v[u].x * v[u].x + v[u].y * v[u].y) + (v[u].z * v[u].z + v[u].w * v[u].w);
    s.y += (w[u].x * w[u].x + w[u].y * w[u].y) + (w[u].z * w[u].z + w[u].w * w[u].w);
  }
  s = make_float2(warp_sum(s.x), warp_sum(s.y));
  const int lane = threadIdx.x & 31;
  if (lane == 0) red[threadIdx.x >> 5] = s;
  __syncthreads();
  s = lane < static_cast<int>(blockDim.x >> 5) ? red[lane] : make_float2(0.f, 0.f);
  s = make_float2(warp_sum(s.x), warp_sum(s.y));
  if (kCl > 1) {
    const uint32_t me = cluster_ctarank();
    if (threadIdx.x < kCl) {
      const uint32_t dst = mapa_u32(shared_sums + me, threadIdx.x);
      asm volatile("st.shared::cluster.v2.f32 [%0], {%1, %2};" ::"r"(dst), "f"(s.x), "f"(s.y) : "memory");
    }
    cluster_sync_all();
    s = make_float2(0.f, 0.f);
#pragma unroll
    for (int i = 0; i < kCl; ++i) {
      s.x += shared_sums[i].x;
      s.y += shared_sums[i].y;
    }
  }
  return s;
}

template <typename T, int U, int kCl>
__global__ void __launch_bounds__(kRnThreads) residual_post_kernel(const PostParams p) {
  __shared__ float red[32];
  __shared__ float4 stats[kCl];
  __shared__ float2 sums[kCl], red2[32];
  const size_t t = blockIdx.x / kCl;
  const int pitch = p.norm.pitch;
  const Slice<kCl> sl(pitch);
  griddep_launch_dependents();
  float4 gain[U], bias[U], a[U], b[U], x[U];
  load_norm_weights<T, U, kCl>(p.norm, sl, gain, bias);
  if (kCl > 1) cluster_sync_all();  // every CTA of the cluster runs before any writes to another's shared memory
  griddep_wait();
#pragma unroll
  for (int u = 0; u < U; ++u) {
    const int c = sl.col(u);
    a[u] = b[u] = x[u] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c >= sl.end) continue;
    x[u] = load4(p.x + t * pitch + c);
    a[u] = load4(static_cast<const T*>(p.a) + t * pitch + c);
    if (p.b != nullptr) b[u] = load4(static_cast<const T*>(p.b) + t * pitch + c);
  }
  const float2 ss = row_squares<U, kCl>(a, b, red2, sums);
  const float ia = p.mult / sqrtf(ss.x / p.norm.width + p.eps), ib = p.mult / sqrtf(ss.y / p.norm.width + p.eps);
#pragma unroll
  for (int u = 0; u < U; ++u) {
    const int c = sl.col(u);
    if (c >= sl.end) continue;
    const float4 ga = load4(static_cast<const T*>(p.gain_a) + c);
    x[u].x = fmaf(a[u].x * ia, ga.x, x[u].x); x[u].y = fmaf(a[u].y * ia, ga.y, x[u].y);
    x[u].z = fmaf(a[u].z * ia, ga.z, x[u].z); x[u].w = fmaf(a[u].w * ia, ga.w, x[u].w);
    if (p.b != nullptr) {
      const float4 gb = load4(static_cast<const T*>(p.gain_b) + c);
      x[u].x = fmaf(b[u].x * ib, gb.x, x[u].x); x[u].y = fmaf(b[u].y * ib, gb.y, x[u].y);
      x[u].z = fmaf(b[u].z * ib, gb.z, x[u].z); x[u].w = fmaf(b[u].w * ib, gb.w, x[u].w);
    }
    store4(p.x + t * pitch + c, x[u]);
  }
  norm_row<T, U, kCl>(p.norm, sl, t, x, gain, bias, red, stats);
}

static int check_norm(const NormParams& n) {
  B200_REQUIRE(n.width > 0 && n.pitch % 4 == 0 && n.pitch >= n.width, "row pitch (%d) must be a multiple of 4 and >= width (%d)",
               n.pitch, n.width);
  B200_REQUIRE(n.pitch <= 4 * 8 * kRnThreads, "width (%d) is limited to %d", n.width, 4 * 8 * kRnThreads);
  B200_REQUIRE(n.kind >= kNormRms && n.kind <= kNormCopy, "unknown norm kind %d", n.kind);
  B200_REQUIRE((n.gain == nullptr || n.h != nullptr) && (n.h == nullptr || n.kind == kNormCopy || n.gain != nullptr),
               "the norm needs a gain and an output");
  return kOk;
}
// groups of four columns per thread, from the kernels' instantiations, and the threads that then cover a row
static int row_groups(int pitch) {
  const int g = (pitch / 4 + kRnThreads - 1) / kRnThreads;
  return g <= 4 ? g : 8;
}
static int row_threads(int pitch) {
  const int g = row_groups(pitch);
  return ((pitch / 4 + g - 1) / g + 31) / 32 * 32;
}

template <typename P>
static int launch_cluster(void (*kernel)(P), const P& p, int rows, int cl, int threads, cudaStream_t s) {
  cudaLaunchConfig_t cfg;
  memset(&cfg, 0, sizeof(cfg));
  cfg.gridDim = dim3(rows * cl);
  cfg.blockDim = dim3(threads);
  cfg.stream = s;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = cl;
  attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = pdl_enabled() ? 2 : 1;
  B200_CHECK_CUDA(cudaLaunchKernelEx(&cfg, kernel, p));
  return kOk;
}

// CTAs that share a row: several when the rows alone leave most of the machine idle
static int row_cluster(int rows, int pitch) {
  if (pitch < 1024) return 1;
  if (rows * 8 <= sm_count() && pitch >= 2048) return 8;
  return rows * 4 <= sm_count() ? 4 : 1;
}

template <typename P>
using RowKernel = void (*)(P);

// `k`: kernels for 1, 2, 3, 4 and 8 groups per thread; `k4`, `k8`: one group per thread in clusters of 4 and 8
template <typename P>
static int launch_rows(const RowKernel<P> (&k)[5], RowKernel<P> k4, RowKernel<P> k8, const P& p, int rows, cudaStream_t s) {
  const int pitch = p.norm.pitch, cl = row_cluster(rows, pitch);
  if (cl > 1) {
    const int groups = (pitch / 4 + cl - 1) / cl;
    if (groups <= kRnThreads) return launch_cluster(cl == 8 ? k8 : k4, p, rows, cl, (groups + 31) / 32 * 32, s);
  }
  const int g = row_groups(pitch);
  B200_CHECK_CUDA(launch_pdl(k[g == 8 ? 4 : g - 1], dim3(rows), dim3(row_threads(pitch)), 0, s, p));
  return kOk;
}

#define B200_ROW_KERNELS(K, P)                                                                                   \
  const RowKernel<P> k[5] = {K<T, 1, 1>, K<T, 2, 1>, K<T, 3, 1>, K<T, 4, 1>, K<T, 8, 1>};                          \
  return launch_rows<P>(k, K<T, 1, 4>, K<T, 1, 8>, p, rows, static_cast<cudaStream_t>(stream))

}  // namespace b200

using namespace b200;

B200_API int b200_embed_norm(const long long* ids, const void* table, int rows, long long V, int width, int pitch, float scale,
                             float* x, float* state0, const void* gain, const void* bias, float eps, int kind, void* h,
                             int dtype, void* stream) {
  if (rows <= 0) return kOk;
  EmbedParams p;
  memset(&p, 0, sizeof(p));
  p.ids = ids; p.table = table; p.V = V; p.scale = scale; p.x = x; p.state0 = state0;
  p.norm = NormParams{width, pitch, kind, eps, gain, bias, h};
  int rc = check_norm(p.norm);
  if (rc != kOk) return rc;
  B200_DISPATCH_FLOAT(dtype, B200_ROW_KERNELS(embed_norm_kernel, EmbedParams););
}

// `states` holds n_prev earlier states of [rows, pitch] each, state_stride elements apart; with keep != 0 the new state
// is stored behind them. weights [n_prev + 1] fp32 on the device, null = no depth average.
B200_API int b200_residual_norm(const void* a, const void* gate_a, const void* bias_a, const void* b, const void* gate_b,
                                const void* bias_b, int ldg, float mult, float* x, float* states, long long state_stride,
                                const float* weights, int n_prev, int keep, int rows, int width, int pitch, const void* gain,
                                const void* bias, float eps, int kind, void* h, int dtype, void* stream) {
  if (rows <= 0) return kOk;
  B200_REQUIRE(a != nullptr && x != nullptr, "residual_norm needs a sublayer result and the stream");
  B200_REQUIRE(weights == nullptr || (states != nullptr && n_prev >= 1), "the depth average needs the earlier states");
  B200_REQUIRE(ldg % 4 == 0, "the gates' row pitch (%d) must be a multiple of 4", ldg);
  ResidualParams p;
  memset(&p, 0, sizeof(p));
  p.a = a; p.b = b; p.gate_a = gate_a; p.gate_b = gate_b; p.bias_a = bias_a; p.bias_b = bias_b; p.ldg = ldg; p.mult = mult;
  p.x = x; p.states = states; p.state_stride = state_stride; p.weights = weights; p.n_prev = n_prev; p.keep = keep;
  p.norm = NormParams{width, pitch, kind, eps, gain, bias, h};
  int rc = check_norm(p.norm);
  if (rc != kOk) return rc;
  B200_DISPATCH_FLOAT(dtype, B200_ROW_KERNELS(residual_norm_kernel, ResidualParams););
}

// x += mult * (rms(a) * gain_a + rms(b) * gain_b) over rows of `width` (b, gain_b nullable), then the norm as above.
B200_API int b200_residual_post(const void* a, const void* gain_a, const void* b, const void* gain_b, float post_eps, float mult,
                                float* x, int rows, int width, int pitch, const void* gain, const void* bias, float eps, int kind,
                                void* h, int dtype, void* stream) {
  if (rows <= 0) return kOk;
  B200_REQUIRE(a != nullptr && gain_a != nullptr && x != nullptr && (b == nullptr) == (gain_b == nullptr),
               "residual_post needs sublayer results with their gains, and the stream");
  PostParams p;
  memset(&p, 0, sizeof(p));
  p.a = a; p.b = b; p.gain_a = gain_a; p.gain_b = gain_b; p.eps = post_eps; p.mult = mult; p.x = x;
  p.norm = NormParams{width, pitch, kind, eps, gain, bias, h};
  int rc = check_norm(p.norm);
  if (rc != kOk) return rc;
  B200_DISPATCH_FLOAT(dtype, B200_ROW_KERNELS(residual_post_kernel, PostParams););
}
