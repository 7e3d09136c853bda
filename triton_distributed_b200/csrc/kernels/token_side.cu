// Per-layer token input: act[t, i] = gelu(g[t, i]) * table[id[t], offset + i], with the tanh form of gelu. The table holds one
// vector per token id with a part for every layer; g is the stream's image under a small gate matrix.
#include "b200/elem.cuh"
#include "b200/host.h"

namespace b200 {

template <typename T>
__device__ __forceinline__ float gelu_tanh(float z) {
  return 0.5f * z * (1.f + tanh_t<T>(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

struct TokenSideParams {
  const void* g;           // [T, pitch]
  const long long* ids;    // [T]; an id outside the table reads as zeros
  const void* table;       // [V, ldt]
  void* act;               // [T, pitch]
  long long V;
  int T, dim, pitch, ldt, offset;
};

// Four columns per thread. Rows of the table start anywhere (the parts of the layers need no alignment).
template <typename T>
__global__ void __launch_bounds__(256) token_side_kernel(const TokenSideParams p) {
  const int groups = p.pitch / 4;
  const size_t at = blockIdx.x * static_cast<size_t>(blockDim.x) + threadIdx.x;
  griddep_launch_dependents();
  griddep_wait();
  if (at >= static_cast<size_t>(p.T) * groups) return;
  const size_t t = at / groups;
  const int c = static_cast<int>(at - t * groups) * 4;
  const long long id = p.ids[t];
  const bool ok = id >= 0 && id < p.V;
  const T* e = static_cast<const T*>(p.table) + (ok ? static_cast<size_t>(id) : 0) * p.ldt + p.offset + c;
  const float4 g = load4(static_cast<const T*>(p.g) + t * p.pitch + c);
  const float z[4] = {g.x, g.y, g.z, g.w};
  float o[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) o[i] = ok && c + i < p.dim ? gelu_tanh<T>(z[i]) * to_float(e[i]) : 0.f;
  store4(static_cast<T*>(p.act) + t * p.pitch + c, make_float4(o[0], o[1], o[2], o[3]));
}

}  // namespace b200

using namespace b200;

// act [T, pitch]: columns [0, dim) as above, zeros behind. table [V, ldt] with the layer's part in columns [offset, offset + dim).
B200_API int b200_token_side(const void* g, const long long* ids, const void* table, void* act, int rows, long long V, int dim, int pitch,
                             int ldt, int offset, int dtype, void* stream) {
  if (rows <= 0) return kOk;
  B200_REQUIRE(dim >= 1 && pitch >= dim && pitch % 4 == 0 && offset >= 0 && offset + dim <= ldt, "token_side: bad sizes");
  const TokenSideParams p{g, ids, table, act, V, rows, dim, pitch, ldt, offset};
  const size_t n = static_cast<size_t>(rows) * (pitch / 4);
  B200_DISPATCH_FLOAT(dtype, B200_CHECK_CUDA(launch_pdl(token_side_kernel<T>, dim3(static_cast<unsigned>((n + 255) / 256)), dim3(256), 0,
                                                        static_cast<cudaStream_t>(stream), p));
                      return kOk;);
}
