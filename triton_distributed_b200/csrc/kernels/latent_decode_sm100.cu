// Absorbed latent attention for sm_100a on the tensor cores: one cached row per token is key and value of all heads.
//
// The roles of the operands are swapped so that the few query rows (query token x head, N of them) are the narrow side of
// every tcgen05.mma and no tensor-core row is padding:
//   scores   S^T [64 keys, N]   = C [64 keys, rank] . Q [N, rank]^T         (C and Q K-major)
//   values   O^T [rank, N]     += C^T [rank, 64 keys] . P [N, 64 keys]^T   (C^T is the same shared-memory tile read MN-major)
// so a latent row is loaded once and used twice, and the running output stays in tensor memory: lane = column of the latent
// (in chunks of 128), column = query row.
//
// One CTA owns N query rows of a sequence and a range of 64-key tiles (split-KV; latent_combine merges, and adds the sink):
//   warp 0     TMA producer: the Q tile once, then the tiles in slots of 64 keys x 128 columns (two 64-column swizzle atoms)
//   warp 1     MMA issuer: the scores of tile j + 1 are computed while tile j is in the softmax (two score buffers, two P
//              tiles); a slot is given back as soon as its chunk of the output has been accumulated
//   warps 4-11 softmax, half of the query rows each: exponentials against a reference maximum per row, P as 16-bit into a
//              swizzled tile. The scores are read in the 16-lane x 256-bit shape (a 64-row accumulator occupies 16 lanes of every
//              quarter), whose fragments stmatrix writes transposed, eight keys of a row at a time. The reference only moves when a score exceeds it by more than
//              2^8: one vote per tile decides, and only then are the maxima reduced over the keys and the sums and the output in
//              tensor memory rescaled. Sums and output share the reference, which cancels in the end.
// The producer also asks L2 for tiles beyond the ring, so that a slot that becomes free is refilled at L2 latency.
// Every barrier wait is bounded; on expiry the CTA unwinds through an abort flag and reports a status.
#include "b200/host.h"
#include "b200/primitives.cuh"
#include "b200/tcgen05.cuh"

#include <cstring>

namespace b200 {

constexpr int kLdKeys = 64;               // keys per tile
constexpr int kLdAtom = kLdKeys * 128;    // 64 keys x 64 columns: 8 KB
constexpr int kLdSlot = 2 * kLdAtom;      // 64 keys x 128 columns
constexpr int kLdThreads = 384;
constexpr float kLdSlack = 8.f;           // how far (log2) a score may exceed the reference before it moves
constexpr int kLdSmemMax = 226 * 1024;

constexpr int ld_fixed_bytes(int n, int rk) { return (rk / 64 + 2) * n * 128 + 1024 + 512 + n * 44; }
constexpr int ld_slots(int n, int rk) {
  const int fit = (kLdSmemMax - ld_fixed_bytes(n, rk)) / kLdSlot, want = 4 * (rk / 128) + 2 < 16 ? 4 * (rk / 128) + 2 : 16;
  return fit < want ? fit : want;
}
constexpr int ld_smem_bytes(int n, int rk) { return ld_fixed_bytes(n, rk) + ld_slots(n, rk) * kLdSlot; }

struct LatentDecodeParams {
  const int* block_table;  // [B, bt_stride]
  const int* kv_lens;      // [B]
  float* o_part;           // [B * S * H, splits, pitch]
  float* lse_part;         // [B * S * H, splits]
  int bt_stride, page, H, S, pitch, splits, bf16;
  float scale_log2e;       // positive
  uint32_t* status;
};

// MN-major operand in 128-byte-swizzled atoms of 64 (MN) x 8 (K): 8-row K groups 1024 bytes apart, the next 64 MN elements
// `mn_stride` bytes away
__device__ __forceinline__ uint64_t umma_desc_sw128_mnmajor(uint32_t smem_addr, uint32_t mn_stride) {
  uint64_t d = umma_desc_sw128_kmajor(smem_addr);
  d &= ~(static_cast<uint64_t>(0x3FFF) << 16);
  d |= static_cast<uint64_t>(mn_stride >> 4) << 16;
  return d;
}
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void tmem_st_32x8(uint32_t taddr, const uint32_t (&r)[8]) {
  asm volatile("tcgen05.st.sync.aligned.32x32b.x8.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8};" ::"r"(taddr), "r"(r[0]), "r"(r[1]),
               "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7])
               : "memory");
}
__device__ __forceinline__ void tmem_st_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }
// barrier of the 256 softmax threads, and the same with a vote
__device__ __forceinline__ void ld_softmax_bar() { asm volatile("bar.sync 1, 256;" ::: "memory"); }
__device__ __forceinline__ bool ld_softmax_any(bool v) {
  uint32_t r;
  asm volatile(
      "{\n"
      ".reg .pred P, Q;\n"
      "setp.ne.u32 P, %1, 0;\n"
      "barrier.cta.red.or.pred Q, 2, 256, P;\n"
      "selp.u32 %0, 1, 0, Q;\n"
      "}\n"
      : "=r"(r)
      : "r"(v ? 1u : 0u)
      : "memory");
  return r != 0;
}
// reads kCols (8, 16 or 32) consecutive columns of this thread's lane
template <int kCols>
__device__ __forceinline__ void tmem_ld_cols(uint32_t taddr, float (&v)[kCols]) {
  uint32_t r[kCols];
  if constexpr (kCols == 8) tmem_ld_32x8(taddr, r);
  else if constexpr (kCols == 16) tmem_ld_32x16(taddr, r);
  else tmem_ld_32x32(taddr, r);
  tmem_ld_wait();
#pragma unroll
  for (int i = 0; i < kCols; ++i) v[i] = __uint_as_float(r[i]);
}
// 16 lanes x 8 columns per group of four registers, as an m16n8 fragment: registers 0, 1 hold lane (thread / 4), columns
// 2 (thread % 4) and the next; registers 2, 3 the same columns of lane (thread / 4) + 8
template <int kGroups>
__device__ __forceinline__ void tmem_ld_frag(uint32_t taddr, float (&v)[4 * kGroups]) {
  uint32_t r[4 * kGroups];
  if constexpr (kGroups == 1)
    asm volatile("tcgen05.ld.sync.aligned.16x256b.x1.b32 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(taddr) : "memory");
  else if constexpr (kGroups == 2)
    asm volatile("tcgen05.ld.sync.aligned.16x256b.x2.b32 {%0, %1, %2, %3, %4, %5, %6, %7}, [%8];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7])
                 : "r"(taddr) : "memory");
  else
    asm volatile("tcgen05.ld.sync.aligned.16x256b.x4.b32 {%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15}, [%16];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]),
                   "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
                 : "r"(taddr) : "memory");
  tmem_ld_wait();
#pragma unroll
  for (int i = 0; i < 4 * kGroups; ++i) v[i] = __uint_as_float(r[i]);
}
// 8 x 8 fragments stored transposed; lanes 8 m ... 8 m + 7 address the rows of matrix m
__device__ __forceinline__ void stmatrix_x2_trans(uint32_t addr, uint32_t r0, uint32_t r1) {
  asm volatile("stmatrix.sync.aligned.m8n8.x2.trans.shared.b16 [%0], {%1, %2};" ::"r"(addr), "r"(r0), "r"(r1) : "memory");
}
__device__ __forceinline__ void stmatrix_x4_trans(uint32_t addr, uint32_t r0, uint32_t r1, uint32_t r2, uint32_t r3) {
  asm volatile("stmatrix.sync.aligned.m8n8.x4.trans.shared.b16 [%0], {%1, %2, %3, %4};" ::"r"(addr), "r"(r0), "r"(r1), "r"(r2), "r"(r3)
               : "memory");
}
__device__ __forceinline__ void tma_prefetch_l2_2d(const CUtensorMap* map, int x, int y) {
  asm volatile("cp.async.bulk.prefetch.tensor.2d.L2.global [%0, {%1, %2}];" ::"l"(map), "r"(x), "r"(y) : "memory");
}

// N: query rows per CTA (16, 32 or 64); RK: rank rounded up to a multiple of 128 (TMA fills the padding columns with zeros)
template <int N, int RK>
__global__ void __launch_bounds__(kLdThreads, 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap tmC, const __grid_constant__ CUtensorMap tmQ, const LatentDecodeParams p) {
  constexpr int kPairs = RK / 128, kSlots = ld_slots(N, RK), kRowAtom = N * 128;
  static_assert(kSlots >= 2 * kPairs && kSlots <= 16, "two tiles must fit in the ring, the ring in the barrier layout");
  constexpr uint32_t kTmemNeed = N * (2 + kPairs);
  constexpr uint32_t kTmemCols = kTmemNeed <= 32 ? 32 : kTmemNeed <= 64 ? 64 : kTmemNeed <= 128 ? 128 : kTmemNeed <= 256 ? 256 : 512;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* ring = smem;                             // [kSlots][2 atoms][64 keys][128 B]
  uint8_t* sQ = ring + kSlots * kLdSlot;            // [RK / 64 atoms][N rows][128 B]
  uint8_t* sP = sQ + (RK / 64) * kRowAtom;          // [2 tile parities][N rows][128 B], columns = keys
  uint64_t* bars = reinterpret_cast<uint64_t*>(sP + 2 * kRowAtom);
  uint64_t* full = bars;                // [kSlots]
  uint64_t* empty = bars + 16;          // [kSlots]
  uint64_t* q_full = bars + 32;
  uint64_t* s_full = bars + 33;         // [2] by tile parity
  uint64_t* p_full = bars + 35;         // [2]
  uint64_t* o_done = bars + 37;         // one phase per tile: its values have been accumulated
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 38);
  volatile uint32_t* abort_flag = tmem_slot + 1;
  float* xmax = reinterpret_cast<float*>(reinterpret_cast<uint8_t*>(bars) + 512);  // [4 warps][N]
  float* mref = xmax + 4 * N;                                                      // [N]
  float* corr = mref + N;                                                          // [N]; at the end 1 / row sum
  float* xsum = corr + N;                                                          // [4][N]
  int* limit = reinterpret_cast<int*>(xsum + 4 * N);                               // [N] last key a row attends

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int split = blockIdx.x, r0 = blockIdx.y * N, b = blockIdx.z;
  const int n_rows = p.S * p.H;
  const uint64_t timeout_ns = 4000000000ull;
  griddep_launch_dependents();
  if (threadIdx.x == 0) {
    for (int i = 0; i < kSlots; ++i) {
      mbar_init(full + i, 1);
      mbar_init(empty + i, 1);
    }
    mbar_init(q_full, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(s_full + i, 1);
      mbar_init(p_full + i, 8);
    }
    mbar_init(o_done, 1);
    *abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tmC);
    tma_prefetch_desc(&tmQ);
  }
  if (warp == 2) tmem_alloc(tmem_slot, kTmemCols);
  griddep_wait();
  const int kv_len = p.kv_lens[b];
  const int first_limit = kv_len - p.S;  // last key of token 0; token i adds i
  const int n_keys = max(0, min(kv_len, first_limit + (min(r0 + N, n_rows) - 1) / p.H + 1));
  const int n_tiles = (n_keys + kLdKeys - 1) / kLdKeys;
  const int per = (n_tiles + p.splits - 1) / p.splits;
  const int tile0 = min(n_tiles, split * per), tile1 = min(n_tiles, tile0 + per);
  const int row_base = b * n_rows + r0;
  for (int n = threadIdx.x; n < N; n += kLdThreads) {
    limit[n] = r0 + n < n_rows ? first_limit + (r0 + n) / p.H : -1;
    mref[n] = -INFINITY;
    corr[n] = 1.f;
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem_base = *tmem_slot;  // 2 x N columns of S^T, then kPairs x N columns of O^T

  if (warp == 0) {
    if (elect_one() && tile0 < tile1) {
      fence_proxy_async();  // queries and latents were written by earlier kernels through the generic proxy
      mbar_expect_tx(q_full, (RK / 64) * kRowAtom);
      for (int a = 0; a < RK / 64; ++a) tma_load_2d(sQ + a * kRowAtom, &tmQ, q_full, a * 64, row_base);
      const int* table = p.block_table + static_cast<size_t>(b) * p.bt_stride;
      auto slot_row = [&](int tile) { return table[tile * kLdKeys / p.page] * p.page + tile * kLdKeys % p.page; };
      auto prefetch = [&](int tile) {
        if (tile >= tile1) return;
        const int row = slot_row(tile);
        for (int a = 0; a < RK / 64; ++a)
          if (a * 64 < p.pitch) tma_prefetch_l2_2d(&tmC, a * 64, row);
      };
      int it = 0;
      bool ok = true;
      prefetch(tile0 + 2);
      for (int tile = tile0; tile < tile1 && ok; ++tile) {
        const int row = slot_row(tile);
        prefetch(tile + 3);
        for (int pr = 0; pr < kPairs && ok; ++pr, ++it) {
          const int slot = it % kSlots;
          ok = mbar_wait(empty + slot, ((it / kSlots) & 1) ^ 1, abort_flag, timeout_ns);
          if (!ok) break;
          mbar_expect_tx(full + slot, kLdSlot);
#pragma unroll
          for (int a = 0; a < 2; ++a)
            tma_load_2d(ring + slot * kLdSlot + a * kLdAtom, &tmC, full + slot, pr * 128 + a * 64, row);
        }
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    if (elect_one() && tile0 < tile1) {
      const uint32_t idesc_s = umma_idesc_f16(kLdKeys, N, p.bf16 != 0);
      const uint32_t idesc_o = umma_idesc_f16(128, N, p.bf16 != 0) | (1u << 15);  // A is MN-major
      bool ok = mbar_wait(q_full, 0, abort_flag, timeout_ns);
      const int n = tile1 - tile0;
      auto issue_scores = [&](int j) -> bool {  // tile j of this CTA
        for (int pr = 0; pr < kPairs; ++pr) {
          const int it = j * kPairs + pr, slot = it % kSlots;
          if (!mbar_wait(full + slot, (it / kSlots) & 1, abort_flag, timeout_ns)) return false;
          tc_fence_after_sync();
#pragma unroll
          for (int kk = 0; kk < 8; ++kk) {
            const uint64_t da = umma_desc_sw128_kmajor(smem_u32(ring + slot * kLdSlot + (kk >> 2) * kLdAtom)) + 2 * (kk & 3);
            const uint64_t db = umma_desc_sw128_kmajor(smem_u32(sQ + (2 * pr + (kk >> 2)) * kRowAtom)) + 2 * (kk & 3);
            umma_f16(tmem_base + (j & 1) * N, da, db, idesc_s, (pr | kk) != 0 ? 1u : 0u);
          }
        }
        umma_commit(s_full + (j & 1));  // also: the values of tile j - 2 have been accumulated
        return true;
      };
      if (ok) ok = issue_scores(0);
      for (int j = 0; j < n && ok; ++j) {
        if (j + 1 < n) ok = issue_scores(j + 1);
        if (!ok) break;
        ok = mbar_wait(p_full + (j & 1), (j >> 1) & 1, abort_flag, timeout_ns);
        if (!ok) break;
        tc_fence_after_sync();
        for (int pr = 0; pr < kPairs; ++pr) {
          const int slot = (j * kPairs + pr) % kSlots;
#pragma unroll
          for (int kk = 0; kk < kLdKeys / 16; ++kk) {
            const uint64_t da = umma_desc_sw128_mnmajor(smem_u32(ring + slot * kLdSlot + kk * 16 * 128), kLdAtom);
            const uint64_t db = umma_desc_sw128_kmajor(smem_u32(sP + (j & 1) * kRowAtom)) + 2 * kk;
            umma_f16(tmem_base + N * (2 + pr), da, db, idesc_o, (j | kk) != 0 ? 1u : 0u);
          }
          umma_commit(empty + slot);
        }
        umma_commit(o_done);
      }
    }
    __syncwarp();
  } else if (warp >= 4) {
    constexpr int kCols = N / 2, kGroups = kCols / 8;  // query rows of this warp, in groups of eight
    const int w4 = warp & 3, half = (warp - 4) >> 2;
    // a 64-row accumulator keeps keys 16 q ... 16 q + 15 in the first 16 lanes of quarter q: this thread has keys kt and kt + 8
    // of the tile and query rows n0 + 8 g + 2 (lane % 4) + {0, 1} for every group g
    const int kt = w4 * 16 + (lane >> 2);
    const int n0 = half * kCols, nq = n0 + 2 * (lane & 3);
    const uint32_t lane_base = tmem_base + (static_cast<uint32_t>(w4 * 32) << 16) + n0;
    float l[2 * kGroups];  // share of these keys in the row sums
#pragma unroll
    for (int i = 0; i < 2 * kGroups; ++i) l[i] = 0.f;
    const int all_below = r0 + N <= n_rows ? first_limit + r0 / p.H : -1;  // keys up to here are visible to all rows
    // row of this lane's matrix for stmatrix: matrices alternate between the key blocks (8 keys) and go on to the next group
    const int p_chunk = w4 * 2 + ((lane >> 3) & 1), p_row = n0 + 8 * (lane >> 4) + (lane & 7);
    const uint32_t p_addr = smem_u32(sP + p_row * 128 + ((p_chunk ^ (lane & 7)) << 4));
    const int n_mine = tile1 - tile0;
    bool ok = true;
    // every thread meets the barriers of every tile, also after a pipeline wait has failed
    for (int j = 0; j < n_mine; ++j) {
      if (ok) ok = mbar_wait(s_full + (j & 1), (j >> 1) & 1, abort_flag, timeout_ns);
      ok = __all_sync(0xffffffffu, ok);
      tc_fence_after_sync();
      const int key0 = (tile0 + j) * kLdKeys;
      const bool masked = key0 + kLdKeys - 1 > all_below;
      float s[4 * kGroups];  // [group][key block][row of the pair]
      bool exceeds = false;
      if (ok) {
        tmem_ld_frag<kGroups>(lane_base + (j & 1) * N, s);
#pragma unroll
        for (int g = 0; g < kGroups; ++g) {
          const float2 m = *reinterpret_cast<const float2*>(mref + nq + 8 * g);
#pragma unroll
          for (int e = 0; e < 4; ++e) s[4 * g + e] *= p.scale_log2e;
          if (masked) {
            const int2 lim = *reinterpret_cast<const int2*>(limit + nq + 8 * g);
            const int key = key0 + kt;
            s[4 * g] = key <= lim.x ? s[4 * g] : -INFINITY;
            s[4 * g + 1] = key <= lim.y ? s[4 * g + 1] : -INFINITY;
            s[4 * g + 2] = key + 8 <= lim.x ? s[4 * g + 2] : -INFINITY;
            s[4 * g + 3] = key + 8 <= lim.y ? s[4 * g + 3] : -INFINITY;
          }
          // (always when a row has no reference yet and sees a key)
          exceeds |= fmaxf(s[4 * g], s[4 * g + 2]) > m.x + kLdSlack || fmaxf(s[4 * g + 1], s[4 * g + 3]) > m.y + kLdSlack;
        }
      }
      if (ld_softmax_any(exceeds)) {
        if (ok) {
#pragma unroll
          for (int i = 0; i < 2 * kGroups; ++i) {
            const int g = i >> 1, e = i & 1;
            float m = fmaxf(s[4 * g + e], s[4 * g + 2 + e]);
#pragma unroll
            for (int o = 4; o < 32; o <<= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
            if (lane < 4) xmax[w4 * N + nq + 8 * g + e] = m;
          }
        }
        ld_softmax_bar();
        const int r = threadIdx.x - 128;
        if (r < N) {
          const float mx = fmaxf(fmaxf(xmax[r], xmax[N + r]), fmaxf(xmax[2 * N + r], xmax[3 * N + r]));
          const float old = mref[r];
          const bool up = mx > old + kLdSlack;
          corr[r] = up ? ex2(old - mx) : 1.f;
          if (up) mref[r] = mx;
        }
        ld_softmax_bar();
        if (ok && j > 0) ok = mbar_wait(o_done, (j - 1) & 1, abort_flag, timeout_ns);  // nothing is being added to the output
        ok = __all_sync(0xffffffffu, ok);
        tc_fence_after_sync();
        if (ok && j > 0) {
#pragma unroll
          for (int i = 0; i < 2 * kGroups; ++i) l[i] *= corr[nq + 8 * (i >> 1) + (i & 1)];
#pragma unroll 1
          for (int pr = 0; pr < kPairs; ++pr) {
#pragma unroll
            for (int c = 0; c < kCols / 8; ++c) {
              uint32_t r[8];
              const uint32_t at = lane_base + N * (2 + pr) + c * 8;
              tmem_ld_32x8(at, r);
              tmem_ld_wait();
#pragma unroll
              for (int i = 0; i < 8; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * corr[n0 + c * 8 + i]);
              tmem_st_32x8(at, r);
            }
          }
          tmem_st_wait();
        }
      }
      if (!ok) continue;
      uint32_t pk[2 * kGroups];  // [group][key block]
#pragma unroll
      for (int g = 0; g < kGroups; ++g) {
        const float2 m = *reinterpret_cast<const float2*>(mref + nq + 8 * g);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float x = ex2(s[4 * g + e] - ((e & 1) ? m.y : m.x));
          s[4 * g + e] = masked && !(s[4 * g + e] > -INFINITY) ? 0.f : x;  // a masked score is -inf, also without a reference
        }
        l[2 * g] += s[4 * g] + s[4 * g + 2];
        l[2 * g + 1] += s[4 * g + 1] + s[4 * g + 3];
#pragma unroll
        for (int kb = 0; kb < 2; ++kb)
          pk[2 * g + kb] = p.bf16 ? pack_bf16x2(s[4 * g + 2 * kb], s[4 * g + 2 * kb + 1]) : pack_f16x2(s[4 * g + 2 * kb], s[4 * g + 2 * kb + 1]);
      }
      const uint32_t dst = p_addr + (j & 1) * kRowAtom;
      if constexpr (kGroups == 1) {
        stmatrix_x2_trans(dst, pk[0], pk[1]);
      } else {
#pragma unroll
        for (int g = 0; g < kGroups; g += 2) stmatrix_x4_trans(dst + g * 8 * 128, pk[2 * g], pk[2 * g + 1], pk[2 * g + 2], pk[2 * g + 3]);
      }
      if (lane < 16 && key0 + w4 * 16 + lane >= n_keys) {  // slots beyond the sequence may hold anything: zero weight, zero value
        for (int pr = 0; pr < kPairs; ++pr) {
          uint4* row = reinterpret_cast<uint4*>(ring + ((j * kPairs + pr) % kSlots) * kLdSlot + half * kLdAtom + (w4 * 16 + lane) * 128);
#pragma unroll
          for (int i = 0; i < 8; ++i) row[i] = make_uint4(0, 0, 0, 0);
        }
      }
      __syncwarp();
      tc_fence_before_sync();     // this thread's TMEM accesses are done
      fence_view_async_shared();  // its shared-memory writes are visible to the tensor core
      __syncwarp();
      if (lane == 0) mbar_arrive(p_full + (j & 1));
    }
    // ---- row sums over the keys, then the normalised partial output and its log-sum-exp
#pragma unroll
    for (int i = 0; i < 2 * kGroups; ++i) {
      float sum = l[i];
#pragma unroll
      for (int o = 4; o < 32; o <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
      if (lane < 4) xsum[w4 * N + nq + 8 * (i >> 1) + (i & 1)] = sum;
    }
    ld_softmax_bar();
    const int r = threadIdx.x - 128;
    if (r < N) {
      const float sum = (xsum[r] + xsum[N + r]) + (xsum[2 * N + r] + xsum[3 * N + r]);
      corr[r] = sum > 0.f ? 1.f / sum : 0.f;
      if (r0 + r < n_rows)
        p.lse_part[static_cast<size_t>(row_base + r) * p.splits + split] =
            sum > 0.f ? (mref[r] + log2f(sum)) * 0.6931471805599453f : -INFINITY;
    }
    ld_softmax_bar();
    if (tile0 < tile1) {
      if (ok) ok = mbar_wait(o_done, (n_mine - 1) & 1, abort_flag, timeout_ns);
      ok = __all_sync(0xffffffffu, ok);
      tc_fence_after_sync();
      if (ok) {
#pragma unroll 1
        for (int pr = 0; pr < kPairs; ++pr) {
          const int col = pr * 128 + w4 * 32 + lane;
          float o[kCols];
          tmem_ld_cols<kCols>(lane_base + N * (2 + pr), o);
#pragma unroll
          for (int i = 0; i < kCols; ++i)
            if (r0 + n0 + i < n_rows && col < p.pitch)
              p.o_part[(static_cast<size_t>(row_base + n0 + i) * p.splits + split) * p.pitch + col] = o[i] * corr[n0 + i];
        }
      }
    }
  }

  tc_fence_before_sync();
  __syncthreads();
  if (warp == 2) tmem_dealloc(tmem_base, kTmemCols);
  if (threadIdx.x == 0 && *abort_flag != 0u && p.status != nullptr) atomicMax(p.status, static_cast<uint32_t>(kStatusPipeTimeout));
}

template <int N, int RK>
static int launch_latent_decode(const CUtensorMap& tc, const CUtensorMap& tq, const LatentDecodeParams& p, int B, cudaStream_t s) {
  static bool configured[64] = {false};
  int dev = 0;
  B200_CHECK_CUDA(cudaGetDevice(&dev));
  if (!configured[dev & 63]) {
    B200_CHECK_CUDA(cudaFuncSetAttribute(latent_decode_kernel<N, RK>, cudaFuncAttributeMaxDynamicSharedMemorySize, ld_smem_bytes(N, RK)));
    configured[dev & 63] = true;
  }
  const dim3 grid(p.splits, (p.S * p.H + N - 1) / N, B);
  B200_CHECK_CUDA(launch_pdl(latent_decode_kernel<N, RK>, grid, dim3(kLdThreads), ld_smem_bytes(N, RK), s, tc, tq, p));
  return kOk;
}
template <int N>
static int launch_latent_decode_rank(const CUtensorMap& tc, const CUtensorMap& tq, const LatentDecodeParams& p, int B, cudaStream_t s) {
  if (p.pitch <= 128) return launch_latent_decode<N, 128>(tc, tq, p, B, s);
  if (p.pitch <= 256) return launch_latent_decode<N, 256>(tc, tq, p, B, s);
  if (p.pitch <= 384) return launch_latent_decode<N, 384>(tc, tq, p, B, s);
  return launch_latent_decode<N, 512>(tc, tq, p, B, s);
}

}  // namespace b200

using namespace b200;

// q [B * S * H, pitch]; cache [num_slots, pitch] in pages of `page` slots (a multiple of 64); partial results as in
// b200_latent_combine. rows_per_cta: 16, 32 or 64.
B200_API int b200_latent_decode(const void* q, const void* cache, long long num_slots, const int* block_table, int bt_stride,
                                const int* kv_lens, int B, int S, int H, int pitch, int page, float scale, int splits,
                                int rows_per_cta, float* o_part, float* lse_part, int dtype, uint32_t* status, void* stream) {
  B200_REQUIRE(dtype == kBF16 || dtype == kF16, "latent decode attention supports bf16 / f16");
  B200_REQUIRE(rows_per_cta == 16 || rows_per_cta == 32 || rows_per_cta == 64, "rows_per_cta must be 16, 32 or 64, got %d", rows_per_cta);
  B200_REQUIRE(B >= 1 && S >= 1 && H >= 1 && B <= 65535 && num_slots >= 64, "bad latent attention shape");
  B200_REQUIRE(pitch >= 8 && pitch % 8 == 0 && pitch <= 512, "the latent row (%d elements) must be a multiple of 8 and at most 512", pitch);
  B200_REQUIRE(page >= 64 && page % 64 == 0, "the page size (%d) must be a multiple of 64", page);
  B200_REQUIRE(scale > 0.f, "the score scale must be positive");
  B200_REQUIRE(splits >= 1 && o_part && lse_part, "latent attention needs its partial buffers");
  B200_REQUIRE((S * H + rows_per_cta - 1) / rows_per_cta <= 65535, "too many query rows (%d)", S * H);
  CUtensorMap tc, tq;
  int rc = make_tma_2d(&tc, cache, dtype, num_slots, pitch, pitch, 64, 64, true);
  if (rc != kOk) return rc;
  rc = make_tma_2d(&tq, q, dtype, static_cast<uint64_t>(B) * S * H, pitch, pitch, rows_per_cta, 64, true);
  if (rc != kOk) return rc;
  LatentDecodeParams p;
  memset(&p, 0, sizeof(p));
  p.block_table = block_table; p.kv_lens = kv_lens; p.o_part = o_part; p.lse_part = lse_part; p.bt_stride = bt_stride; p.page = page;
  p.H = H; p.S = S; p.pitch = pitch; p.splits = splits; p.bf16 = dtype == kBF16; p.scale_log2e = scale * 1.4426950408889634f;
  p.status = status;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (rows_per_cta == 16) return launch_latent_decode_rank<16>(tc, tq, p, B, s);
  if (rows_per_cta == 32) return launch_latent_decode_rank<32>(tc, tq, p, B, s);
  return launch_latent_decode_rank<64>(tc, tq, p, B, s);
}
