// Experts: many small linear layers of which every token uses a few. A step's (token, choice) pairs are sorted by expert, and one launch
// per projection runs all experts that the step uses, each on its own rows; an expert that nobody chose costs neither products nor bytes.
//
// `expert_choose_kernel`: a warp per token turns a router's logits into the token's `top` experts, those with the largest logits, and their
// weights, sigmoid(logit) each; one more logit behind the experts' may be turned into a gate per token, its sigmoid.
// `expert_sort_kernel` (one CTA): the experts of every token come from a stored table of token ids or from the choice above, `top` of them
// per token; pair p = k n + token stands for the token's k-th choice. It writes the pairs in expert order (which of an expert's pairs comes first does not
// matter: every row is computed on its own) and the list of row tiles, (expert, first row, end), cut to the tile size of the products.
// `expert_gather_kernel` copies the tokens' activations into that order, so that a tile's rows lie one behind the other.
//
// bfloat16: `grouped_tc_kernel`, tcgen05 with the accumulator in tensor memory, the single-tile form of gemm_tc.cu (128 weight rows by BN
// rows, K in one range, TMA through a ring of stages) with the tile's expert read from the list; the weights of all experts are one
// matrix [E M, K]. float32: `grouped_f32_kernel`, the additions of gemm_f32.cu (32 classes of k, joined by a butterfly). Both have two
// epilogues: the gated product silu(gate) * up of an expert's gate rows and up rows, which stays in expert order, and a store that
// scatters row p to [k][token], so that the choices of a token are `top` partial sums in a fixed order for whoever adds them. Where a pair's
// weight multiplies the expert's input, it is applied to the two sums in front of the gate, in 32-bit.
//
// What a pair's result is depends on its token and expert alone, never on the tile it falls into.
#include <algorithm>

#include "gemm_tc_tile.cuh"
#include "step_ops.h"

SB_DEFINE_LAST_ERROR()

namespace {

using namespace sb::tc5;
using namespace sb::gemm_tile;

constexpr int kMaxExperts = 1024;
constexpr int kSortThreads = 1024;
constexpr int kMaxStages = 8;
constexpr int kThreads = 192;
constexpr int kSmemBudget = 200 * 1024;

// ------------------------------------------------------------------ routing
// logits [n][ldz] float32; choice [n][top] the experts by descending logit (the smaller index among equals), weights [top][n] (pair
// p = k n + token) their sigmoids, gate [n] (or null) the sigmoid of logit E. PER: experts a lane holds.
__device__ __forceinline__ float sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }

template <int PER>
__global__ void __launch_bounds__(128) expert_choose_kernel(const float* __restrict__ logits, int ldz, int n, int E, int top,
                                                            int32_t* __restrict__ choice, float* __restrict__ weights, float* __restrict__ gate) {
  sb::grid_launch_dependents();
  sb::grid_dependency_wait();
  const int row = (blockIdx.x * blockDim.x + threadIdx.x) >> 5, lane = threadIdx.x & 31;
  if (row >= n) return;
  const float* z = logits + static_cast<int64_t>(row) * ldz;
  float v[PER];
#pragma unroll
  for (int i = 0; i < PER; ++i) v[i] = lane + 32 * i < E ? z[lane + 32 * i] : -INFINITY;
  if (gate != nullptr && lane == 0) gate[row] = sigmoid(z[E]);
  uint32_t taken = 0;               // bit i: this lane's i-th expert has been chosen
  for (int k = 0; k < top; ++k) {
    float best = -INFINITY;
    int at = 0x7fffffff;
#pragma unroll
    for (int i = 0; i < PER; ++i)
      if (!((taken >> i) & 1u) && lane + 32 * i < E && (at == 0x7fffffff || v[i] > best)) best = v[i], at = lane + 32 * i;
    for (int o = 16; o > 0; o >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, o);
      const int oa = __shfl_xor_sync(0xffffffffu, at, o);
      if (oa != 0x7fffffff && (at == 0x7fffffff || ob > best || (ob == best && oa < at))) best = ob, at = oa;
    }
    if ((at & 31) == lane) taken |= 1u << (at >> 5);
    if (lane == 0) choice[static_cast<int64_t>(row) * top + k] = min(at, E - 1), weights[static_cast<int64_t>(k) * n + row] = sigmoid(best);
  }
}

// order [pairs]; tiles: [0] = how many, then (expert, first row, end row) each.
__global__ void __launch_bounds__(kSortThreads) expert_sort_kernel(const int32_t* __restrict__ tokens, const int32_t* __restrict__ slots,
                                                                   const int32_t* __restrict__ sampled, const int32_t* __restrict__ table, int vocab,      // vocab 0: the table's rows are the step's tokens
                                                                   int n, int top, int E, int tile, int32_t* __restrict__ order,
                                                                   int32_t* __restrict__ tiles, int max_tiles) {
  __shared__ int count[kMaxExperts], place[kMaxExperts], tile_at[kMaxExperts + 1];
  sb::grid_launch_dependents();
  for (int e = threadIdx.x; e < E; e += blockDim.x) count[e] = 0;
  __syncthreads();
  sb::grid_dependency_wait();
  const int pairs = n * top;
  auto expert_of = [&](int p) {
    const int row = p % n;
    if (vocab == 0) return min(max(table[static_cast<int64_t>(row) * top + p / n], 0), E - 1);
    int tok = tokens[row];
    if (tok == -1 && sampled != nullptr) tok = sampled[slots[row]];
    if (tok < 0 || tok >= vocab) tok = 0;
    return min(max(table[static_cast<int64_t>(tok) * top + p / n], 0), E - 1);
  };
  for (int p = threadIdx.x; p < pairs; p += blockDim.x) atomicAdd(&count[expert_of(p)], 1);
  __syncthreads();
  if (threadIdx.x < 32) {          // one warp: running sums of the counts and of the tiles, 32 experts at a time
    const int lane = threadIdx.x;
    int rows_before = 0, tiles_before = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
      const int e = e0 + lane, c = e < E ? count[e] : 0, t = (c + tile - 1) / tile;
      int cs = c, ts = t;
      for (int o = 1; o < 32; o <<= 1) {
        const int a = __shfl_up_sync(0xffffffffu, cs, o), b = __shfl_up_sync(0xffffffffu, ts, o);
        if (lane >= o) cs += a, ts += b;
      }
      if (e < E) place[e] = rows_before + cs - c, tile_at[e] = tiles_before + ts - t;
      rows_before += __shfl_sync(0xffffffffu, cs, 31), tiles_before += __shfl_sync(0xffffffffu, ts, 31);
    }
    if (lane == 0) tiles[0] = min(tiles_before, max_tiles);
  }
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += blockDim.x) {
    const int first = place[e], end = first + count[e];
    for (int i = 0, r = first; r < end; ++i, r += tile) {
      const int t = tile_at[e] + i;
      if (t < max_tiles) tiles[1 + 3 * t] = e, tiles[2 + 3 * t] = r, tiles[3 + 3 * t] = end;
    }
  }
  __syncthreads();
  for (int p = threadIdx.x; p < pairs; p += blockDim.x) order[atomicAdd(&place[expert_of(p)], 1)] = p;
}

// out[i] = x[order[i] % n], rows of `chunks` pieces of T.
template <class T>
__global__ void __launch_bounds__(128) expert_gather_kernel(const T* __restrict__ x, int64_t ldx, const int32_t* __restrict__ order, int n,
                                                            T* __restrict__ out, int chunks) {
  sb::grid_launch_dependents();
  sb::grid_dependency_wait();
  const T* src = x + static_cast<int64_t>(order[blockIdx.x] % n) * ldx;
  T* dst = out + static_cast<int64_t>(blockIdx.x) * chunks;
  for (int c = threadIdx.x; c < chunks; c += blockDim.x) dst[c] = src[c];
}

// ------------------------------------------------------------------ tensor cores
struct TcParams {
  void* out;            // kSwiglu: bfloat16 [pairs, half_rows] in expert order; kStore: float32 [top][n][M]
  int M, K;             // one expert's rows (kSwiglu: gate rows, then up rows) and columns
  int half_rows;
  int block_n, stages;
  const int32_t* tiles;
  const int32_t* order;
  const float* pair_weight;      // kSwiglu: a factor on every pair's input, by pair, or null
  int* status;
};

template <int EPI>
__global__ void __launch_bounds__(kThreads, 1)
grouped_tc_kernel(const __grid_constant__ CUtensorMap map_w, const __grid_constant__ CUtensorMap map_x, const TcParams p) {
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  __shared__ __align__(8) uint64_t full_bar[kMaxStages];
  __shared__ __align__(8) uint64_t empty_bar[kMaxStages];
  __shared__ __align__(8) uint64_t accum_bar;
  __shared__ uint32_t tmem_base_s;
  __shared__ float column_weight[EPI == kSwiglu ? 128 : 1];

  sb::grid_launch_dependents();
  sb::grid_dependency_wait();                    // which expert this tile belongs to is the sort's result
  if (static_cast<int>(blockIdx.y) >= p.tiles[0]) return;
  const int expert = p.tiles[1 + 3 * blockIdx.y], n0 = p.tiles[2 + 3 * blockIdx.y], end = p.tiles[3 + 3 * blockIdx.y];

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int BN = p.block_n;
  const int stage_bytes = kStageA + BN * 128;
  const uint32_t smem0 = (smem_u32(smem_raw) + 1023u) & ~1023u;
  const int tile_m = blockIdx.x, iters = (p.K + kTileK - 1) / kTileK;
  const uint32_t tmem_cols = tmem_alloc_cols(BN);

  if (EPI == kSwiglu && p.pair_weight != nullptr && threadIdx.x >= 64) {       // (the epilogue's warps: a tile has at most 128 rows)
    const int n = n0 + threadIdx.x - 64;
    column_weight[threadIdx.x - 64] = n < end ? p.pair_weight[p.order[n]] : 0.0f;
  }
  if (threadIdx.x == 0) {
    prefetch_tensormap(&map_w);
    prefetch_tensormap(&map_x);
    for (int s = 0; s < p.stages; ++s) {
      mbar_init(smem_u32(&full_bar[s]), 1);
      mbar_init(smem_u32(&empty_bar[s]), 1);
    }
    mbar_init(smem_u32(&accum_bar), 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) tmem_alloc(smem_u32(&tmem_base_s), tmem_cols);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = tmem_base_s;

  if (warp == 0) {
    if (lane == 0) {
      // ---------------- producer: TMA loads
      const int row_w = expert * p.M + (EPI == kSwiglu ? tile_m * 64 : tile_m * kTileM);
      int st = 0;
      uint32_t par = 1;                          // (a wait on this parity of a barrier nobody has arrived on yet returns at once)
      for (int i = 0; i < iters; ++i) {
        mbar_wait(smem_u32(&empty_bar[st]), par, p.status, 1);
        const uint32_t bar = smem_u32(&full_bar[st]);
        const uint32_t a = smem0 + st * stage_bytes;
        mbar_expect_tx(bar, stage_bytes);
        tma_load_2d(a, &map_w, bar, i * kTileK, row_w);
        if (EPI == kSwiglu) tma_load_2d(a + kStageA / 2, &map_w, bar, i * kTileK, row_w + p.half_rows);
        tma_load_2d(a + kStageA, &map_x, bar, i * kTileK, n0);
        if (++st == p.stages) st = 0, par ^= 1;
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      // ---------------- MMA issuer
      const uint32_t idesc = instr_desc(BN);
      const uint64_t desc_fixed = smem_desc_sw128(0);
      const uint32_t a_lo = (smem0 & 0x3FFFF) >> 4, stage_lo = static_cast<uint32_t>(stage_bytes) >> 4;
      uint32_t st = 0, par = 0, accumulate = 0;
      for (int i = 0; i < iters; ++i) {
        mbar_wait(smem_u32(&full_bar[st]), par, p.status, 2);
        tc_fence_after();
        const uint64_t da = desc_fixed | (a_lo + st * stage_lo), db = da + (kStageA >> 4);
        umma_bf16(tmem_base, da, db, idesc, accumulate);
        umma_bf16(tmem_base, da + 2, db + 2, idesc, 1u);
        umma_bf16(tmem_base, da + 4, db + 4, idesc, 1u);
        umma_bf16(tmem_base, da + 6, db + 6, idesc, 1u);
        accumulate = 1u;
        umma_commit(smem_u32(&empty_bar[st]));
        if (++st == static_cast<uint32_t>(p.stages)) st = 0, par ^= 1;
      }
      umma_commit(smem_u32(&accum_bar));
    }
    __syncwarp();
  } else {
    // ---------------- epilogue: warps 2..5 own TMEM lanes 32 * (warp % 4) ..
    const int quarter = warp & 3;
    const bool ok = mbar_wait(smem_u32(&accum_bar), 0, p.status, 3);
    tc_fence_after();
    if (EPI == kSwiglu) {
      float* xch = reinterpret_cast<float*>(smem_raw + (smem0 - smem_u32(smem_raw)));      // stage 0 is free by now
      swiglu_tile(tmem_base, xch, static_cast<bf16*>(p.out), p.half_rows, tile_m, p.half_rows, n0, end, BN, quarter, lane, ok,
                  Gate(), p.pair_weight != nullptr ? column_weight : nullptr);
    } else {
      const int m = tile_m * kTileM + quarter * 32 + lane;
      for (int c0 = 0; c0 < BN && n0 + c0 < end; c0 += 16) {
        float v[16];
        tmem_load16(tmem_base + (static_cast<uint32_t>(quarter * 32) << 16) + c0, v);
        if (m < p.M && ok) {
#pragma unroll
          for (int c = 0; c < 16; ++c)
            if (n0 + c0 + c < end) static_cast<float*>(p.out)[static_cast<int64_t>(p.order[n0 + c0 + c]) * p.M + m] = v[c];
        }
      }
    }
    tc_fence_before();
  }
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, tmem_cols);
  }
}

// ------------------------------------------------------------------ 32-bit
template <bool VEC>
__device__ __forceinline__ void load8(const bf16* p, int left, float* v) {
  if (VEC) {
    const uint4 raw = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      v[2 * i] = __uint_as_float(w[i] << 16);
      v[2 * i + 1] = __uint_as_float(w[i] & 0xFFFF0000u);
    }
  } else {
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] = e < left ? __bfloat162float(p[e]) : 0.0f;
  }
}
template <bool VEC>
__device__ __forceinline__ void load8(const float* p, int left, float* v) {
  if (VEC) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    v[0] = a.x, v[1] = a.y, v[2] = a.z, v[3] = a.w, v[4] = b.x, v[5] = b.y, v[6] = b.z, v[7] = b.w;
  } else {
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] = e < left ? p[e] : 0.0f;
  }
}

constexpr int kWarps = 4, kF32Rows = 8, kF32Features = 2;

// A warp makes kF32Features features (GATED: one gate row and its up row) of the rows of a tile; lane c is class c of k.
// GATED: rows of x through order[i] % n, out [pairs][half] in expert order. Else: row i of x, out row order[i].
template <class TX, class TW, class TO, bool VEC, bool GATED>
__global__ void __launch_bounds__(kWarps * 32) grouped_f32_kernel(const TX* __restrict__ x, int64_t ldx, const TW* __restrict__ w, TO* __restrict__ out,
                                                                  int M, int K, int n, const int32_t* __restrict__ tiles,
                                                                  const int32_t* __restrict__ order, const float* __restrict__ pair_weight) {
  sb::grid_launch_dependents();
  sb::grid_dependency_wait();
  if (static_cast<int>(blockIdx.y) >= tiles[0]) return;
  const int expert = tiles[1 + 3 * blockIdx.y], n0 = tiles[2 + 3 * blockIdx.y], end = tiles[3 + 3 * blockIdx.y];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int half = M / 2, f0 = (blockIdx.x * kWarps + warp) * (GATED ? 1 : kF32Features);
  if (f0 >= (GATED ? half : M)) return;
  const TW* wrow[kF32Features];
#pragma unroll
  for (int i = 0; i < kF32Features; ++i)
    wrow[i] = w + (static_cast<int64_t>(expert) * M + (GATED ? f0 + i * half : min(f0 + i, M - 1))) * K;
  const TX* xrow[kF32Rows];
#pragma unroll
  for (int j = 0; j < kF32Rows; ++j) {
    const int r = min(n0 + j, end - 1);
    xrow[j] = x + static_cast<int64_t>(GATED ? order[r] % n : r) * ldx;
  }
  float acc[kF32Features][kF32Rows];
#pragma unroll
  for (int i = 0; i < kF32Features; ++i)
#pragma unroll
    for (int j = 0; j < kF32Rows; ++j) acc[i][j] = 0.0f;
  for (int k = lane * 8; k < K; k += 256) {
    float wv[kF32Features][8];
#pragma unroll
    for (int i = 0; i < kF32Features; ++i) load8<VEC>(wrow[i] + k, K - k, wv[i]);
#pragma unroll
    for (int j = 0; j < kF32Rows; ++j) {
      float xv[8];
      load8<VEC>(xrow[j] + k, K - k, xv);
#pragma unroll
      for (int e = 0; e < 8; ++e)
#pragma unroll
        for (int i = 0; i < kF32Features; ++i) acc[i][j] = fmaf(xv[e], wv[i][e], acc[i][j]);
    }
  }
#pragma unroll
  for (int i = 0; i < kF32Features; ++i)
#pragma unroll
    for (int j = 0; j < kF32Rows; ++j)
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) acc[i][j] += __shfl_xor_sync(0xffffffffu, acc[i][j], o);
#pragma unroll
  for (int j = 0; j < kF32Rows; ++j) {
    if (lane != j || n0 + j >= end) continue;
    if (GATED) {
      const float weight = pair_weight != nullptr ? pair_weight[order[n0 + j]] : 1.0f;
      const float g = acc[0][j] * weight, u = acc[1][j] * weight;
      out[static_cast<int64_t>(n0 + j) * half + f0] = sb::narrow<TO>((g / (1.0f + expf(-g))) * u);
    } else {
#pragma unroll
      for (int i = 0; i < kF32Features; ++i)
        if (f0 + i < M) out[static_cast<int64_t>(order[n0 + j]) * M + f0 + i] = sb::narrow<TO>(acc[i][j]);
    }
  }
}

template <class TX, class TW, class TO, bool GATED>
int launch_f32(const void* x, int64_t ldx, const void* w, void* out, int M, int K, int n, int max_tiles, const int32_t* tiles, const int32_t* order,
               const float* pair_weight, cudaStream_t stream) {
  const int features = kWarps * (GATED ? 1 : kF32Features);
  const dim3 grid(((GATED ? M / 2 : M) + features - 1) / features, max_tiles);
  const bool vec = K % 8 == 0 && (ldx * sizeof(TX)) % 16 == 0 && ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(w)) & 15) == 0;
  if (vec) sb::launch_pdl(grouped_f32_kernel<TX, TW, TO, true, GATED>, grid, dim3(kWarps * 32), 0, stream, static_cast<const TX*>(x), ldx,
                          static_cast<const TW*>(w), static_cast<TO*>(out), M, K, n, tiles, order, pair_weight);
  else sb::launch_pdl(grouped_f32_kernel<TX, TW, TO, false, GATED>, grid, dim3(kWarps * 32), 0, stream, static_cast<const TX*>(x), ldx,
                      static_cast<const TW*>(w), static_cast<TO*>(out), M, K, n, tiles, order, pair_weight);
  return sb::check_launch("sb_op_expert_linear");
}

// Rows of a tile of the tensor-core products: near the rows an expert gets on average, so that few weights are streamed for empty columns
// and few tiles share an expert. (A row's result does not depend on it.)
int tile_rows(int pairs, int E, bool tc) {
  if (!tc) return kF32Rows;
  const int mean = (pairs + E - 1) / E;
  int t = 16;
  while (t < mean && t < 128) t *= 2;
  return t;
}
// The most tiles that `pairs` rows over E experts can be cut into.
int most_tiles(int pairs, int E, int tile) { return std::min(pairs, pairs / tile + std::min(pairs, E)); }

}  // namespace

SB_EXPORT int sb_expert_max() { return kMaxExperts; }

// Elements of the tile list for up to `tokens` tokens.
SB_EXPORT int sb_expert_tile_ints(int tokens, int top, int E) { return 1 + 3 * most_tiles(tokens * top, E, 1); }

SB_EXPORT void sb_grouped_gemm_use_status_word(int* device_word) { status_word_given() = device_word; }

// i: 0 logits, 1 ldz, 2 experts, 3 top, 4 choice [n][top], 5 weights [top][n], 6 gate [n] from the logit behind the experts' (or 0)
SB_EXPORT int sb_op_expert_choose(const SbOp* op, const SbStep* s, void* stream) {
  using namespace sbstep;
  if (s->n <= 0) return SB_OP_SKIPPED;
  const int ldz = (int)op->i[1], E = (int)op->i[2], top = (int)op->i[3];
  if (top < 1 || E < top || E > kMaxExperts || ldz < E + (op->i[6] != 0 ? 1 : 0))
    return sb::fail("sb_op_expert_choose: %d of %d experts (at most %d) in rows of %d logits", top, E, kMaxExperts, ldz), SB_OP_FAILED;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
#define SB_CHOOSE(PER)                                                                                                                   \
  sb::launch_pdl(expert_choose_kernel<PER>, dim3((s->n + 3) / 4), dim3(128), 0, st, ptr<const float>(op->i[0]), ldz, s->n, E, top,       \
                 ptr<int32_t>(op->i[4]), ptr<float>(op->i[5]), ptr<float>(op->i[6]))
  if (E <= 32) SB_CHOOSE(1);
  else if (E <= 128) SB_CHOOSE(4);
  else SB_CHOOSE(32);
#undef SB_CHOOSE
  return sb::check_launch("sb_op_expert_choose");
}

// i: 0 table [vocab][top], 1 vocab (0: the table is the step's choice [n][top]), 2 top, 3 experts, 4 sampled tokens per slot (or 0), 5 order, 6 tiles, 7 products on the tensor cores
SB_EXPORT int sb_op_expert_sort(const SbOp* op, const SbStep* s, void* stream) {
  using namespace sbstep;
  if (s->n <= 0) return SB_OP_SKIPPED;
  const int top = (int)op->i[2], E = (int)op->i[3], pairs = s->n * top;
  if (top < 1 || E < top || E > kMaxExperts) return sb::fail("sb_op_expert_sort: %d of %d experts (at most %d)", top, E, kMaxExperts), SB_OP_FAILED;
  const int tile = tile_rows(pairs, E, op->i[7] != 0);
  sb::launch_pdl(expert_sort_kernel, dim3(1), dim3(pairs <= 128 ? 128 : kSortThreads), 0, static_cast<cudaStream_t>(stream), tokens(s), slots(s),
                 ptr<const int32_t>(op->i[4]), ptr<const int32_t>(op->i[0]), (int)op->i[1], s->n, top, E, tile, ptr<int32_t>(op->i[5]),
                 ptr<int32_t>(op->i[6]), most_tiles(pairs, E, tile));
  return sb::check_launch("sb_op_expert_sort");
}

// i: 0 x, 1 ldx, 2 element bytes, 3 order, 4 top, 5 out, 6 width
SB_EXPORT int sb_op_expert_gather(const SbOp* op, const SbStep* s, void* stream) {
  using namespace sbstep;
  if (s->n <= 0) return SB_OP_SKIPPED;
  const int64_t row_bytes = op->i[6] * op->i[2], ld_bytes = op->i[1] * op->i[2];
  const dim3 grid(s->n * (int)op->i[4]);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (row_bytes % 16 == 0 && ld_bytes % 16 == 0 && ((op->i[0] | op->i[5]) & 15) == 0)
    sb::launch_pdl(expert_gather_kernel<uint4>, grid, dim3(128), 0, st, ptr<const uint4>(op->i[0]), ld_bytes / 16, ptr<const int32_t>(op->i[3]), s->n,
                   ptr<uint4>(op->i[5]), (int)(row_bytes / 16));
  else if (row_bytes % 2 == 0 && ld_bytes % 2 == 0)
    sb::launch_pdl(expert_gather_kernel<uint16_t>, grid, dim3(128), 0, st, ptr<const uint16_t>(op->i[0]), ld_bytes / 2, ptr<const int32_t>(op->i[3]), s->n,
                   ptr<uint16_t>(op->i[5]), (int)(row_bytes / 2));
  else
    return sb::fail("sb_op_expert_gather: rows of %lld bytes", (long long)row_bytes), SB_OP_FAILED;
  return sb::check_launch("sb_op_expert_gather");
}

// i: 0 x (tensor cores: rows in expert order; 32-bit gated: rows by token), 1 ldx, 2 x dtype, 3 weights [E M][K], 4 their dtype, 5 out, 6 out dtype,
//    7 M, 8 K, 9 experts, 10 top, 11 gated (1) or scattered store (0), 12 order, 13 tiles, 14 on the tensor cores,
//    15 a factor on every pair's input [top][n] float32 (gated only; 0: none)
SB_EXPORT int sb_op_expert_linear(const SbOp* op, const SbStep* s, void* stream) {
  using namespace sbstep;
  if (s->n <= 0) return SB_OP_SKIPPED;
  const int M = (int)op->i[7], K = (int)op->i[8], E = (int)op->i[9], top = (int)op->i[10], pairs = s->n * top;
  const bool gated = op->i[11] != 0, tc = op->i[14] != 0;
  const int32_t* order = ptr<const int32_t>(op->i[12]);
  const int32_t* tiles = ptr<const int32_t>(op->i[13]);
  const void* x = ptr<const void>(op->i[0]);
  const void* w = ptr<const void>(op->i[3]);
  void* out = ptr<void>(op->i[5]);
  const float* pair_weight = ptr<const float>(op->i[15]);
  const int64_t ldx = op->i[1];
  if (pair_weight != nullptr && !gated) return sb::fail("sb_op_expert_linear: factors on the pairs' inputs go with the gated product"), SB_OP_FAILED;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (M <= 0 || K <= 0 || (gated && M % 2 != 0)) return sb::fail("sb_op_expert_linear: %d x %d", M, K), SB_OP_FAILED;
  const int tile = tile_rows(pairs, E, tc), max_tiles = most_tiles(pairs, E, tile);
  if (max_tiles > 65535) return sb::fail("sb_op_expert_linear: %d tiles exceed the grid", max_tiles), SB_OP_FAILED;
  if (!tc) {
    const int xd = (int)op->i[2], wd = (int)op->i[4], od = (int)op->i[6];
#define SB_EXPERT(TX, TW, TO)                                                                                              \
  (gated ? launch_f32<TX, TW, TO, true>(x, ldx, w, out, M, K, s->n, max_tiles, tiles, order, pair_weight, st)               \
         : launch_f32<TX, TW, float, false>(x, ldx, w, out, M, K, s->n, max_tiles, tiles, order, pair_weight, st))
    if (xd == 0 && wd == 0) return SB_EXPERT(float, float, float);
    if (xd == 0 && wd == 1) return SB_EXPERT(float, bf16, float);
    if (xd == 1 && wd == 0) return SB_EXPERT(bf16, float, bf16);
    if (xd == 1 && wd == 1) return SB_EXPERT(bf16, bf16, bf16);
#undef SB_EXPERT
    return sb::fail("sb_op_expert_linear: dtypes %d, %d, %d", xd, wd, od), SB_OP_FAILED;
  }
  if (K % 8 != 0 || ldx % 8 != 0 || ((op->i[0] | op->i[3]) & 15) != 0)
    return sb::fail("sb_op_expert_linear: K %d and the leading dimension %lld must be multiples of 8, operands 16-byte aligned", K, (long long)ldx), SB_OP_FAILED;
  TcParams p{};
  p.out = out, p.M = M, p.K = K, p.half_rows = M / 2, p.tiles = tiles, p.order = order, p.block_n = tile, p.pair_weight = pair_weight;
  p.status = status_word();
  if (!p.status) return sb::fail("sb_op_expert_linear: cannot allocate the status word"), SB_OP_FAILED;
  const int stage_bytes = kStageA + tile * 128;
  // two CTAs an SM: one's prologue and epilogue run beside the other's products
  p.stages = std::max(2, std::min({kMaxStages, (kSmemBudget / 2) / stage_bytes, (K + kTileK - 1) / kTileK}));
  const int64_t wd[2] = {K, static_cast<int64_t>(E) * M}, ws[2] = {1, K}, xd[2] = {K, pairs}, xs[2] = {1, ldx};
  const int wb[2] = {kTileK, gated ? 64 : kTileM}, xb[2] = {kTileK, tile};
  CUtensorMap map_w, map_x;
  if (!tensor_map_bf16(w, 2, wd, ws, wb, &map_w) || !tensor_map_bf16(x, 2, xd, xs, xb, &map_x))
    return sb::fail("sb_op_expert_linear: cuTensorMapEncodeTiled failed (M %d K %d)", M, K), SB_OP_FAILED;
  const dim3 grid(gated ? (M / 2 + 63) / 64 : (M + kTileM - 1) / kTileM, max_tiles);
  const size_t smem = static_cast<size_t>(p.stages) * stage_bytes + 1024;
  static sb::DeviceOnce once;
  if (once.needed()) {
    if (cudaFuncSetAttribute(grouped_tc_kernel<kSwiglu>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmemBudget + 2048) != cudaSuccess ||
        cudaFuncSetAttribute(grouped_tc_kernel<kStore>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmemBudget + 2048) != cudaSuccess)
      return sb::fail("sb_op_expert_linear: cannot raise the shared memory limit"), SB_OP_FAILED;
    once.done();
  }
  if (gated) sb::launch_pdl(grouped_tc_kernel<kSwiglu>, grid, dim3(kThreads), smem, st, map_w, map_x, p);
  else sb::launch_pdl(grouped_tc_kernel<kStore>, grid, dim3(kThreads), smem, st, map_w, map_x, p);
  return sb::check_launch("sb_op_expert_linear");
}
