// What stands between the q | k | v projection and the attention in designs with a short convolution on it, in one kernel:
//
//   y_t[c] = sum_j taps[c, j] u_(t - K + 1 + j)[c]      a causal convolution over time on every channel of q, k and v, u being the projection's
//                                                       output; zeros in front of the sequence
//   q, k: the first `rot` elements of every head turned by the token's position (pairs i, i + rot / 2), then, if asked for, the head divided
//         by its root mean square, x / sqrt(mean(x^2) + eps)
//   v:    as it is; or kept aside for later layers of the step; or mixed with what an earlier layer kept, (1 - lambda) v + lambda v_kept
//
// q is stored, k and v are appended to the token's pages. All of it is 32-bit. The last K - 1 inputs of a request, [K - 1][C] float32,
// oldest first, are its record; where the sequence starts in the step nothing of the record is read. A token's result has the same bits
// however the sequence was cut into steps: its inputs are the same sums wherever they come from, the taps are added oldest first, and a
// head's squares are added by lane over fixed elements and then by xor shuffles (which elements, the sizes alone decide).
#include "common.cuh"
#include "step_ops.h"

SB_DEFINE_LAST_ERROR()

namespace {

using bf16 = __nv_bfloat16;
constexpr int kInFlight = 8;
constexpr int kMaxTaps = 16;
constexpr int kTile = 16;         // tokens of an entry a block takes in steps with longer entries

__device__ __forceinline__ float folded(const float* p, int n_partials, int64_t stride) {
  float part[kInFlight];
#pragma unroll
  for (int s = 0; s < kInFlight; ++s)
    if (s < n_partials) part[s] = p[s * stride];
  float sum = part[0];
#pragma unroll
  for (int s = 1; s < kInFlight; ++s)
    if (s < n_partials) sum += part[s];
  for (int s = kInFlight; s < n_partials; ++s) sum += p[s * stride];
  return sum;
}
__device__ __forceinline__ float4 folded4(const float* p, int n_partials, int64_t stride) {
  float4 part[kInFlight];
#pragma unroll
  for (int s = 0; s < kInFlight; ++s)
    if (s < n_partials) part[s] = *reinterpret_cast<const float4*>(p + s * stride);
  float4 sum = part[0];
#pragma unroll
  for (int s = 1; s < kInFlight; ++s)
    if (s < n_partials) sum.x += part[s].x, sum.y += part[s].y, sum.z += part[s].z, sum.w += part[s].w;
  for (int s = kInFlight; s < n_partials; ++s) {
    const float4 a = *reinterpret_cast<const float4*>(p + s * stride);
    sum.x += a.x, sum.y += a.y, sum.z += a.z, sum.w += a.w;
  }
  return sum;
}

enum ValueMix { kOwn = 0, kKeep = 1, kMix = 2 };

struct ConvParams {
  const float* proj;         // [P][n][width]: q (Hq D) | k (Hkv D) | v (Hkv Dv) | whatever else the projection carries
  int n_partials;
  int64_t partial_stride;
  int width;
  const float* conv;         // [taps][C], C = Hq D + Hkv (D + Dv), or null: no convolution
  int taps;
  float* record;             // [slots][record_size]: the last taps - 1 inputs, [taps - 1][C]
  int64_t record_size;
  const int32_t* meta;       // [4][meta_stride]: slot, first row, length, first position of every entry
  int meta_stride, entries, tile;
  const float* cos_sin;      // [positions][rot / 2][2]
  int rot, unit;
  float eps;
  float* kept;               // [n][Hkv Dv]: the values an earlier layer kept, or null
  int mix;
  float lambda, rest;        // rest = 1 - lambda
  void* q_out;               // [n][Hq D]
  void* pages;
  const int32_t* block_table;
  int max_pages, page_size;
  int64_t page_stride, v_offset, head_stride;
  int Dc;
  int Hq, Hkv, D, Dv;
};

// The general form: any sizes, any number of taps. A block per (tile of an entry's tokens, head of q, k or v). The tile's inputs and the taps - 1 in front of it wait in shared memory, then a
// warp takes a token at a time. The block of an entry's first tile is the only one that touches the request's record: it reads what it
// needs of it first and writes the new one, its columns of it, when it is done.
template <class T, bool VEC>
__global__ void __launch_bounds__(128) conv_qkv_kernel(ConvParams p) {
  extern __shared__ __align__(16) float smem[];
  sb::grid_launch_dependents();
  const int unit = blockIdx.y, taps = p.taps, halo = taps - 1;
  const bool is_q = unit < p.Hq, is_v = unit >= p.Hq + p.Hkv;
  const int head = is_q ? unit : is_v ? unit - p.Hq - p.Hkv : unit - p.Hq;
  const int nq = p.Hq * p.D, nk = p.Hkv * p.D, C = nq + nk + p.Hkv * p.Dv;
  const int dim = is_v ? p.Dv : p.D, c0 = is_q ? head * p.D : is_v ? nq + nk + head * p.Dv : nq + head * p.D;
  float* w = smem;                                   // [taps][dim]
  float* in = w + taps * dim;                      // [halo + tile][dim]: row i is position first + i - halo
  float* out = in + (halo + p.tile) * dim;           // [tile][dim]
  int e = 0, tile = blockIdx.x, len = 1;
  if (p.tile == 1) {
    e = tile, tile = 0;
  } else {
    for (; e < p.entries; ++e) {
      len = p.meta[2 * p.meta_stride + e];
      const int tiles = (len + p.tile - 1) / p.tile;
      if (tile < tiles) break;
      tile -= tiles;
    }
  }
  if (e >= p.entries) return;
  const int slot = p.meta[e], row0 = p.meta[p.meta_stride + e], pos0 = p.meta[3 * p.meta_stride + e];
  const int t0 = tile * p.tile, nt = min(p.tile, len - t0);
  constexpr int VE = VEC ? 4 : 1;
  const int per = dim / VE;
  if (p.conv != nullptr)
    for (int i = threadIdx.x; i < taps * dim; i += blockDim.x) w[i] = p.conv[static_cast<int64_t>(i / dim) * C + c0 + i % dim];
  float* record = p.record != nullptr ? p.record + static_cast<int64_t>(slot) * p.record_size + c0 : nullptr;
  sb::grid_dependency_wait();
  for (int i = threadIdx.x; i < (halo + nt) * per; i += blockDim.x) {
    const int r = i / per, c = (i % per) * VE, t = t0 + r - halo;        // the t-th token of the entry
    float* dst = in + r * dim + c;
    if (t >= 0) {
      const float* src = p.proj + static_cast<int64_t>(row0 + t) * p.width + c0 + c;
      if constexpr (VEC) *reinterpret_cast<float4*>(dst) = folded4(src, p.n_partials, p.partial_stride);
      else *dst = folded(src, p.n_partials, p.partial_stride);
    } else if (pos0 + t >= 0) {                                          // in front of the step: the record's row halo + t
      const float* src = record + static_cast<int64_t>(halo + t) * C + c;
      if constexpr (VEC) *reinterpret_cast<float4*>(dst) = *reinterpret_cast<const float4*>(src);
      else *dst = *src;
    } else {
      if constexpr (VEC) *reinterpret_cast<float4*>(dst) = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
      else *dst = 0.0f;
    }
  }
  __syncthreads();
  if (t0 == 0 && halo > 0)       // the record behind the step: its row j is the entry's token len - halo + j
    for (int i = threadIdx.x; i < halo * per; i += blockDim.x) {
      const int j = i / per, c = (i % per) * VE, t = len - halo + j;
      float* dst = record + static_cast<int64_t>(j) * C + c;
      const float* far = p.proj + static_cast<int64_t>(row0 + t) * p.width + c0 + c;      // (read only where t lies behind this tile)
      const float* near = in + (t + halo) * dim + c;
      if constexpr (VEC) *reinterpret_cast<float4*>(dst) = t < nt ? *reinterpret_cast<const float4*>(near) : folded4(far, p.n_partials, p.partial_stride);
      else *dst = t < nt ? *near : folded(far, p.n_partials, p.partial_stride);
    }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, rh = p.rot / 2;
  for (int t = warp; t < nt; t += blockDim.x >> 5) {
    const float* u = in + t * dim;
    float* y = out + t * dim;
    auto convolved = [&](int d) {
      if (p.conv == nullptr) return u[d + halo * dim];
      float acc = 0.0f;
      for (int j = 0; j < taps; ++j) acc = fmaf(w[j * dim + d], u[j * dim + d], acc);
      return acc;
    };
    const int row = row0 + t0 + t, pos = pos0 + t0 + t;
    T* cached = nullptr;
    if (!is_q) {
      const int page = p.block_table[static_cast<int64_t>(slot) * p.max_pages + pos / p.page_size];
      cached = static_cast<T*>(p.pages) + static_cast<int64_t>(page) * p.page_stride + (is_v ? p.v_offset : 0) +
               static_cast<int64_t>(head) * p.head_stride + static_cast<int64_t>(pos % p.page_size) * p.Dc;
    }
    if (is_v) {
      float* kept = p.kept != nullptr ? p.kept + static_cast<int64_t>(row) * p.Hkv * p.Dv + head * p.Dv : nullptr;
      for (int d = lane; d < dim; d += 32) {
        float v = convolved(d);
        if (p.mix == kKeep) kept[d] = v;
        else if (p.mix == kMix) v = fmaf(p.lambda, kept[d], __fmul_rn(p.rest, v));
        cached[d] = sb::narrow<T>(v);
      }
      continue;
    }
    float ss = 0.0f;
    for (int i = lane; i < rh; i += 32) {
      const float a = convolved(i), b = convolved(i + rh);
      const float2 cs = *reinterpret_cast<const float2*>(p.cos_sin + (static_cast<int64_t>(pos) * rh + i) * 2);
      const float ra = __fsub_rn(__fmul_rn(a, cs.x), __fmul_rn(b, cs.y)), rb = __fadd_rn(__fmul_rn(b, cs.x), __fmul_rn(a, cs.y));
      y[i] = ra, y[i + rh] = rb;
      ss = fmaf(ra, ra, ss), ss = fmaf(rb, rb, ss);
    }
    for (int d = p.rot + lane; d < dim; d += 32) {
      const float a = convolved(d);
      y[d] = a;
      ss = fmaf(a, a, ss);
    }
    float scale = 1.0f;
    if (p.unit) {
      for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      scale = 1.0f / sqrtf(ss / static_cast<float>(dim) + p.eps);
    }
    __syncwarp();
    T* dst = is_q ? static_cast<T*>(p.q_out) + static_cast<int64_t>(row) * nq + head * p.D : cached;
    for (int d = lane; d < dim; d += 32) dst[d] = sb::narrow<T>(__fmul_rn(y[d], scale));
  }
}

// The form for two to four taps and heads of up to 128 elements, in fours: L lanes (a power of two) own a head of q, k or v, four elements
// each, and walk kRun consecutive tokens of an entry with the last inputs in registers: nothing passes through shared memory. The lanes of an
// entry's first run read and write the request's record, each its own columns of it.
constexpr int kRun = 8;

__device__ __forceinline__ float4 fma4(float4 w, float4 u, float4 acc) {
  return make_float4(fmaf(w.x, u.x, acc.x), fmaf(w.y, u.y, acc.y), fmaf(w.z, u.z, acc.z), fmaf(w.w, u.w, acc.w));
}
__device__ __forceinline__ void store4(float* dst, float4 v) { *reinterpret_cast<float4*>(dst) = v; }
__device__ __forceinline__ void store4(bf16* dst, float4 v) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  uint2 packed;
  packed.x = *reinterpret_cast<const uint32_t*>(&lo);
  packed.y = *reinterpret_cast<const uint32_t*>(&hi);
  *reinterpret_cast<uint2*>(dst) = packed;
}

// ONE: the projection left one buffer (long steps), nothing is folded.
template <class T, int TAPS, bool ONE>
__global__ void __launch_bounds__(128) conv_qkv_run_kernel(ConvParams p, int L) {
  constexpr int HALO = TAPS - 1;
  sb::grid_launch_dependents();
  const int lane = threadIdx.x & (L - 1), units = p.Hq + 2 * p.Hkv;
  const int unit = min(static_cast<int>(blockIdx.y) * (128 / L) + static_cast<int>(threadIdx.x) / L, units - 1);     // (surplus lanes repeat the
  const bool real = static_cast<int>(blockIdx.y) * (128 / L) + static_cast<int>(threadIdx.x) / L < units;            //  last unit, storing nothing)
  const bool is_q = unit < p.Hq, is_v = unit >= p.Hq + p.Hkv;
  const int head = is_q ? unit : is_v ? unit - p.Hq - p.Hkv : unit - p.Hq;
  const int nq = p.Hq * p.D, nk = p.Hkv * p.D, C = nq + nk + p.Hkv * p.Dv;
  const int dim = is_v ? p.Dv : p.D, d = lane * 4;
  const bool mine = d < dim, stores = mine && real;
  const int c = (is_q ? head * p.D : is_v ? nq + nk + head * p.Dv : nq + head * p.D) + (mine ? d : 0);
  int e = 0, run = blockIdx.x, len = 1;
  if (p.tile == 1) {
    e = run, run = 0;
  } else {
    for (; e < p.entries; ++e) {
      len = p.meta[2 * p.meta_stride + e];
      const int runs = (len + kRun - 1) / kRun;
      if (run < runs) break;
      run -= runs;
    }
  }
  if (e >= p.entries) return;
  const int slot = p.meta[e], row0 = p.meta[p.meta_stride + e], pos0 = p.meta[3 * p.meta_stride + e];
  const int t0 = run * kRun, nt = min(kRun, len - t0);
  const int rh = p.rot / 2;
  const bool turned = !is_v && d < p.rot, low = d < rh;
  const int partner = turned ? (low ? lane + rh / 4 : lane - rh / 4) : lane, pair = low ? d : d - rh;
  const float4 zero = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  float4 w[TAPS], u[TAPS];                          // u: the inputs of the token and of those in front of it, oldest first
#pragma unroll
  for (int j = 0; j < TAPS; ++j) w[j] = *reinterpret_cast<const float4*>(p.conv + static_cast<int64_t>(j) * C + c);
  float* record = p.record + static_cast<int64_t>(slot) * p.record_size + c;
  const float* src = p.proj + static_cast<int64_t>(row0) * p.width + c;
  sb::grid_dependency_wait();
  auto input = [&](int t) {
    const float* at = src + static_cast<int64_t>(t) * p.width;
    return ONE ? *reinterpret_cast<const float4*>(at) : folded4(at, p.n_partials, p.partial_stride);
  };
  float4 last[HALO];                                // the inputs in front of the run
#pragma unroll
  for (int j = 0; j < HALO; ++j) {
    const int t = t0 - HALO + j;
    last[j] = t >= 0 ? input(t) : pos0 + t >= 0 ? *reinterpret_cast<const float4*>(record + static_cast<int64_t>(HALO + t) * C) : zero;
  }
  float4 first_inputs[HALO];
#pragma unroll
  for (int j = 0; j < HALO; ++j) first_inputs[j] = u[j + 1] = last[j];
  constexpr int kAhead = ONE ? 4 : 1;               // tokens whose inputs are requested together
  for (int t1 = 0; t1 < nt; t1 += kAhead) {
    float4 next[kAhead];
#pragma unroll
    for (int i = 0; i < kAhead; ++i)
      if (t1 + i < nt) next[i] = input(t0 + t1 + i);
#pragma unroll
    for (int i = 0; i < kAhead; ++i) {
      if (t1 + i >= nt) break;
      const int row = row0 + t0 + t1 + i, pos = pos0 + t0 + t1 + i;
#pragma unroll
      for (int j = 0; j < HALO; ++j) u[j] = u[j + 1];
      u[HALO] = next[i];
      float4 y = zero;
#pragma unroll
      for (int j = 0; j < TAPS; ++j) y = fma4(w[j], u[j], y);
      if (!mine) y = zero;
      // (the lanes of v and of elements that are not turned take part in the exchange and leave its result)
      const float4 b = make_float4(__shfl_sync(0xffffffffu, y.x, partner, L), __shfl_sync(0xffffffffu, y.y, partner, L),
                                   __shfl_sync(0xffffffffu, y.z, partner, L), __shfl_sync(0xffffffffu, y.w, partner, L));
      if (turned) {
        const float4* cs = reinterpret_cast<const float4*>(p.cos_sin + (static_cast<int64_t>(pos) * rh + pair) * 2);
        const float4 c01 = cs[0], c23 = cs[1];       // cos, sin of pairs 0 and 1; of pairs 2 and 3
        auto turn = [&](float a, float o, float cs_, float sn) {
          return low ? __fsub_rn(__fmul_rn(a, cs_), __fmul_rn(o, sn)) : __fadd_rn(__fmul_rn(a, cs_), __fmul_rn(o, sn));
        };
        y = make_float4(turn(y.x, b.x, c01.x, c01.y), turn(y.y, b.y, c01.z, c01.w), turn(y.z, b.z, c23.x, c23.y), turn(y.w, b.w, c23.z, c23.w));
      }
      if (p.unit) {
        float ss = fmaf(y.w, y.w, fmaf(y.z, y.z, fmaf(y.y, y.y, __fmul_rn(y.x, y.x))));
        for (int o = L / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o, L);
        const float scale = is_v ? 1.0f : 1.0f / sqrtf(ss / static_cast<float>(dim) + p.eps);
        y = make_float4(__fmul_rn(y.x, scale), __fmul_rn(y.y, scale), __fmul_rn(y.z, scale), __fmul_rn(y.w, scale));
      }
      if (!stores) continue;
      if (is_q) {
        store4(static_cast<T*>(p.q_out) + static_cast<int64_t>(row) * nq + c, y);
        continue;
      }
      if (is_v && p.mix != kOwn) {
        float* kept = p.kept + static_cast<int64_t>(row) * p.Hkv * p.Dv + head * p.Dv + d;
        if (p.mix == kKeep) {
          store4(kept, y);
        } else {
          const float4 k = *reinterpret_cast<const float4*>(kept);
          y = make_float4(fmaf(p.lambda, k.x, __fmul_rn(p.rest, y.x)), fmaf(p.lambda, k.y, __fmul_rn(p.rest, y.y)),
                          fmaf(p.lambda, k.z, __fmul_rn(p.rest, y.z)), fmaf(p.lambda, k.w, __fmul_rn(p.rest, y.w)));
        }
      }
      const int page = p.block_table[static_cast<int64_t>(slot) * p.max_pages + pos / p.page_size];
      store4(static_cast<T*>(p.pages) + static_cast<int64_t>(page) * p.page_stride + (is_v ? p.v_offset : 0) + static_cast<int64_t>(head) * p.head_stride +
                 static_cast<int64_t>(pos % p.page_size) * p.Dc + d, y);
    }
  }
  if (t0 != 0 || !stores) return;
#pragma unroll
  for (int j = 0; j < HALO; ++j) {                  // the record behind the step: its row j is the entry's token len - HALO + j
    const int t = len - HALO + j;
    float4 v = zero;
    if (t >= 0) {
      v = input(t);
    } else {                                        // (a step shorter than the record: t = -1 is the newest of the inputs in front of it)
#pragma unroll
      for (int k = 0; k < HALO; ++k)
        if (k == HALO + t) v = first_inputs[k];
    }
    *reinterpret_cast<float4*>(record + static_cast<int64_t>(j) * C) = v;
  }
}

template <class T>
void launch_run(const ConvParams& p, int n, int L, cudaStream_t stream) {
  const int groups = 128 / L, units = p.Hq + 2 * p.Hkv;
  const dim3 grid(p.tile == 1 ? p.entries : (n + kRun - 1) / kRun + p.entries, (units + groups - 1) / groups);
#define SB_RUN(N)                                                                                                   \
  do {                                                                                                              \
    if (p.n_partials == 1) sb::launch_pdl(conv_qkv_run_kernel<T, N, true>, grid, dim3(128), 0, stream, p, L);       \
    else sb::launch_pdl(conv_qkv_run_kernel<T, N, false>, grid, dim3(128), 0, stream, p, L);                        \
  } while (0)
  if (p.taps == 4) SB_RUN(4);
  else if (p.taps == 3) SB_RUN(3);
  else SB_RUN(2);
#undef SB_RUN
}

}  // namespace

// i: 0 projection partial sums (flat), 1 their width, 2 K ranges S, 3 most tokens with a buffer per range, 4 the taps [taps][C] (0: no
//    convolution), 5 taps, 6 records, 7 elements of a record, 8 cos_sin, 9 rot, 10 heads divided by their root mean square, 11 the step's kept
//    values (or 0), 12 values: 0 as they are, 1 kept, 2 mixed, 13 q out, 14 dtype (q out and cache), 15 pages, 16 block table, 17 max_pages,
//    18 page_size, 19 page_stride, 20 v_offset, 21 head_stride, 22 Hq, 23 Hkv, 24 D, 25 Dv, 26 Dc
// f: 0 eps, 1 lambda
SB_EXPORT int sb_op_conv_qkv(const SbOp* op, const SbStep* s, void* stream) {
  using namespace sbstep;
  const int n = s->n;
  if (n <= 0 || s->entries <= 0) return SB_OP_SKIPPED;
  ConvParams p{};
  p.proj = ptr<const float>(op->i[0]), p.width = (int)op->i[1], p.n_partials = partial_count(op->i[2], op->i[3], n);
  p.partial_stride = static_cast<int64_t>(n) * p.width;
  p.conv = ptr<const float>(op->i[4]), p.taps = p.conv != nullptr ? (int)op->i[5] : 1;
  p.record = ptr<float>(op->i[6]), p.record_size = op->i[7];
  p.meta = entry_meta(s), p.meta_stride = s->max_rows, p.entries = s->entries, p.tile = n == s->entries ? 1 : kTile;
  p.cos_sin = ptr<const float>(op->i[8]), p.rot = (int)op->i[9], p.unit = (int)op->i[10], p.eps = (float)op->f[0];
  p.kept = ptr<float>(op->i[11]), p.mix = (int)op->i[12], p.lambda = (float)op->f[1], p.rest = (float)(1.0 - op->f[1]);
  p.q_out = ptr<void>(op->i[13]);
  const int dtype = (int)op->i[14];
  p.pages = ptr<void>(op->i[15]), p.block_table = ptr<const int32_t>(op->i[16]), p.max_pages = (int)op->i[17], p.page_size = (int)op->i[18];
  p.page_stride = op->i[19], p.v_offset = op->i[20], p.head_stride = op->i[21], p.Dc = (int)op->i[26];
  p.Hq = (int)op->i[22], p.Hkv = (int)op->i[23], p.D = (int)op->i[24], p.Dv = (int)op->i[25];
  const int64_t C = static_cast<int64_t>(p.Hq) * p.D + static_cast<int64_t>(p.Hkv) * (p.D + p.Dv);
  if (p.Hq <= 0 || p.Hkv <= 0 || p.D <= 0 || p.Dv <= 0 || C > p.width || p.Dc < p.D || p.Dc < p.Dv)
    return sb::fail("sb_op_conv_qkv: heads %d / %d, sizes %d / %d, rows of %d and %d", p.Hq, p.Hkv, p.D, p.Dv, p.width, p.Dc), SB_OP_FAILED;
  if (p.rot < 0 || p.rot % 2 != 0 || p.rot > p.D) return sb::fail("sb_op_conv_qkv: %d rotated elements of %d", p.rot, p.D), SB_OP_FAILED;
  if (p.taps < 1 || p.taps > kMaxTaps) return sb::fail("sb_op_conv_qkv: %d taps (1 to %d)", p.taps, kMaxTaps), SB_OP_FAILED;
  if (p.taps > 1 && (p.record == nullptr || p.record_size < (p.taps - 1) * C))
    return sb::fail("sb_op_conv_qkv: a record of %lld elements does not hold %d x %lld", (long long)p.record_size, p.taps - 1, (long long)C), SB_OP_FAILED;
  if (p.mix < kOwn || p.mix > kMix || (p.mix != kOwn && p.kept == nullptr)) return sb::fail("sb_op_conv_qkv: value mixing %d", p.mix), SB_OP_FAILED;
  const int dim = p.D > p.Dv ? p.D : p.Dv;
  const size_t smem = sizeof(float) * static_cast<size_t>(dim) * (p.taps + (p.taps - 1 + p.tile) + p.tile);
  if (smem > 200 * 1024) return sb::fail("sb_op_conv_qkv: heads of %d elements do not fit shared memory", dim), SB_OP_FAILED;
  const bool vec = p.D % 4 == 0 && p.Dv % 4 == 0 && p.width % 4 == 0 && p.record_size % 4 == 0 && ((op->i[0] | op->i[6]) & 15) == 0;
  if (dtype != 0 && dtype != 1) return sb::fail("sb_op_conv_qkv: unsupported dtype %d", dtype), SB_OP_FAILED;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  // (which form runs depends on the sizes and the buffers alone, never on the rows of the step)
  if (vec && p.taps >= 2 && p.taps <= 4 && dim <= 128 && p.rot % 8 == 0 && p.Dc % 4 == 0 && p.page_stride % 4 == 0 && p.v_offset % 4 == 0 &&
      p.head_stride % 4 == 0 && ((op->i[4] | op->i[8] | op->i[11] | op->i[13] | op->i[15]) & 15) == 0) {
    int L = 1;
    while (L * 4 < dim) L *= 2;
    if (dtype == 0) launch_run<float>(p, n, L, st);
    else launch_run<bf16>(p, n, L, st);
    return sb::check_launch("sb_op_conv_qkv");
  }
  const dim3 grid(p.tile == 1 ? p.entries : (n + kTile - 1) / kTile + p.entries, p.Hq + 2 * p.Hkv), block(p.tile == 1 ? 64 : 128);
#define SB_CONV(T, V)                                                                                                            \
  do {                                                                                                                           \
    if (smem > 48 * 1024) cudaFuncSetAttribute(conv_qkv_kernel<T, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);   \
    sb::launch_pdl(conv_qkv_kernel<T, V>, grid, block, smem, st, p);                                                             \
  } while (0)
  if (dtype == 0 && vec) SB_CONV(float, true);
  else if (dtype == 0) SB_CONV(float, false);
  else if (vec) SB_CONV(bf16, true);
  else SB_CONV(bf16, false);
#undef SB_CONV
  return sb::check_launch("sb_op_conv_qkv");
}
