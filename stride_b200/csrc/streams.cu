// Several residual streams side by side. A sublayer reads one weighted sum of the streams and every stream takes a weighted sum of
// all of them plus its share of the sublayer's result:
//
//   u[r, :]    = sum_s in[s] x[r, s, :];        y = sublayer(norm(u))
//   x'[r, t, :] = sum_s mix[s, t] x[r, s, :] + out[t] y[r, :]            every x' from the old x
//
// `streams_step_kernel` is what stands between two sublayers, in one pass over the streams: it takes the result of the sublayer before
// into them (x'), stores them, forms the next sublayer's u from the new values, norms it (a layer norm or an RMS norm) and stores it in the
// activations' type. y arrives as it was left: up to two sources, each a buffer and / or the partial sums of a projection's K ranges, times
// a constant. In front of the first sublayer all streams are the embedding output: the kernel then reads one row for all of them (stream
// stride 0). Behind the last one it runs on the rows whose logits are wanted alone, with in = 1 for every stream (their sum) and stores no
// streams. All in 32-bit, in a fixed order: a row's result does not depend on the other rows of the step.
#include "common.cuh"
#include "step_ops.h"

SB_DEFINE_LAST_ERROR()

namespace {

using bf16 = __nv_bfloat16;
constexpr int kInFlight = 4;
constexpr int kMaxStreams = 16;

struct Source {
  const float* buffer;      // [n][W] or null
  const float* partials;    // [P][n][W] or null
  int n_partials;
  float c;
};

struct StepParams {
  const float* x;           // stream s of row r: x + r row_stride + s stream_stride
  int64_t row_stride, stream_stride;
  float* x_new;             // [n][S][W] (may be x itself), or null: the new streams are not stored
  Source a, b;              // the result of the sublayer before; both empty: the streams stay as they are
  int64_t partial_stride;   // n W
  const float* mix;         // [S][S], from the first index to the second
  const float* out;         // [S]
  const float* in;          // [S], or null: 1 for every stream
  const float* gain;        // [W]
  const float* bias;        // [W] or null
  float eps;
  int centred;              // 1: layer norm, 0: RMS norm
  const int32_t* rows;      // null, or which row of the streams row i of `normed` is made of
  void* normed;             // [rows][W]
  int S, W;
};

__device__ __forceinline__ float mad(float c, float a, float b) { return fmaf(c, a, b); }
__device__ __forceinline__ float4 mad(float c, float4 a, float4 b) { return make_float4(fmaf(c, a.x, b.x), fmaf(c, a.y, b.y), fmaf(c, a.z, b.z), fmaf(c, a.w, b.w)); }
__device__ __forceinline__ float times(float a, float c) { return __fmul_rn(a, c); }
__device__ __forceinline__ float4 times(float4 a, float c) { return make_float4(__fmul_rn(a.x, c), __fmul_rn(a.y, c), __fmul_rn(a.z, c), __fmul_rn(a.w, c)); }
__device__ __forceinline__ float plus(float a, float b) { return __fadd_rn(a, b); }
__device__ __forceinline__ float4 plus(float4 a, float4 b) { return make_float4(__fadd_rn(a.x, b.x), __fadd_rn(a.y, b.y), __fadd_rn(a.z, b.z), __fadd_rn(a.w, b.w)); }
__device__ __forceinline__ float total_of(float v) { return v; }
__device__ __forceinline__ float total_of(float4 v) { return ((v.x + v.y) + v.z) + v.w; }

// buffer + (p0 + p1 + ..), times the source's constant; up to kInFlight partial sums requested at once.
template <class V>
__device__ __forceinline__ V source_value(const Source& s, int64_t partial_stride, int64_t i) {      // i and the stride in units of V
  V v = {};
  if (s.partials != nullptr) {
    const V* p = reinterpret_cast<const V*>(s.partials) + i;
    v = p[0];
    for (int k0 = 1; k0 < s.n_partials; k0 += kInFlight) {
      V part[kInFlight];
#pragma unroll
      for (int k = 0; k < kInFlight; ++k)
        if (k0 + k < s.n_partials) part[k] = p[(k0 + k) * partial_stride];
#pragma unroll
      for (int k = 0; k < kInFlight; ++k)
        if (k0 + k < s.n_partials) v = plus(v, part[k]);
    }
    if (s.buffer != nullptr) v = plus(reinterpret_cast<const V*>(s.buffer)[i], v);
  } else if (s.buffer != nullptr) {
    v = reinterpret_cast<const V*>(s.buffer)[i];
  }
  return times(v, s.c);
}

template <class TO>
__device__ __forceinline__ void store(TO* dst, float v) { *dst = sb::narrow<TO>(v); }
__device__ __forceinline__ void store(float* dst, float4 v) { *reinterpret_cast<float4*>(dst) = v; }
__device__ __forceinline__ void store(bf16* dst, float4 v) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  uint2 packed;
  packed.x = *reinterpret_cast<const uint32_t*>(&lo);
  packed.y = *reinterpret_cast<const uint32_t*>(&hi);
  *reinterpret_cast<uint2*>(dst) = packed;
}

// A block per row; u stays in shared memory between the norm's sums. SM: the most streams (EXACT: their number). V: float4 where the width
// is a multiple of four and every buffer 16-byte aligned, else float: which one depends on the width and the buffers, never on the rows.
template <class TO, class V, int SM, bool EXACT>
__global__ void __launch_bounds__(256, SM <= 4 ? 3 : 1) streams_step_kernel(StepParams p) {
  extern __shared__ __align__(16) float row_values[];
  __shared__ float red[32];
  __shared__ float coef[kMaxStreams * (kMaxStreams + 2)];       // mix | out | in
  constexpr int VE = sizeof(V) / sizeof(float);
  sb::grid_launch_dependents();
  const int S = EXACT ? SM : p.S, W = p.W, units = W / VE;
  const bool update = p.a.buffer != nullptr || p.a.partials != nullptr;
  const bool two = p.b.buffer != nullptr || p.b.partials != nullptr;
  for (int i = threadIdx.x; i < S * (S + 2); i += blockDim.x)
    coef[i] = i >= S * S + S ? (p.in != nullptr ? p.in[i - S * S - S] : 1.0f) : !update ? 0.0f : i < S * S ? p.mix[i] : p.out[i - S * S];
  __syncthreads();
  sb::grid_dependency_wait();
  const int64_t row = p.rows != nullptr ? p.rows[blockIdx.x] : static_cast<int>(blockIdx.x);
  const V* x = reinterpret_cast<const V*>(p.x + row * p.row_stride);
  V* x_new = reinterpret_cast<V*>(p.x_new + row * static_cast<int64_t>(S) * W);
  const int64_t xs = p.stream_stride / VE, ps = p.partial_stride / VE;
  V* held = reinterpret_cast<V*>(row_values);
  const float* mix = coef;
  const float* out = coef + S * S;
  const float* in = out + S;
  float sum = 0.0f;
  for (int c = threadIdx.x; c < units; c += blockDim.x) {
    V v[SM];
#pragma unroll
    for (int s = 0; s < SM; ++s)
      if (EXACT || s < S) v[s] = x[s * xs + c];
    V u = {};
    if (update) {
      V y = source_value<V>(p.a, ps, row * units + c);
      if (two) y = plus(y, source_value<V>(p.b, ps, row * units + c));
#pragma unroll
      for (int t = 0; t < SM; ++t)
        if (EXACT || t < S) {
          V n = times(y, out[t]);
#pragma unroll
          for (int s = 0; s < SM; ++s)
            if (EXACT || s < S) n = mad(mix[s * S + t], v[s], n);
          if (p.x_new != nullptr) x_new[static_cast<int64_t>(t) * units + c] = n;
          u = mad(in[t], n, u);
        }
    } else {
#pragma unroll
      for (int s = 0; s < SM; ++s)
        if (EXACT || s < S) u = mad(in[s], v[s], u);
    }
    held[c] = u;
    if (p.centred) {
      sum += total_of(u);
    } else if constexpr (VE == 4) {
      sum = fmaf(u.x, u.x, sum), sum = fmaf(u.y, u.y, sum), sum = fmaf(u.z, u.z, sum), sum = fmaf(u.w, u.w, sum);
    } else {
      sum = fmaf(u, u, sum);
    }
  }
  float mean = 0.0f, sq = sb::block_sum(sum, red);
  if (p.centred) {
    mean = sq / static_cast<float>(W);
    float d2 = 0.0f;
    for (int c = threadIdx.x; c < units; c += blockDim.x) {       // (a thread reads back what it wrote)
      const V u = held[c];
      if constexpr (VE == 4) {
        const float dx = u.x - mean, dy = u.y - mean, dz = u.z - mean, dw = u.w - mean;
        d2 = fmaf(dx, dx, d2), d2 = fmaf(dy, dy, d2), d2 = fmaf(dz, dz, d2), d2 = fmaf(dw, dw, d2);
      } else {
        d2 = fmaf(u - mean, u - mean, d2);
      }
    }
    sq = sb::block_sum(d2, red);
  }
  const float scale = 1.0f / sqrtf(sq / static_cast<float>(W) + p.eps);
  TO* o = static_cast<TO*>(p.normed) + static_cast<int64_t>(blockIdx.x) * W;
  for (int c = threadIdx.x; c < units; c += blockDim.x) {
    const V u = held[c], g = reinterpret_cast<const V*>(p.gain)[c];
    V b = {};
    if (p.bias != nullptr) b = reinterpret_cast<const V*>(p.bias)[c];
    if constexpr (VE == 4)
      store(o + 4 * c, make_float4(fmaf((u.x - mean) * scale, g.x, b.x), fmaf((u.y - mean) * scale, g.y, b.y),
                                   fmaf((u.z - mean) * scale, g.z, b.z), fmaf((u.w - mean) * scale, g.w, b.w)));
    else
      store(o + c, fmaf((u - mean) * scale, g, b));
  }
}

inline bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

template <class TO>
int launch(const StepParams& p, int rows, bool vec, cudaStream_t stream) {
  const size_t smem = static_cast<size_t>(p.W) * sizeof(float);
  vec = vec && p.S <= 4;        // (more streams: one element of each a thread, or the registers do not hold them)
  const int units = vec ? p.W / 4 : p.W;
  const int threads = units >= 256 ? 256 : 128;
#define SB_STREAMS(V, SM, EXACT)                                                                                                          \
  do {                                                                                                                                    \
    if (smem > 40 * 1024) cudaFuncSetAttribute(streams_step_kernel<TO, V, SM, EXACT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    sb::launch_pdl(streams_step_kernel<TO, V, SM, EXACT>, dim3(rows), dim3(threads), smem, stream, p);                                    \
  } while (0)
#define SB_STREAMS_V(SM, EXACT)            \
  do {                                     \
    if (vec) SB_STREAMS(float4, SM, EXACT); \
    else SB_STREAMS(float, SM, EXACT);     \
  } while (0)
  switch (p.S) {
    case 1: SB_STREAMS_V(1, true); break;
    case 2: SB_STREAMS_V(2, true); break;
    case 3: SB_STREAMS_V(3, true); break;
    case 4: SB_STREAMS_V(4, true); break;
    default:
      if (p.S <= 8) SB_STREAMS(float, 8, false);
      else SB_STREAMS(float, kMaxStreams, false);
  }
#undef SB_STREAMS_V
#undef SB_STREAMS
  return sb::check_launch("sb_op_streams_step");
}

}  // namespace

// i: 0 streams read, 1 their row stride, 2 their stream stride, 3 streams written (or 0),
//    4 first source: buffer (or 0), 5 partial sums (flat, or 0), 6 K ranges S, 7 most tokens with a buffer per range,
//    8 second source: buffer, 9 partial sums, 10 S, 11 most tokens,
//    12 mix, 13 out, 14 in (or 0: ones), 15 gain, 16 bias (or 0), 17 layer norm (1) or RMS norm (0), 18 normed, 19 its dtype, 20 streams, 21 W,
//    22 rows: 0 = the step's tokens, 1 = the rows whose logits are wanted
// f: 0 the first source's constant, 1 the second's, 2 eps
SB_EXPORT int sb_op_streams_step(const SbOp* op, const SbStep* s, void* stream) {
  using namespace sbstep;
  const int n = s->n, rows = op->i[22] ? s->wanted : n;
  if (rows <= 0) return SB_OP_SKIPPED;
  const int S = (int)op->i[20], W = (int)op->i[21];
  if (S < 1 || S > kMaxStreams || W <= 0) return sb::fail("sb_op_streams_step: %d streams (1 to %d) of %d elements", S, kMaxStreams, W), SB_OP_FAILED;
  if (static_cast<size_t>(W) * sizeof(float) > 200 * 1024) return sb::fail("sb_op_streams_step: width %d does not fit the row buffer (max 51200)", W), SB_OP_FAILED;
  auto source = [&](int at, float c) {
    const float* partials = ptr<const float>(op->i[at + 1]);
    return Source{ptr<const float>(op->i[at]), partials, partials ? partial_count(op->i[at + 2], op->i[at + 3], n) : 0, c};
  };
  StepParams p{ptr<const float>(op->i[0]), op->i[1], op->i[2], ptr<float>(op->i[3]), source(4, static_cast<float>(op->f[0])),
               source(8, static_cast<float>(op->f[1])), static_cast<int64_t>(n) * W, ptr<const float>(op->i[12]), ptr<const float>(op->i[13]),
               ptr<const float>(op->i[14]), ptr<const float>(op->i[15]), ptr<const float>(op->i[16]), static_cast<float>(op->f[2]), (int)op->i[17],
               op->i[22] ? wanted_rows(s) : nullptr, ptr<void>(op->i[18]), S, W};
  const bool vec = W % 4 == 0 && p.row_stride % 4 == 0 && p.stream_stride % 4 == 0 && aligned16(p.x) && aligned16(p.x_new) && aligned16(p.a.buffer) &&
                   aligned16(p.a.partials) && aligned16(p.b.buffer) && aligned16(p.b.partials) && aligned16(p.gain) && aligned16(p.bias) &&
                   aligned16(p.normed);
  if (op->i[19] == 0) return launch<float>(p, rows, vec, static_cast<cudaStream_t>(stream));
  if (op->i[19] == 1) return launch<bf16>(p, rows, vec, static_cast<cudaStream_t>(stream));
  return sb::fail("sb_op_streams_step: unsupported dtype %d", (int)op->i[19]), SB_OP_FAILED;
}
