// Everything that two sublayers side by side leave for the residual stream, added in one pass, with the norm that reads the new sum:
//
//     x    = x + (a [+ bias]) + (sum_k share[t, k] * y[slot_of[t, k]] + same_share[t] * same[t])
//     out  = x / sqrt(mean(x^2) + eps) * weight       (in the compute dtype)
//
// all in float32.  a: the mixer's output, [T, width] in the compute dtype or float32 partial sums [parts, T, width] whose sum it is, and a
// float32 bias [width].  y: the feed-forward's, in either form, row t for token t; or, with slot_of, rows of experts in slots, token t's the
// rows slot_of[t * top + k] (-1: none), each times share[t * top + k] where shares are given.  same: rows in the compute dtype that experts
// hand back as they are, each times same_share[t].  Every one of them may be missing, and so may the norm.  With `rows` only those tokens
// are normed and x stays as it is: what is added to it is added on the fly.
//
// A block takes one token; a thread keeps its columns between the sum of squares and the result.
#include "common.cuh"

namespace pylon {

struct JoinParams {
  float* x;
  const void* a;
  int a_parts;              // 0: in T; > 0: float32 partial sums
  long long a_stride;       // elements between the parts
  const float* bias;
  const void* y;
  int y_parts;
  long long y_stride;
  const int* slot_of;
  const float* share;
  int top;
  const void* same;
  long long same_ld;
  const float* same_share;
  const float* weight;      // null: no norm
  const int* rows;
  void* out;
  int width;
  float eps;
};

__device__ __forceinline__ void add_4(float4& sum, const float4& more) { sum.x += more.x; sum.y += more.y; sum.z += more.z; sum.w += more.w; }
__device__ __forceinline__ void add_4_times(float4& sum, float factor, const float4& more) {
  sum.x = fmaf(factor, more.x, sum.x); sum.y = fmaf(factor, more.y, sum.y); sum.z = fmaf(factor, more.z, sum.z); sum.w = fmaf(factor, more.w, sum.w);
}
template <typename T>
__device__ __forceinline__ float4 four(const void* from, long long at) {
  if constexpr (sizeof(T) == 4) return *reinterpret_cast<const float4*>((const float*)from + at);
  else {
    const uint2 raw = *reinterpret_cast<const uint2*>((const __nv_bfloat16*)from + at);
    const float2 low = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x)), high = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    return make_float4(low.x, low.y, high.x, high.y);
  }
}
// Four columns of a block in either form.
template <typename T>
__device__ __forceinline__ float4 four_of(const void* from, int parts, long long stride, long long at) {
  if (parts == 0) return four<T>(from, at);
  float4 sum = four<float>(from, at);
  if (parts == 1) return sum;
  for (int first = 1; first < parts; first += 3) {   // three parts' loads on their way at once
    float4 part[3];
#pragma unroll
    for (int k = 0; k < 3; ++k) part[k] = four<float>(from, (first + k < parts ? first + k : first) * stride + at);
#pragma unroll
    for (int k = 0; k < 3; ++k)
      if (first + k < parts) add_4(sum, part[k]);
  }
  return sum;
}

// HELD: the 4-column pieces a thread keeps.
template <typename T, int HELD>
__global__ void __launch_bounds__(512, HELD > 2 ? 1 : 2) join_norm_vec_kernel(const JoinParams p) {
  __shared__ float scratch[34];
  const int pieces = p.width / 4;
  float4 w[HELD];   // weights and bias are nobody's work: on their way before the wait for the kernel ahead
#pragma unroll
  for (int i = 0; i < HELD; ++i) {
    const int piece = threadIdx.x + i * blockDim.x;
    w[i] = p.weight && piece < pieces ? four<float>(p.weight, 4 * piece) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  float4 mixer[HELD];
#pragma unroll
  for (int i = 0; i < HELD; ++i) {
    const int piece = threadIdx.x + i * blockDim.x;
    mixer[i] = p.bias && piece < pieces ? four<float>(p.bias, 4 * piece) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  grid_dependency_wait();
  allow_dependents();
  const long long t = p.rows ? p.rows[blockIdx.x] : blockIdx.x;
  // Where the token's first rows lie, asked for before all else: the loads of the rows wait for nothing but these.
  constexpr int SIDE = 4 / HELD;   // rows of a token on their way at once: more of them cost more in registers than they gain
  int slot[SIDE];
  float share[SIDE];
  auto find = [&](int first) {
#pragma unroll
    for (int j = 0; j < SIDE; ++j) {
      slot[j] = first + j < p.top ? p.slot_of[t * p.top + first + j] : -1;
      share[j] = first + j < p.top && p.share ? p.share[t * p.top + first + j] : 1.f;
    }
  };
  if (p.slot_of) find(0);
  float4 x[HELD], ff[HELD];
  const float same_share = p.same ? p.same_share[t] : 0.f;
#pragma unroll
  for (int i = 0; i < HELD; ++i) {
    const int piece = threadIdx.x + i * blockDim.x;
    x[i] = ff[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (piece >= pieces) continue;
    const long long at = t * p.width + 4 * piece;
    x[i] = *reinterpret_cast<const float4*>(p.x + at);
    if (p.a) add_4(mixer[i], four_of<T>(p.a, p.a_parts, p.a_stride, at));
    if (p.same && same_share != 0.f) add_4_times(ff[i], same_share, four<T>(p.same, t * p.same_ld + 4 * piece));
    if (p.y && !p.slot_of) add_4(ff[i], four_of<T>(p.y, p.y_parts, p.y_stride, at));
  }
  if (p.slot_of) {
    for (int first = 0; first < p.top; first += SIDE) {
      if (first > 0) find(first);
      const int parts = p.y_parts > 0 ? p.y_parts : 1;
      for (int part = 0; part < parts; ++part) {
        float4 row[HELD][SIDE];   // all of them on their way at once
#pragma unroll
        for (int i = 0; i < HELD; ++i) {
          const int piece = threadIdx.x + i * blockDim.x;
#pragma unroll
          for (int j = 0; j < SIDE; ++j) {
            row[i][j] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (slot[j] < 0 || piece >= pieces) continue;
            const long long at = (long long)slot[j] * p.width + 4 * piece;
            row[i][j] = p.y_parts > 0 ? four<float>(p.y, part * p.y_stride + at) : four<T>(p.y, at);
          }
        }
#pragma unroll
        for (int i = 0; i < HELD; ++i)
#pragma unroll
          for (int j = 0; j < SIDE; ++j) add_4_times(ff[i], share[j], row[i][j]);
      }
    }
  }
  float squares = 0.f;
#pragma unroll
  for (int i = 0; i < HELD; ++i) {
    add_4(mixer[i], ff[i]);
    add_4(x[i], mixer[i]);
    squares = fmaf(x[i].x, x[i].x, fmaf(x[i].y, x[i].y, fmaf(x[i].z, x[i].z, fmaf(x[i].w, x[i].w, squares))));
    const int piece = threadIdx.x + i * blockDim.x;
    if (!p.rows && piece < pieces) *reinterpret_cast<float4*>(p.x + t * p.width + 4 * piece) = x[i];
  }
  if (!p.weight) return;
  const float inv = 1.f / sqrtf(block_sum(squares, scratch) / p.width + p.eps);
#pragma unroll
  for (int i = 0; i < HELD; ++i) {
    const int piece = threadIdx.x + i * blockDim.x;
    if (piece >= pieces) continue;
    const float4 r = make_float4(x[i].x * inv * w[i].x, x[i].y * inv * w[i].y, x[i].z * inv * w[i].z, x[i].w * inv * w[i].w);
    const long long at = (long long)blockIdx.x * p.width + 4 * piece;
    if constexpr (sizeof(T) == 4) *reinterpret_cast<float4*>((float*)p.out + at) = r;
    else {
      __nv_bfloat162 low = __floats2bfloat162_rn(r.x, r.y), high = __floats2bfloat162_rn(r.z, r.w);
      *reinterpret_cast<uint2*>((__nv_bfloat16*)p.out + at) = make_uint2(*reinterpret_cast<unsigned*>(&low), *reinterpret_cast<unsigned*>(&high));
    }
  }
}

// Any width and alignment; the sum is formed a second time for the result where it was not written.
template <typename T>
__global__ void __launch_bounds__(256) join_norm_kernel(const JoinParams p) {
  __shared__ float scratch[34];
  grid_dependency_wait();
  allow_dependents();
  const long long t = p.rows ? p.rows[blockIdx.x] : blockIdx.x;
  auto value = [&](const void* from, int parts, long long stride, long long at) {
    if (parts == 0) return to_float<T>(((const T*)from)[at]);
    float sum = 0.f;
    for (int part = 0; part < parts; ++part) sum += ((const float*)from)[part * stride + at];
    return sum;
  };
  auto sum = [&](int c) {
    const long long at = t * p.width + c;
    float mixer = p.bias ? p.bias[c] : 0.f, ff = 0.f;
    if (p.a) mixer += value(p.a, p.a_parts, p.a_stride, at);
    if (p.same) ff = fmaf(p.same_share[t], to_float<T>(((const T*)p.same)[t * p.same_ld + c]), ff);
    if (p.y && !p.slot_of) ff += value(p.y, p.y_parts, p.y_stride, at);
    if (p.slot_of) {
      for (int k = 0; k < p.top; ++k) {
        const int slot = p.slot_of[t * p.top + k];
        if (slot >= 0) ff = fmaf(p.share ? p.share[t * p.top + k] : 1.f, value(p.y, p.y_parts, p.y_stride, (long long)slot * p.width + c), ff);
      }
    }
    return p.x[at] + (mixer + ff);
  };
  float squares = 0.f;
  for (int c = threadIdx.x; c < p.width; c += blockDim.x) {
    const float x = sum(c);
    if (!p.rows) p.x[t * p.width + c] = x;
    squares = fmaf(x, x, squares);
  }
  if (!p.weight) return;
  const float inv = 1.f / sqrtf(block_sum(squares, scratch) / p.width + p.eps);
  for (int c = threadIdx.x; c < p.width; c += blockDim.x)
    ((T*)p.out)[(long long)blockIdx.x * p.width + c] = from_float<T>((p.rows ? sum(c) : p.x[t * p.width + c]) * inv * p.weight[c]);
}

}  // namespace pylon

using namespace pylon;

// x float32 [tokens, width]; a [tokens, width] in dtype (a_parts 0) or float32 [a_parts, tokens, width], or null; bias float32 [width] or null; y
// likewise with y_rows rows (tokens, or with slot_of the slots) or null; slot_of int32 [tokens, top] or null; share float32 [tokens, top] or
// null; same [tokens, same_ld] in dtype with same_share float32 [tokens], or both null; weight float32 [width] with out [n_rows, width] in
// dtype, or both null; rows int32 [n_rows] or null (then n_rows is tokens).
extern "C" int pylon_join_norm(float* x, const void* a, int a_parts, const float* bias, const void* y, int y_parts, long long y_rows, const int* slot_of,
                               const float* share, int top, const void* same, long long same_ld, const float* same_share, const float* weight, const int* rows,
                               void* out, int n_rows, int tokens, int width, float eps, int dtype, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (width < 1 || a_parts < 0 || y_parts < 0 || (!rows && n_rows != tokens) || (weight != nullptr) != (out != nullptr) || (rows && !weight))
    PYLON_REFUSE("join_norm: width %d, %d and %d parts, %d of %d rows", width, a_parts, y_parts, n_rows, tokens);
  if ((slot_of && (!y || top < 1 || y_rows < 1)) || (share && !slot_of) || (same != nullptr) != (same_share != nullptr)) PYLON_REFUSE("join_norm: experts' rows without slots, or shares without rows");
  if (dtype != PYLON_DTYPE_F32 && dtype != PYLON_DTYPE_BF16) PYLON_REFUSE("join_norm: unknown dtype %d", dtype);
  const JoinParams p{x, a, a_parts, (long long)tokens * width, bias, y, y_parts, y_rows * width, slot_of, share, slot_of ? top : 1, same, same_ld, same_share, weight, rows, out, width, eps};
  // threads by the width alone, so that a token's sum does not depend on the step
  int threads = 64;
  while (threads < 512 && threads < width / 4) threads *= 2;
  const uintptr_t piece = dtype == PYLON_DTYPE_F32 ? 16 : 8;
  const bool pieces = width % 4 == 0 && same_ld % 4 == 0 && width / 4 <= threads * 4 && (uintptr_t)x % 16 == 0 && (uintptr_t)a % (a_parts ? 16 : piece) == 0 &&
                      (uintptr_t)y % (y_parts ? 16 : piece) == 0 && (uintptr_t)same % piece == 0 && (uintptr_t)out % piece == 0 && (uintptr_t)weight % 16 == 0 && (uintptr_t)bias % 16 == 0;
#define PYLON_JOIN_NORM(T)                                                                                                                        \
  if (pieces && width / 4 <= threads) launch_dependent(join_norm_vec_kernel<T, 1>, dim3((unsigned)n_rows), dim3(threads), 0, stream, p);          \
  else if (pieces && width / 4 <= threads * 2) launch_dependent(join_norm_vec_kernel<T, 2>, dim3((unsigned)n_rows), dim3(threads), 0, stream, p); \
  else if (pieces) launch_dependent(join_norm_vec_kernel<T, 4>, dim3((unsigned)n_rows), dim3(threads), 0, stream, p);                             \
  else launch_dependent(join_norm_kernel<T>, dim3((unsigned)n_rows), dim3(256), 0, stream, p)
  if (dtype == PYLON_DTYPE_F32) { PYLON_JOIN_NORM(float); } else { PYLON_JOIN_NORM(__nv_bfloat16); }
#undef PYLON_JOIN_NORM
  PYLON_CHECK_LAUNCH("join_norm");
}
