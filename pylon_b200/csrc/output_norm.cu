// The norm that stands on a sublayer's output, with what follows it: per token
//
//     n = y / sqrt(mean(y^2) + eps) * weight
//     x = x + n        (or x = n: the first of the stream)
//     copy = x in the compute dtype, what the next sublayer reads
//
// all in float32.  y comes as [T, width] in the compute dtype, as float32 partial sums [parts, T, width] whose sum it is, as rows of
// a table [vocab, width] times a factor, picked by ids (the embedding), or as rows that lie in slots (a mixture of experts): token t's
// output is the sum of the rows slot_of[t * top + k], k < top, each times share[t * top + k] where shares are given.  A block takes one token; a thread keeps its columns of y between
// the sum of squares and the result.
#include "common.cuh"

namespace pylon {

struct OutputNormParams {
  const void* y;
  int parts;                // 0: in T; > 0: float32 partial sums
  long long part_stride;    // elements between the parts
  const int* ids;           // null, or which row of y a token reads
  const int* slot_of;       // null, or the `top` rows a token's output is the sum of
  const float* share;       // [T, top] or null: factors on them
  int top;
  int vocab;
  float y_scale;
  float* x;
  void* copy;               // null: none (the compute dtype is float32: x itself serves)
  const float* weight;
  int width;
  float eps;
  int accumulate;
};

template <typename T>
__device__ __forceinline__ float4 output_norm_piece(const OutputNormParams& p, long long at) {
  if (p.parts > 0) {
    float4 sum = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int first = 0; first < p.parts; first += 4) {   // four parts' loads on their way at once
      float4 part[4];
#pragma unroll
      for (int k = 0; k < 4; ++k) part[k] = *reinterpret_cast<const float4*>((const float*)p.y + (first + k < p.parts ? first + k : first) * p.part_stride + at);
#pragma unroll
      for (int k = 0; k < 4; ++k)
        if (first + k < p.parts) { sum.x += part[k].x; sum.y += part[k].y; sum.z += part[k].z; sum.w += part[k].w; }
    }
    return sum;
  }
  if constexpr (sizeof(T) == 4) return *reinterpret_cast<const float4*>((const float*)p.y + at);
  else {
    const uint2 raw = *reinterpret_cast<const uint2*>((const __nv_bfloat16*)p.y + at);
    const float2 low = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x)), high = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    return make_float4(low.x, low.y, high.x, high.y);
  }
}

// Where the (k-th) row of a token's output starts.
__device__ __forceinline__ long long output_norm_row(const OutputNormParams& p, int t, int k) {
  if (p.slot_of) return (long long)p.slot_of[(long long)t * p.top + k] * p.width;
  if (!p.ids) return (long long)t * p.width;
  const int id = p.ids[t];
  return (long long)(id < 0 ? 0 : (id < p.vocab ? id : p.vocab - 1)) * p.width;
}

// HELD: the 4-column pieces a thread keeps.
template <typename T, int HELD>
__global__ void __launch_bounds__(1024) output_norm_vec_kernel(const OutputNormParams p) {
  __shared__ float scratch[34];
  const int t = blockIdx.x, pieces = p.width / 4;
  float4 w[HELD];   // the weights are nobody's work: on their way before the wait for the kernel ahead
#pragma unroll
  for (int i = 0; i < HELD; ++i) {
    const int piece = threadIdx.x + i * blockDim.x;
    if (piece < pieces) w[i] = *reinterpret_cast<const float4*>(p.weight + 4 * piece);
  }
  grid_dependency_wait();
  allow_dependents();
  const long long from = output_norm_row(p, t, 0);
  const float first_share = p.share ? p.share[(long long)t * p.top] : 1.f;
  float4 y[HELD], x[HELD];
  float squares = 0.f;
#pragma unroll
  for (int i = 0; i < HELD; ++i) {
    const int piece = threadIdx.x + i * blockDim.x;
    if (piece < pieces) {
      y[i] = output_norm_piece<T>(p, from + 4 * piece);
      if (p.accumulate) x[i] = *reinterpret_cast<const float4*>(p.x + (long long)t * p.width + 4 * piece);   // on its way while the squares are summed
      else x[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    } else y[i] = x[i] = make_float4(0.f, 0.f, 0.f, 0.f);
  }
#pragma unroll
  for (int i = 0; i < HELD; ++i) { y[i].x *= first_share; y[i].y *= first_share; y[i].z *= first_share; y[i].w *= first_share; }
  for (int k = 1; k < p.top; ++k) {
    const long long other = output_norm_row(p, t, k);
    const float share = p.share ? p.share[(long long)t * p.top + k] : 1.f;
#pragma unroll
    for (int i = 0; i < HELD; ++i) {
      const int piece = threadIdx.x + i * blockDim.x;
      if (piece >= pieces) continue;
      const float4 more = output_norm_piece<T>(p, other + 4 * piece);
      y[i].x = fmaf(share, more.x, y[i].x); y[i].y = fmaf(share, more.y, y[i].y); y[i].z = fmaf(share, more.z, y[i].z); y[i].w = fmaf(share, more.w, y[i].w);
    }
  }
#pragma unroll
  for (int i = 0; i < HELD; ++i) {
    y[i].x *= p.y_scale; y[i].y *= p.y_scale; y[i].z *= p.y_scale; y[i].w *= p.y_scale;
    squares = fmaf(y[i].x, y[i].x, fmaf(y[i].y, y[i].y, fmaf(y[i].z, y[i].z, fmaf(y[i].w, y[i].w, squares))));
  }
  const float inv = 1.f / sqrtf(block_sum(squares, scratch) / p.width + p.eps);
#pragma unroll
  for (int i = 0; i < HELD; ++i) {
    const int piece = threadIdx.x + i * blockDim.x;
    if (piece >= pieces) continue;
    const float4 r = make_float4(fmaf(y[i].x * inv, w[i].x, x[i].x), fmaf(y[i].y * inv, w[i].y, x[i].y), fmaf(y[i].z * inv, w[i].z, x[i].z), fmaf(y[i].w * inv, w[i].w, x[i].w));
    const long long at = (long long)t * p.width + 4 * piece;
    *reinterpret_cast<float4*>(p.x + at) = r;
    if (p.copy) {
      __nv_bfloat162 low = __floats2bfloat162_rn(r.x, r.y), high = __floats2bfloat162_rn(r.z, r.w);
      *reinterpret_cast<uint2*>((__nv_bfloat16*)p.copy + at) = make_uint2(*reinterpret_cast<unsigned*>(&low), *reinterpret_cast<unsigned*>(&high));
    }
  }
}

// Any width and alignment: y is read twice.
template <typename T>
__global__ void output_norm_kernel(const OutputNormParams p) {
  __shared__ float scratch[34];
  const int t = blockIdx.x;
  grid_dependency_wait();
  allow_dependents();
  auto value = [&](int c) {
    float total = 0.f;
    for (int k = 0; k < p.top; ++k) {
      const long long from = output_norm_row(p, t, k);
      float v = 0.f;
      if (p.parts > 0) { for (int part = 0; part < p.parts; ++part) v += ((const float*)p.y)[part * p.part_stride + from + c]; }
      else v = to_float<T>(((const T*)p.y)[from + c]);
      total = fmaf(p.share ? p.share[(long long)t * p.top + k] : 1.f, v, total);
    }
    return total * p.y_scale;
  };
  float squares = 0.f;
  for (int c = threadIdx.x; c < p.width; c += blockDim.x) { const float v = value(c); squares = fmaf(v, v, squares); }
  const float inv = 1.f / sqrtf(block_sum(squares, scratch) / p.width + p.eps);
  for (int c = threadIdx.x; c < p.width; c += blockDim.x) {
    const long long at = (long long)t * p.width + c;
    const float r = fmaf(value(c) * inv, p.weight[c], p.accumulate ? p.x[at] : 0.f);
    p.x[at] = r;
    if (p.copy) ((T*)p.copy)[at] = from_float<T>(r);
  }
}

}  // namespace pylon

using namespace pylon;

// y: [tokens, width] in dtype (parts 0) or float32 [parts, tokens, width]; with ids (int32 [tokens]) rows of y [vocab, width] in dtype.
// With slot_of (int32 [tokens, top]) rows of y [slots, width] in dtype, or float32 [parts, slots, width], with share float32 [tokens, top] or null.
// x float32 [tokens, width], read if accumulate != 0 and written; copy [tokens, width] in dtype, or null; weight float32 [width].
extern "C" int pylon_output_norm(const void* y, int parts, const int* ids, int vocab, const int* slot_of, const float* share, int top, long long slots,
                                 float y_scale, float* x, void* copy, const float* weight, int tokens, int width, float eps, int accumulate, int dtype, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (width < 1 || parts < 0 || (ids && (parts > 0 || vocab < 1 || slot_of)) || (slot_of && (top < 1 || slots < 1)) || (share && !slot_of)) PYLON_REFUSE("output_norm: width %d, %d parts, %d table rows", width, parts, vocab);
  if (dtype != PYLON_DTYPE_F32 && dtype != PYLON_DTYPE_BF16) PYLON_REFUSE("output_norm: unknown dtype %d", dtype);
  const OutputNormParams p{y, parts, (slot_of ? slots : tokens) * width, ids, slot_of, share, slot_of ? top : 1, vocab, y_scale, x, copy, weight, width, eps, accumulate};
  // threads by the width alone, so that a token's sum does not depend on the step: two pieces a thread where a block has room for it
  int threads = 64;
  while (threads < 1024 && threads * 2 < width / 4) threads *= 2;
  const bool pieces = width % 4 == 0 && width / 4 <= threads * 4 && (uintptr_t)y % 16 == 0 && (uintptr_t)x % 16 == 0 && (uintptr_t)copy % 8 == 0 && (uintptr_t)weight % 16 == 0;
#define PYLON_OUTPUT_NORM(T)                                                                                            \
  if (pieces && width / 4 <= threads * 2) launch_dependent(output_norm_vec_kernel<T, 2>, dim3((unsigned)tokens), dim3(threads), 0, stream, p); \
  else if (pieces) launch_dependent(output_norm_vec_kernel<T, 4>, dim3((unsigned)tokens), dim3(threads), 0, stream, p); \
  else launch_dependent(output_norm_kernel<T>, dim3((unsigned)tokens), dim3(256), 0, stream, p)
  if (dtype == PYLON_DTYPE_F32) { PYLON_OUTPUT_NORM(float); } else { PYLON_OUTPUT_NORM(__nv_bfloat16); }
#undef PYLON_OUTPUT_NORM
  PYLON_CHECK_LAUNCH("output_norm");
}
