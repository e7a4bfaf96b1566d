// The norm that stands on a sublayer's output, with what follows it: per token
//
//     n = y / sqrt(mean(y^2) + eps) * weight
//     x = x + n        (or x = n: the first of the stream)
//     copy = x in the compute dtype, what the next sublayer reads
//
// all in float32.  y comes as [T, width] in the compute dtype, as float32 partial sums [parts, T, width] whose sum it is, or as rows of
// a table [vocab, width] times a factor, picked by ids (the embedding).  A block takes one token; a thread keeps its columns of y between
// the sum of squares and the result.
#include "common.cuh"

namespace pylon {

constexpr int OUTPUT_NORM_HELD = 4;   // 4-column pieces a thread keeps

struct OutputNormParams {
  const void* y;
  int parts;                // 0: in T; > 0: float32 partial sums
  long long part_stride;    // elements between the parts
  const int* ids;           // null, or which row of y a token reads
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
    float4 sum = *reinterpret_cast<const float4*>((const float*)p.y + at);
    for (int part = 1; part < p.parts; ++part) {
      const float4 more = *reinterpret_cast<const float4*>((const float*)p.y + part * p.part_stride + at);
      sum.x += more.x; sum.y += more.y; sum.z += more.z; sum.w += more.w;
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

template <typename T>
__global__ void output_norm_vec_kernel(const OutputNormParams p) {
  __shared__ float scratch[34];
  const int t = blockIdx.x, pieces = p.width / 4;
  grid_dependency_wait();
  allow_dependents();
  long long from = (long long)t * p.width;
  if (p.ids) {
    const int id = p.ids[t];
    from = (long long)(id < 0 ? 0 : (id < p.vocab ? id : p.vocab - 1)) * p.width;
  }
  float4 y[OUTPUT_NORM_HELD], x[OUTPUT_NORM_HELD];
  float squares = 0.f;
#pragma unroll
  for (int i = 0; i < OUTPUT_NORM_HELD; ++i) {
    const int piece = threadIdx.x + i * blockDim.x;
    if (piece < pieces) {
      y[i] = output_norm_piece<T>(p, from + 4 * piece);
      if (p.accumulate) x[i] = *reinterpret_cast<const float4*>(p.x + (long long)t * p.width + 4 * piece);   // on its way while the squares are summed
      else x[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    } else y[i] = x[i] = make_float4(0.f, 0.f, 0.f, 0.f);
  }
#pragma unroll
  for (int i = 0; i < OUTPUT_NORM_HELD; ++i) {
    y[i].x *= p.y_scale; y[i].y *= p.y_scale; y[i].z *= p.y_scale; y[i].w *= p.y_scale;
    squares = fmaf(y[i].x, y[i].x, fmaf(y[i].y, y[i].y, fmaf(y[i].z, y[i].z, fmaf(y[i].w, y[i].w, squares))));
  }
  const float inv = 1.f / sqrtf(block_sum(squares, scratch) / p.width + p.eps);
#pragma unroll
  for (int i = 0; i < OUTPUT_NORM_HELD; ++i) {
    const int piece = threadIdx.x + i * blockDim.x;
    if (piece >= pieces) continue;
    const float4 w = *reinterpret_cast<const float4*>(p.weight + 4 * piece);
    const float4 r = make_float4(fmaf(y[i].x * inv, w.x, x[i].x), fmaf(y[i].y * inv, w.y, x[i].y), fmaf(y[i].z * inv, w.z, x[i].z), fmaf(y[i].w * inv, w.w, x[i].w));
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
  long long from = (long long)t * p.width;
  if (p.ids) {
    const int id = p.ids[t];
    from = (long long)(id < 0 ? 0 : (id < p.vocab ? id : p.vocab - 1)) * p.width;
  }
  auto value = [&](int c) {
    float v = 0.f;
    if (p.parts > 0) { for (int part = 0; part < p.parts; ++part) v += ((const float*)p.y)[part * p.part_stride + from + c]; }
    else v = to_float<T>(((const T*)p.y)[from + c]);
    return v * p.y_scale;
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
// x float32 [tokens, width], read if accumulate != 0 and written; copy [tokens, width] in dtype, or null; weight float32 [width].
extern "C" int pylon_output_norm(const void* y, int parts, const int* ids, int vocab, float y_scale, float* x, void* copy, const float* weight, int tokens,
                                 int width, float eps, int accumulate, int dtype, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (width < 1 || parts < 0 || (ids && (parts > 0 || vocab < 1))) PYLON_REFUSE("output_norm: width %d, %d parts, %d table rows", width, parts, vocab);
  if (dtype != PYLON_DTYPE_F32 && dtype != PYLON_DTYPE_BF16) PYLON_REFUSE("output_norm: unknown dtype %d", dtype);
  const OutputNormParams p{y, parts, (long long)tokens * width, ids, vocab, y_scale, x, copy, weight, width, eps, accumulate};
  // threads by the width alone, so that a token's sum does not depend on the step: two pieces a thread where a block has room for it
  int threads = 64;
  while (threads < 1024 && threads * 2 < width / 4) threads *= 2;
  const bool pieces = width % 4 == 0 && width / 4 <= threads * OUTPUT_NORM_HELD && (uintptr_t)y % 16 == 0 && (uintptr_t)x % 16 == 0 && (uintptr_t)copy % 8 == 0 && (uintptr_t)weight % 16 == 0;
#define PYLON_OUTPUT_NORM(T)                                                                                            \
  if (pieces) launch_dependent(output_norm_vec_kernel<T>, dim3((unsigned)tokens), dim3(threads), 0, stream, p);         \
  else launch_dependent(output_norm_kernel<T>, dim3((unsigned)tokens), dim3(256), 0, stream, p)
  if (dtype == PYLON_DTYPE_F32) { PYLON_OUTPUT_NORM(float); } else { PYLON_OUTPUT_NORM(__nv_bfloat16); }
#undef PYLON_OUTPUT_NORM
  PYLON_CHECK_LAUNCH("output_norm");
}
