// What stands between an attention mixer's projections and its attention, for the forms the fused
// kernels of elementwise.cu are not written for: biases, rotation of part of a head, either layout of
// the rotated pairs, the per-head norm before or after the rotation and with or without a weight,
// values of another width than the keys, and a latent row per token in place of keys and values.
//
// A rotation turns the pair (u, v) of a head at position p into (u cos a - v sin a, v cos a + u sin a);
// a = p * f_i comes as float32 tables cos/sin [positions, rot / 2] (any scaling of the frequencies, and
// any factor on cos and sin, is in the tables).  Layout 0 pairs element i with i + rot / 2, layout 1
// element 2 i with 2 i + 1, i < rot / 2; elements from `rot` on pass unchanged.  All arithmetic is float32.
//
// Further: the norm may run over a token's whole q row and whole k row, all heads at once (weights as long as those rows); a query may be
// multiplied by a factor by position (q_factors [positions]); and the values may be the projected keys, biases included, as they are before
// norm and rotation (values_from_keys: there are no value columns then).
#include "common.cuh"

namespace pylon {

// norm_mode 0: no norm of q and k, 1: per head before the rotation, 2: per head after it, 3: over the whole row, before it.
struct RotaryOptions {
  int norm_mode;
  int values_from_keys;
  const float* q_factors;   // float32 [factor_positions] or null
  int factor_positions;
};

constexpr int ROTARY_THREADS = 128;
constexpr int ROTARY_WARPS = ROTARY_THREADS / 32;

// Rotates buf[0 .. rot) in place; one lane owns a pair.  The caller orders the warp before and after.
__device__ __forceinline__ void rotate_pairs(float* buf, const float* __restrict__ cos_row, const float* __restrict__ sin_row, int rot, int layout, int lane) {
  const int half = rot >> 1;
  for (int i = lane; i < half; i += 32) {
    const int a = layout ? 2 * i : i, b = layout ? 2 * i + 1 : i + half;
    const float c = cos_row[i], s = sin_row[i], u = buf[a], v = buf[b];
    buf[a] = u * c - v * s;
    buf[b] = v * c + u * s;
  }
}

// buf[0 .. n) divided by its root mean square, times weight (or 1).  `size`: how many of the n elements are the vector's own; the rest are zeros.
__device__ __forceinline__ void unit_rms(float* buf, int n, int size, const float* __restrict__ weight, float eps, int lane) {
  float squares = 0.f;
  for (int e = lane; e < n; e += 32) squares = fmaf(buf[e], buf[e], squares);
  const float inv = rsqrtf(warp_sum(squares) / size + eps);
  for (int e = lane; e < n; e += 32) buf[e] *= weight ? inv * weight[e] : inv;
}

// One warp per (token, head of q, k or v); WHOLE: a block per token, whose warps take the heads in turn behind the two sums.  qkv [T, ld] holds [q: nq x d | k: nkv x d | v: nkv x dv] per token; q is
// written back in place, k and v go into the token's slot of its pages.
template <typename T, bool WHOLE>
__global__ void __launch_bounds__(ROTARY_THREADS) qkv_rotate_write_kernel(
    T* __restrict__ qkv, long long ld, const float* __restrict__ bias, const float* __restrict__ cos_table, const float* __restrict__ sin_table,
    int rot, int layout, int table_positions, RotaryOptions options, const float* __restrict__ q_weight, const float* __restrict__ k_weight, float eps,
    const int* __restrict__ positions, const int* __restrict__ token_row, const int* __restrict__ block_table, int table_width, int page_size,
    T* __restrict__ k_pages, T* __restrict__ v_pages, int num_pages, int nq, int nkv, int d, int dv, int norm_size, int num_tokens, int* __restrict__ error_word) {
  extern __shared__ float rotary_shared[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int widest = d > dv ? d : dv;
  float* buf = rotary_shared + (size_t)warp * widest;
  const int per_token = nq + 2 * nkv, norm_mode = options.norm_mode;
  const long long item = WHOLE ? 0 : (long long)blockIdx.x * ROTARY_WARPS + warp;
  if (!WHOLE && item >= (long long)num_tokens * per_token) return;
  const int t = WHOLE ? (int)blockIdx.x : (int)(item / per_token);
  const int row = token_row[t];
  if (row < 0) return;   // a padding token: nothing of it is kept
  const int pos = positions[t];
  float q_inv = 1.f, k_inv = 1.f;
  if (WHOLE) {
    float* scratch = rotary_shared + (size_t)ROTARY_WARPS * widest;   // [34]
    float q_squares = 0.f, k_squares = 0.f;
    for (int e = threadIdx.x; e < (nq + nkv) * d; e += ROTARY_THREADS) {
      const float x = to_float<T>(qkv[(size_t)t * ld + e]) + (bias ? bias[e] : 0.f);
      if (e < nq * d) q_squares = fmaf(x, x, q_squares);
      else k_squares = fmaf(x, x, k_squares);
    }
    q_inv = rsqrtf(block_sum(q_squares, scratch) / (nq * norm_size) + eps);
    k_inv = rsqrtf(block_sum(k_squares, scratch) / (nkv * norm_size) + eps);
  }
  for (int hh = WHOLE ? warp : (int)(item % per_token); hh < per_token; hh += WHOLE ? ROTARY_WARPS : per_token) {
  __syncwarp();
  const bool is_q = hh < nq, is_v = hh >= nq + nkv;
  const int width = is_v ? dv : d;
  const int column = is_q ? hh * d : (is_v ? (options.values_from_keys ? (hh - nkv) * d : (nq + nkv) * d + (hh - nq - nkv) * dv) : hh * d);
  T* src = qkv + (size_t)t * ld + column;
  for (int e = lane; e < width; e += 32) buf[e] = to_float<T>(src[e]) + (bias ? bias[column + e] : 0.f);
  __syncwarp();
  if (!is_v) {
    const float* weight = is_q ? q_weight : k_weight;
    if (norm_mode == 1) {
      unit_rms(buf, d, norm_size, weight, eps, lane);
      __syncwarp();
    }
    if (WHOLE) {
      for (int e = lane; e < d; e += 32) buf[e] *= is_q ? q_inv * weight[column + e] : k_inv * weight[column - nq * d + e];
      __syncwarp();
    }
    if (rot > 0 && pos < table_positions) {
      rotate_pairs(buf, cos_table + (size_t)pos * (rot >> 1), sin_table + (size_t)pos * (rot >> 1), rot, layout, lane);
      __syncwarp();
    }
    if (norm_mode == 2) {
      unit_rms(buf, d, norm_size, weight, eps, lane);
      __syncwarp();
    }
    if (is_q && options.q_factors && pos < options.factor_positions) {
      for (int e = lane; e < d; e += 32) buf[e] *= options.q_factors[pos];
      __syncwarp();
    }
  }
  T* dst = src;
  if (!is_q) {
    const int logical = pos / page_size;
    const int page = logical < table_width ? block_table[(size_t)row * table_width + logical] : -1;
    if (page < 0 || page >= num_pages) {
      if (lane == 0 && error_word) atomicMax(error_word, PYLON_ERROR_BAD_PAGE);
      continue;
    }
    const int head = is_v ? hh - nq - nkv : hh - nq;
    dst = (is_v ? v_pages : k_pages) + (((size_t)page * nkv + head) * page_size + pos % page_size) * width;
  }
  for (int e = lane; e < width; e += 32) dst[e] = from_float<T>(buf[e]);
  }
}

// The same for bfloat16 rows whose pairs lie rot / 2 apart, rot a multiple of 16.  A block takes one token; `lanes` (a power
// of two) lanes share a head, each with 8 neighbouring elements as one 16-byte piece; the rotation partners of a lane's elements are all in
// one other lane.  A lane meets the same elements of several heads, so it reads its angles once, and four heads' pieces are on their
// way at once.
__device__ __forceinline__ void unpack_8(float (&x)[8], const uint4& raw) {
  const unsigned words[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 pair = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&words[i]));
    x[2 * i] = pair.x; x[2 * i + 1] = pair.y;
  }
}
__device__ __forceinline__ void load_8(float (&x)[8], const float* from) {
  const float4 low = *reinterpret_cast<const float4*>(from), high = *reinterpret_cast<const float4*>(from + 4);
  x[0] = low.x; x[1] = low.y; x[2] = low.z; x[3] = low.w; x[4] = high.x; x[5] = high.y; x[6] = high.z; x[7] = high.w;
}

constexpr int ROTARY_VEC_MOST = 512;   // threads of a block at most: a step of few tokens gives every head lanes of its own

__global__ void __launch_bounds__(ROTARY_VEC_MOST, 2) qkv_rotate_write_vec_kernel(
    __nv_bfloat16* __restrict__ qkv, long long ld, const float* __restrict__ bias, const float* __restrict__ cos_table, const float* __restrict__ sin_table, int rot,
    int table_positions, RotaryOptions options, const float* __restrict__ q_weight, const float* __restrict__ k_weight, float eps, const int* __restrict__ positions,
    const int* __restrict__ token_row, const int* __restrict__ block_table, int table_width, int page_size, __nv_bfloat16* __restrict__ k_pages,
    __nv_bfloat16* __restrict__ v_pages, int num_pages, int nq, int nkv, int d, int dv, int norm_size, int lanes, int* __restrict__ error_word) {
  constexpr int SIDE = 4;                              // heads of a lane on their way at once
  __shared__ float scratch[34];
  const int norm_mode = options.norm_mode;
  const int t = blockIdx.x, row = token_row[t];        // position, page and angles do not depend on the kernel ahead
  if (row < 0) {                                       // a padding token: nothing of it is kept
    grid_dependency_wait();                            // a grid must not end before the grid ahead of it has
    return;
  }
  const int mine = (int)(threadIdx.x % lanes) * 8;     // this lane's first element
  const int group = threadIdx.x / lanes, groups = blockDim.x / lanes;
  const int pos = positions[t], half = rot >> 1, heads = nq + 2 * nkv;
  const bool turned = mine < rot && pos < table_positions;
  float c[8], s[8];
  if (turned) {
    const size_t angle = (size_t)pos * half + (mine < half ? mine : mine - half);
    load_8(c, cos_table + angle);
    load_8(s, sin_table + angle);
  }
  const int logical = pos / page_size;
  const int page = logical < table_width ? block_table[(size_t)row * table_width + logical] : -1;
  const bool page_there = page >= 0 && page < num_pages;
  const size_t slot = (size_t)(page_there ? page : 0) * nkv * page_size + pos % page_size;
  const int lane = threadIdx.x & 31, apart = half >> 3, partner = (mine < half ? lane + apart : lane - apart) & 31;
  const float q_factor = options.q_factors && pos < options.factor_positions ? options.q_factors[pos] : 1.f;
  grid_dependency_wait();
  allow_dependents();
  auto column_of = [&](int hh) { return hh < nq + nkv ? hh * d : (options.values_from_keys ? (hh - nkv) * d : (nq + nkv) * d + (hh - nq - nkv) * dv); };
  auto add_bias = [&](float (&x)[8], int hh) {
    if (!bias) return;
    float b[8];
    load_8(b, bias + column_of(hh) + mine);
#pragma unroll
    for (int i = 0; i < 8; ++i) x[i] += b[i];
  };
  float q_inv = 1.f, k_inv = 1.f;
  if (norm_mode == 3) {                                // over the whole rows: their sums first, the pieces come from the cache the second time
    float q_squares = 0.f, k_squares = 0.f;
    for (int hh = group; hh < nq + nkv; hh += groups) {
      if (mine >= d) continue;
      float x[8];
      unpack_8(x, *reinterpret_cast<const uint4*>(qkv + (size_t)t * ld + hh * d + mine));
      add_bias(x, hh);
      float squares = 0.f;
#pragma unroll
      for (int i = 0; i < 8; ++i) squares = fmaf(x[i], x[i], squares);
      if (hh < nq) q_squares += squares;
      else k_squares += squares;
    }
    q_inv = rsqrtf(block_sum(q_squares, scratch) / (nq * norm_size) + eps);
    k_inv = rsqrtf(block_sum(k_squares, scratch) / (nkv * norm_size) + eps);
  }
  for (int h0 = 0; h0 < heads; h0 += SIDE * groups) {  // the same turns for every lane: all of a warp meet the shuffles
    uint4 raw[SIDE];
#pragma unroll
    for (int k = 0; k < SIDE; ++k) {
      const int hh = h0 + k * groups + group;
      const bool is_v = hh >= nq + nkv;
      const bool live = hh < heads && mine < (is_v ? dv : d);
      raw[k] = live ? *reinterpret_cast<const uint4*>(qkv + (size_t)t * ld + column_of(hh) + mine) : make_uint4(0u, 0u, 0u, 0u);
    }
#pragma unroll
    for (int k = 0; k < SIDE; ++k) {
      if (h0 + k * groups >= heads) break;               // the same for every lane
      const int hh = h0 + k * groups + group;
      const bool is_q = hh < nq, is_v = hh >= nq + nkv;
      float x[8];
      unpack_8(x, raw[k]);
      if (hh < heads && mine < (is_v ? dv : d)) add_bias(x, hh);
      auto unit = [&]() {
        float squares = 0.f;
#pragma unroll
        for (int i = 0; i < 8; ++i) squares = fmaf(x[i], x[i], squares);
        for (int offset = lanes >> 1; offset > 0; offset >>= 1) squares += __shfl_xor_sync(0xffffffffu, squares, offset);
        const float inv = rsqrtf(squares / norm_size + eps);
#pragma unroll
        for (int i = 0; i < 8; ++i) x[i] *= inv;
        const float* weight = is_q ? q_weight : k_weight;
        if (weight && mine < d) {
          float w[8];
          load_8(w, weight + mine);
#pragma unroll
          for (int i = 0; i < 8; ++i) x[i] *= w[i];
        }
      };
      if (norm_mode == 1) unit();
      if (norm_mode == 3 && !is_v && mine < d) {
        float w[8];
        load_8(w, is_q ? q_weight + hh * d + mine : k_weight + (hh - nq) * d + mine);
#pragma unroll
        for (int i = 0; i < 8; ++i) x[i] *= (is_q ? q_inv : k_inv) * w[i];
      }
      if (rot > 0) {
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const float other = __shfl_sync(0xffffffffu, x[i], partner);
          if (turned) x[i] = mine < half ? x[i] * c[i] - other * s[i] : x[i] * c[i] + other * s[i];
        }
      }
      if (norm_mode == 2) unit();
      if (is_q) {
#pragma unroll
        for (int i = 0; i < 8; ++i) x[i] *= q_factor;
      }
      if (hh >= heads || mine >= (is_v ? dv : d)) continue;
      uint4 result = raw[k];                             // a value without a bias stays what it is
      if (is_v && bias) {                                // neither normed nor rotated: its own numbers again
        unpack_8(x, raw[k]);
        add_bias(x, hh);
      }
      if (!is_v || bias) {
        unsigned words[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const __nv_bfloat162 pair = __floats2bfloat162_rn(x[2 * i], x[2 * i + 1]);
          words[i] = *reinterpret_cast<const unsigned*>(&pair);
        }
        result = make_uint4(words[0], words[1], words[2], words[3]);
      }
      if (is_q) *reinterpret_cast<uint4*>(qkv + (size_t)t * ld + hh * d + mine) = result;
      else if (!page_there) { if (mine == 0 && error_word) atomicMax(error_word, PYLON_ERROR_BAD_PAGE); }
      else if (is_v) *reinterpret_cast<uint4*>(v_pages + (slot + (size_t)(hh - nq - nkv) * page_size) * dv + mine) = result;
      else *reinterpret_cast<uint4*>(k_pages + (slot + (size_t)(hh - nq) * page_size) * d + mine) = result;
    }
  }
}

// One block per token.  down [T, ld] holds [query latent: q_rank | key/value latent: kv_rank | shared rotated key part: rot_dim].
// cq [T, q_rank] = RMS norm of the query latent times q_weight; the token's one cache row [kv_rank + rot_dim] = RMS norm of the
// key/value latent times kv_weight, then the rotated key part (its first `rot` elements rotated, not normed).
template <typename T>
__global__ void __launch_bounds__(ROTARY_THREADS) latent_norm_rotate_write_kernel(
    const T* __restrict__ down, long long ld, T* __restrict__ cq, const float* __restrict__ q_weight, const float* __restrict__ kv_weight, float eps,
    const float* __restrict__ cos_table, const float* __restrict__ sin_table, int rot, int layout, int table_positions,
    const int* __restrict__ positions, const int* __restrict__ token_row, const int* __restrict__ block_table, int table_width, int page_size,
    T* __restrict__ pages, int num_pages, int q_rank, int kv_rank, int rot_dim, int* __restrict__ error_word) {
  extern __shared__ float rotary_shared[];
  float* scratch = rotary_shared;        // [34]
  float* staged = rotary_shared + 34;    // [q_rank + kv_rank + rot_dim]: the token's row, read from global memory once
  float* turned = staged + q_rank + kv_rank;
  const int t = blockIdx.x, tid = threadIdx.x;
  const int row = token_row[t];
  if (row < 0) return;
  const int pos = positions[t];
  const T* src = down + (size_t)t * ld;
  const int total = q_rank + kv_rank + rot_dim;
#pragma unroll 4
  for (int e = tid; e < total; e += ROTARY_THREADS) staged[e] = to_float<T>(src[e]);
  const int logical = pos / page_size;
  const int page = logical < table_width ? block_table[(size_t)row * table_width + logical] : -1;
  __syncthreads();
  float q_squares = 0.f, kv_squares = 0.f;
  for (int e = tid; e < q_rank; e += ROTARY_THREADS) q_squares = fmaf(staged[e], staged[e], q_squares);
  for (int e = tid; e < kv_rank; e += ROTARY_THREADS) kv_squares = fmaf(staged[q_rank + e], staged[q_rank + e], kv_squares);
  const float q_inv = rsqrtf(block_sum(q_squares, scratch) / (q_rank > 0 ? q_rank : 1) + eps);
  const float kv_inv = rsqrtf(block_sum(kv_squares, scratch) / kv_rank + eps);
  for (int e = tid; e < q_rank; e += ROTARY_THREADS) cq[(size_t)t * q_rank + e] = from_float<T>(staged[e] * q_inv * q_weight[e]);
  if (tid < 32 && rot > 0 && pos < table_positions)
    rotate_pairs(turned, cos_table + (size_t)pos * (rot >> 1), sin_table + (size_t)pos * (rot >> 1), rot, layout, tid);
  __syncthreads();
  if (page < 0 || page >= num_pages) {
    if (tid == 0 && error_word) atomicMax(error_word, PYLON_ERROR_BAD_PAGE);
    return;
  }
  T* dst = pages + ((size_t)page * page_size + pos % page_size) * (kv_rank + rot_dim);
  for (int e = tid; e < kv_rank; e += ROTARY_THREADS) dst[e] = from_float<T>(staged[q_rank + e] * kv_inv * kv_weight[e]);
  for (int e = tid; e < rot_dim; e += ROTARY_THREADS) dst[kv_rank + e] = from_float<T>(turned[e]);
}

// One warp per (token, head): dst[t, h, 0 .. width) = src[t, h, 0 .. width) with its first `rot` elements rotated.
template <typename T>
__global__ void __launch_bounds__(ROTARY_THREADS) rotate_heads_kernel(
    const T* __restrict__ src, long long src_token_stride, long long src_head_stride, T* __restrict__ dst, long long dst_token_stride,
    long long dst_head_stride, const float* __restrict__ cos_table, const float* __restrict__ sin_table, int rot, int layout, int table_positions,
    const int* __restrict__ positions, int heads, int width, int num_tokens) {
  extern __shared__ float rotary_shared[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* buf = rotary_shared + (size_t)warp * width;
  const long long item = (long long)blockIdx.x * ROTARY_WARPS + warp;
  if (item >= (long long)num_tokens * heads) return;
  const int t = (int)(item / heads), h = (int)(item % heads);
  const int pos = positions[t];
  const T* from = src + (size_t)t * src_token_stride + (size_t)h * src_head_stride;
  for (int e = lane; e < width; e += 32) buf[e] = to_float<T>(from[e]);
  __syncwarp();
  if (rot > 0 && pos >= 0 && pos < table_positions) rotate_pairs(buf, cos_table + (size_t)pos * (rot >> 1), sin_table + (size_t)pos * (rot >> 1), rot, layout, lane);
  __syncwarp();
  T* to = dst + (size_t)t * dst_token_stride + (size_t)h * dst_head_stride;
  for (int e = lane; e < width; e += 32) to[e] = from_float<T>(buf[e]);
}

}  // namespace pylon

using namespace pylon;

extern "C" int pylon_qkv_rotate_write(void* qkv, long long ld, const float* bias, const float* cos_table, const float* sin_table, int rot, int layout,
                                      int table_positions, int norm_mode, const float* q_weight, const float* k_weight, float eps, const int* positions,
                                      const int* token_row, const int* block_table, int table_width, int page_size, void* k_pages, void* v_pages,
                                      int num_pages, int nq, int nkv, int d, int dv, int norm_size, int num_tokens, int dtype, int* error_word, int values_from_keys,
                                      const float* q_factors, int factor_positions, cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  if (values_from_keys && dv != d) PYLON_REFUSE("qkv_rotate_write: values of %d that are keys of %d", dv, d);
  if (norm_mode == 3 && (!q_weight || !k_weight)) PYLON_REFUSE("qkv_rotate_write: a norm over whole rows needs its weights");
  const RotaryOptions options{norm_mode, values_from_keys, q_factors, factor_positions};
  if (norm_size < 1 || norm_size > d) PYLON_REFUSE("qkv_rotate_write: a norm over %d of %d elements", norm_size, d);
  if (nq < 1 || nkv < 1 || d < 1 || dv < 1 || d > 2048 || dv > 2048) PYLON_REFUSE("qkv_rotate_write: %d / %d heads of %d and %d", nq, nkv, d, dv);
  if (rot < 0 || rot > d || rot % 2 || (rot > 0 && (!cos_table || !sin_table))) PYLON_REFUSE("qkv_rotate_write: %d rotated elements of %d", rot, d);
  if (norm_mode < 0 || norm_mode > 3 || page_size < 1 || table_width < 1) PYLON_REFUSE("qkv_rotate_write: norm mode %d, page size %d, table width %d", norm_mode, page_size, table_width);
  const long long items = (long long)num_tokens * (nq + 2 * nkv);
  const bool whole = norm_mode == 3;
  const unsigned blocks = whole ? (unsigned)num_tokens : (unsigned)((items + ROTARY_WARPS - 1) / ROTARY_WARPS);
  const size_t smem = ((size_t)ROTARY_WARPS * (d > dv ? d : dv) + 34) * sizeof(float);
#define PYLON_ROTATE_WRITE(T, WHOLE)                                                                                                                     \
  qkv_rotate_write_kernel<T, WHOLE><<<blocks, ROTARY_THREADS, smem, stream>>>(                                                                           \
      (T*)qkv, ld, bias, cos_table, sin_table, rot, layout, table_positions, options, q_weight, k_weight, eps, positions, token_row, block_table,        \
      table_width, page_size, (T*)k_pages, (T*)v_pages, num_pages, nq, nkv, d, dv, norm_size, num_tokens, error_word)
  if (dtype == PYLON_DTYPE_F32) {
    if (whole) PYLON_ROTATE_WRITE(float, true); else PYLON_ROTATE_WRITE(float, false);
  } else if (dtype == PYLON_DTYPE_BF16 && layout == 0 && (uintptr_t)bias % 16 == 0 && rot % 16 == 0 && d % 8 == 0 && dv % 8 == 0 && d <= 256 && dv <= 256 && ld % 8 == 0 &&
           (uintptr_t)qkv % 16 == 0 && (uintptr_t)k_pages % 16 == 0 && (uintptr_t)v_pages % 16 == 0 && (uintptr_t)cos_table % 16 == 0 && (uintptr_t)sin_table % 16 == 0 &&
           (uintptr_t)q_weight % 16 == 0 && (uintptr_t)k_weight % 16 == 0) {
    int lanes = 1;
    while (lanes * 8 < (d > dv ? d : dv)) lanes *= 2;
    const int threads = num_tokens <= 148 ? ROTARY_VEC_MOST : ROTARY_THREADS;
    launch_dependent(qkv_rotate_write_vec_kernel, dim3((unsigned)num_tokens), dim3(threads), 0, stream, (__nv_bfloat16*)qkv, ld, bias, cos_table, sin_table, rot,
                     table_positions, options, q_weight, k_weight, eps, positions, token_row, block_table, table_width, page_size, (__nv_bfloat16*)k_pages,
                     (__nv_bfloat16*)v_pages, num_pages, nq, nkv, d, dv, norm_size, lanes, error_word);
  } else if (dtype == PYLON_DTYPE_BF16) {
    if (whole) PYLON_ROTATE_WRITE(__nv_bfloat16, true); else PYLON_ROTATE_WRITE(__nv_bfloat16, false);
  }
#undef PYLON_ROTATE_WRITE
  else
    PYLON_REFUSE("qkv_rotate_write: unknown dtype %d", dtype);
  PYLON_CHECK_LAUNCH("qkv_rotate_write");
}

extern "C" int pylon_latent_norm_rotate_write(const void* down, long long ld, void* cq, const float* q_weight, const float* kv_weight, float eps,
                                              const float* cos_table, const float* sin_table, int rot, int layout, int table_positions,
                                              const int* positions, const int* token_row, const int* block_table, int table_width, int page_size,
                                              void* pages, int num_pages, int q_rank, int kv_rank, int rot_dim, int num_tokens, int dtype,
                                              int* error_word, cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  if (q_rank < 0 || kv_rank < 1 || rot_dim < 0 || rot_dim > 8192) PYLON_REFUSE("latent_norm_rotate_write: ranks %d / %d, %d rotated", q_rank, kv_rank, rot_dim);
  if (rot < 0 || rot > rot_dim || rot % 2 || (rot > 0 && (!cos_table || !sin_table))) PYLON_REFUSE("latent_norm_rotate_write: %d rotated elements of %d", rot, rot_dim);
  if (page_size < 1 || table_width < 1) PYLON_REFUSE("latent_norm_rotate_write: page size %d, table width %d", page_size, table_width);
  const size_t smem = (size_t)(34 + q_rank + kv_rank + rot_dim) * sizeof(float);
  if (smem > 48 * 1024) PYLON_REFUSE("latent_norm_rotate_write: a row of %d numbers is too wide", q_rank + kv_rank + rot_dim);
  if (dtype == PYLON_DTYPE_F32)
    latent_norm_rotate_write_kernel<float><<<num_tokens, ROTARY_THREADS, smem, stream>>>(
        (const float*)down, ld, (float*)cq, q_weight, kv_weight, eps, cos_table, sin_table, rot, layout, table_positions, positions, token_row,
        block_table, table_width, page_size, (float*)pages, num_pages, q_rank, kv_rank, rot_dim, error_word);
  else if (dtype == PYLON_DTYPE_BF16)
    latent_norm_rotate_write_kernel<__nv_bfloat16><<<num_tokens, ROTARY_THREADS, smem, stream>>>(
        (const __nv_bfloat16*)down, ld, (__nv_bfloat16*)cq, q_weight, kv_weight, eps, cos_table, sin_table, rot, layout, table_positions, positions,
        token_row, block_table, table_width, page_size, (__nv_bfloat16*)pages, num_pages, q_rank, kv_rank, rot_dim, error_word);
  else
    PYLON_REFUSE("latent_norm_rotate_write: unknown dtype %d", dtype);
  PYLON_CHECK_LAUNCH("latent_norm_rotate_write");
}

extern "C" int pylon_rotate_heads(const void* src, long long src_token_stride, long long src_head_stride, void* dst, long long dst_token_stride,
                                  long long dst_head_stride, const float* cos_table, const float* sin_table, int rot, int layout, int table_positions,
                                  const int* positions, int heads, int width, int num_tokens, int dtype, cudaStream_t stream) {
  if (num_tokens <= 0 || heads <= 0 || width <= 0) return 0;
  if (width > 2048 || rot < 0 || rot > width || rot % 2 || (rot > 0 && (!cos_table || !sin_table))) PYLON_REFUSE("rotate_heads: %d rotated elements of %d", rot, width);
  const long long items = (long long)num_tokens * heads;
  const unsigned blocks = (unsigned)((items + ROTARY_WARPS - 1) / ROTARY_WARPS);
  const size_t smem = (size_t)ROTARY_WARPS * width * sizeof(float);
  if (dtype == PYLON_DTYPE_F32)
    rotate_heads_kernel<float><<<blocks, ROTARY_THREADS, smem, stream>>>((const float*)src, src_token_stride, src_head_stride, (float*)dst, dst_token_stride,
                                                                          dst_head_stride, cos_table, sin_table, rot, layout, table_positions, positions,
                                                                          heads, width, num_tokens);
  else if (dtype == PYLON_DTYPE_BF16)
    rotate_heads_kernel<__nv_bfloat16><<<blocks, ROTARY_THREADS, smem, stream>>>((const __nv_bfloat16*)src, src_token_stride, src_head_stride,
                                                                                  (__nv_bfloat16*)dst, dst_token_stride, dst_head_stride, cos_table, sin_table,
                                                                                  rot, layout, table_positions, positions, heads, width, num_tokens);
  else
    PYLON_REFUSE("rotate_heads: unknown dtype %d", dtype);
  PYLON_CHECK_LAUNCH("rotate_heads");
}
