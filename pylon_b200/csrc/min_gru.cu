// A minimal gated recurrence over channels (minGRU): gate and candidate of a token read that token only.
//
// Per token, from one product of the layer's input, columns [z | x | g] of C channels each (biases b_z, b_x):
//
//     z         = sigmoid(z + b_z)
//     u         = x + b_x           candidate c = u + 1/2 where u >= 0, sigmoid(u) where u < 0
//     S         = (1 - z) S + z c   from S = 0
//     out       = factor * S * silu(g)
//
// What a request carries from token to token is one float32 slot of C numbers, read at state[slots[row]] and advanced in place by
// the row's tokens.  All arithmetic is float32.  The update is formed as S + z (c - S): where a gate is nearly shut, rounding 1 - z
// would change its distance from one by the same share at every token.
//
//   min_gru_walk      a thread per request row and V channels walks the row's tokens: steps of a few tokens a row
//   min_gru_cluster   prompt portions.  The state enters linearly, so a piece of the row walked from S = 0 gives its own share B, and
//                     the product A of its (1 - z) is the factor on what enters it: S_out = A S_in + B.  A thread-block cluster takes a
//                     row's 32 V channels; its warps take equal pieces of the row, in order.  Every warp walks its piece once for A and
//                     B; the pieces meet through shared memory inside a block and through the other blocks' shared memory across the
//                     cluster; then every warp walks its piece again (from L2) from the state that really enters it, and writes.  Two
//                     cluster barriers however long the row is.
#include "common.cuh"

namespace pylon {

constexpr int GRU_CLUSTER = 8;
constexpr int GRU_WALKED = 16;   // up to this many tokens a row is walked by one thread per V channels
constexpr int GRU_AHEAD = 8;     // tokens whose loads are on their way at once

// The hardware's exponential and reciprocal (relative errors of a few 2^-23) for bfloat16 rows, the library's for float32 rows.
template <typename T> __device__ __forceinline__ float gru_sigmoid(float x);
template <> __device__ __forceinline__ float gru_sigmoid<float>(float x) { return 1.f / (1.f + expf(-x)); }
template <> __device__ __forceinline__ float gru_sigmoid<__nv_bfloat16>(float x) {
  float e, y;
  asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(e) : "f"(-1.4426950408889634f * x));
  asm("rcp.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(1.f + e));   // 0 where e is infinite
  return y;
}

// Gate and candidate of a token from z + b_z and u.  (Both sides of the candidate are formed: a branch would split the warp at every token.)
template <typename T> __device__ __forceinline__ void gru_unit(float z, float u, float& gate, float& candidate);
template <> __device__ __forceinline__ void gru_unit<float>(float z, float u, float& gate, float& candidate) {
  const float low = gru_sigmoid<float>(u);
  gate = gru_sigmoid<float>(z);
  candidate = u >= 0.f ? u + 0.5f : low;
}
template <> __device__ __forceinline__ void gru_unit<__nv_bfloat16>(float z, float u, float& gate, float& candidate) {
  // The two sigmoids share a reciprocal: with a = 1 + e^-z and b = 1 + e^-u, 1 / (a b) times b and times a.  The exponentials stop at
  // 2^60, so that the product stays in range: a gate below 2^-60 moves nothing.
  float ez, eu, shared;
  asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(ez) : "f"(-1.4426950408889634f * z));
  asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(eu) : "f"(-1.4426950408889634f * u));
  const float a = 1.f + fminf(ez, 1.152921504606847e18f), b = 1.f + fminf(eu, 1.152921504606847e18f);
  asm("rcp.approx.ftz.f32 %0, %1;\n" : "=f"(shared) : "f"(a * b));
  gate = shared * b;
  candidate = u >= 0.f ? u + 0.5f : shared * a;
}

template <typename T, int V> struct GruVector;
template <typename T> struct GruVector<T, 1> { using Type = T; };
template <> struct GruVector<float, 2> { using Type = float2; };
template <> struct GruVector<__nv_bfloat16, 2> { using Type = __nv_bfloat162; };

template <typename T, int V>
__device__ __forceinline__ void gru_load(float (&v)[V], const T* from) {
  using Vector = typename GruVector<T, V>::Type;
  const Vector raw = *reinterpret_cast<const Vector*>(from);
  if constexpr (V == 1) v[0] = to_float<T>(raw);
  else { v[0] = to_float<T>(raw.x); v[1] = to_float<T>(raw.y); }
}
template <typename T, int V>
__device__ __forceinline__ void gru_store(T* to, const float (&v)[V]) {
  using Vector = typename GruVector<T, V>::Type;
  Vector raw;
  if constexpr (V == 1) raw = from_float<T>(v[0]);
  else { raw.x = from_float<T>(v[0]); raw.y = from_float<T>(v[1]); }
  *reinterpret_cast<Vector*>(to) = raw;
}

struct GruParams {
  const void* proj;      // [T, ld] in T, columns [z | x | g]
  long long ld;
  const float* bias;     // [2, C]
  float* state;          // [slots, C]
  const int* q_start;
  const int* slots;
  void* out;             // [T, ld_out] in T
  long long ld_out;
  int channels;
  float factor;
};

template <typename T, int V>
__global__ void __launch_bounds__(128) min_gru_walk_kernel(const GruParams p) {
  grid_dependency_wait();
  allow_dependents();
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V, row = blockIdx.y;
  if (c >= p.channels) return;
  const int first = p.q_start[row], count = p.q_start[row + 1] - first;
  if (count <= 0) return;   // a row without tokens (a padded step): its state stays as it is
  float* slot = p.state + (long long)p.slots[row] * p.channels + c;
  float s[V], bz[V], bx[V];
#pragma unroll
  for (int v = 0; v < V; ++v) { s[v] = slot[v]; bz[v] = p.bias[c + v]; bx[v] = p.bias[p.channels + c + v]; }
  const T* from = (const T*)p.proj + (long long)first * p.ld + c;
  T* to = (T*)p.out + (long long)first * p.ld_out + c;
#pragma unroll 2
  for (int n = 0; n < count; ++n, from += p.ld, to += p.ld_out) {
    float z[V], x[V], g[V], y[V];
    gru_load<T, V>(z, from);
    gru_load<T, V>(x, from + p.channels);
    gru_load<T, V>(g, from + 2 * (long long)p.channels);
#pragma unroll
    for (int v = 0; v < V; ++v) {
      float gate, candidate;
      gru_unit<T>(z[v] + bz[v], x[v] + bx[v], gate, candidate);
      s[v] = fmaf(gate, candidate - s[v], s[v]);
      y[v] = p.factor * s[v] * g[v] * gru_sigmoid<T>(g[v]);
    }
    gru_store<T, V>(to, y);
  }
#pragma unroll
  for (int v = 0; v < V; ++v) slot[v] = s[v];
}

__device__ __forceinline__ void gru_cluster_store(float* own, unsigned rank, float value) {   // into the same place of another block of the cluster
  unsigned address;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;\n" : "=r"(address) : "r"((unsigned)__cvta_generic_to_shared(own)), "r"(rank));
  asm volatile("st.shared::cluster.f32 [%0], %1;\n" ::"r"(address), "f"(value) : "memory");
}
__device__ __forceinline__ void gru_cluster_barrier() {
  asm volatile("barrier.cluster.arrive.release.aligned;\nbarrier.cluster.wait.acquire.aligned;\n" ::: "memory");
}

// Grid (channel groups x GRU_CLUSTER, rows); WARPS x 32 threads.
template <typename T, int V, int WARPS>
__global__ void __launch_bounds__(WARPS * 32) min_gru_cluster_kernel(const GruParams p) {
  constexpr int GROUP = 32 * V;                                   // channels of a cluster
  __shared__ float warp_parts[WARPS][2][GROUP];                   // [warp][A, B][channel]: the warps' pieces
  __shared__ float block_parts[GRU_CLUSTER][2][GROUP];            // the cluster's blocks' pieces, sent by the blocks
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int rank = blockIdx.x % GRU_CLUSTER, c0 = blockIdx.x / GRU_CLUSTER * GROUP, row = blockIdx.y;
  const int mine = lane * V, c = c0 + mine;
  const bool real = c < p.channels;                               // V divides the channels: a lane has all of its channels or none
  grid_dependency_wait();
  allow_dependents();
  const int first = p.q_start[row], count = p.q_start[row + 1] - first;
  if (count <= 0) return;                                         // the whole cluster leaves: nobody waits for it
  const bool one_piece = count <= GRU_WALKED;                     // a decoded row in a step that also brings portions: one warp has it all
  if (one_piece && (rank > 0 || warp > 0)) return;                // (the same for the whole cluster: no barrier is met)
  const int each = one_piece ? count : (count + GRU_CLUSTER * WARPS - 1) / (GRU_CLUSTER * WARPS);
  const int begin = (rank * WARPS + warp) * each, end = begin + each < count ? begin + each : count;   // this warp's tokens (none where the row is used up)
  float* slot = p.state + (long long)p.slots[row] * p.channels + c;
  float s[V], bz[V], bx[V];
#pragma unroll
  for (int v = 0; v < V; ++v) {
    s[v] = real ? slot[v] : 0.f;
    bz[v] = real ? p.bias[c + v] : 0.f;
    bx[v] = real ? p.bias[p.channels + c + v] : 0.f;
  }
  const T* proj = (const T*)p.proj + (long long)first * p.ld + c;
  if (!one_piece) {
    float a[V], b[V];
#pragma unroll
    for (int v = 0; v < V; ++v) { a[v] = 1.f; b[v] = 0.f; }
    if (real) {
      auto take = [&](const float (&z)[V], const float (&x)[V]) {
#pragma unroll
        for (int v = 0; v < V; ++v) {
          float gate, candidate;
          gru_unit<T>(z[v] + bz[v], x[v] + bx[v], gate, candidate);
          b[v] = fmaf(gate, candidate - b[v], b[v]);
          a[v] = fmaf(-gate, a[v], a[v]);
        }
      };
      int n = begin;
      const T* from = proj + n * p.ld;
      for (; n + GRU_AHEAD <= end; n += GRU_AHEAD) {
        float z[GRU_AHEAD][V], x[GRU_AHEAD][V];
#pragma unroll
        for (int k = 0; k < GRU_AHEAD; ++k, from += p.ld) {
          gru_load<T, V>(z[k], from);
          gru_load<T, V>(x[k], from + p.channels);
        }
#pragma unroll
        for (int k = 0; k < GRU_AHEAD; ++k) take(z[k], x[k]);
      }
      for (; n < end; ++n, from += p.ld) {
        float z[V], x[V];
        gru_load<T, V>(z, from);
        gru_load<T, V>(x, from + p.channels);
        take(z, x);
      }
    }
#pragma unroll
    for (int v = 0; v < V; ++v) { warp_parts[warp][0][mine + v] = a[v]; warp_parts[warp][1][mine + v] = b[v]; }
    gru_cluster_barrier();   // every block has started (its shared memory may be written) and has read the slot (the last one writes it)
    // The block's piece, a thread per channel and block of the cluster.
    for (int x = threadIdx.x; x < GROUP * GRU_CLUSTER; x += WARPS * 32) {
      const int channel = x % GROUP;
      float block_a = 1.f, block_b = 0.f;
#pragma unroll
      for (int w = 0; w < WARPS; ++w) {
        const float wa = warp_parts[w][0][channel];
        block_b = fmaf(wa, block_b, warp_parts[w][1][channel]);
        block_a *= wa;
      }
      gru_cluster_store(&block_parts[rank][0][channel], x / GROUP, block_a);
      gru_cluster_store(&block_parts[rank][1][channel], x / GROUP, block_b);
    }
    gru_cluster_barrier();   // what every block sent is there
#pragma unroll
    for (int v = 0; v < V; ++v) {
      for (int r = 0; r < rank; ++r) s[v] = fmaf(block_parts[r][0][mine + v], s[v], block_parts[r][1][mine + v]);
      for (int w = 0; w < warp; ++w) s[v] = fmaf(warp_parts[w][0][mine + v], s[v], warp_parts[w][1][mine + v]);
    }
  }
  if (!real || begin >= end) return;
  auto give = [&](T* to, const float (&z)[V], const float (&x)[V], const float (&g)[V]) {
    float y[V];
#pragma unroll
    for (int v = 0; v < V; ++v) {
      float gate, candidate;
      gru_unit<T>(z[v] + bz[v], x[v] + bx[v], gate, candidate);
      s[v] = fmaf(gate, candidate - s[v], s[v]);
      y[v] = p.factor * s[v] * g[v] * gru_sigmoid<T>(g[v]);
    }
    gru_store<T, V>(to, y);
  };
  int n = begin;
  const T* from = proj + n * p.ld;
  T* to = (T*)p.out + (long long)(first + n) * p.ld_out + c;
  for (; n + GRU_AHEAD <= end; n += GRU_AHEAD) {
    float z[GRU_AHEAD][V], x[GRU_AHEAD][V], g[GRU_AHEAD][V];
#pragma unroll
    for (int k = 0; k < GRU_AHEAD; ++k, from += p.ld) {
      gru_load<T, V>(z[k], from);
      gru_load<T, V>(x[k], from + p.channels);
      gru_load<T, V>(g[k], from + 2 * p.channels);
    }
#pragma unroll
    for (int k = 0; k < GRU_AHEAD; ++k, to += p.ld_out) give(to, z[k], x[k], g[k]);
  }
  for (; n < end; ++n, from += p.ld, to += p.ld_out) {
    float z[V], x[V], g[V];
    gru_load<T, V>(z, from);
    gru_load<T, V>(x, from + p.channels);
    gru_load<T, V>(g, from + 2 * p.channels);
    give(to, z, x, g);
  }
  if (end == count) {   // the warp that has walked the row's last token
#pragma unroll
    for (int v = 0; v < V; ++v) slot[v] = s[v];
  }
}

template <typename T, int V>
static int launch_min_gru(const GruParams& p, int num_rows, int max_q, cudaStream_t stream) {
  constexpr int WARPS = 16;
  if (max_q <= GRU_WALKED) {
    launch_dependent(min_gru_walk_kernel<T, V>, dim3((unsigned)((p.channels / V + 127) / 128), (unsigned)num_rows), dim3(128), 0, stream, p);
  } else {
    const int groups = (p.channels + 32 * V - 1) / (32 * V);
    launch_dependent_cluster(min_gru_cluster_kernel<T, V, WARPS>, dim3((unsigned)(groups * GRU_CLUSTER), (unsigned)num_rows), dim3(WARPS * 32), 0, stream, GRU_CLUSTER, p);
  }
  PYLON_CHECK_LAUNCH("min_gru");
}

}  // namespace pylon

using namespace pylon;

// proj [T, ld] in dtype, columns [z | x | g] of `channels` each; bias float32 [2, channels]; state float32 [slots, channels]; q_start int32
// [num_rows + 1]; slots int32 [num_rows]; out [T, ld_out] in dtype; max_q: the most tokens a row brings (an upper bound is fine).
extern "C" int pylon_min_gru(const void* proj, long long ld, const float* bias, float* state, const int* q_start, const int* slots, void* out,
                             long long ld_out, int channels, float factor, int num_rows, int max_q, int dtype, cudaStream_t stream) {
  if (num_rows <= 0 || max_q <= 0) return 0;
  if (channels < 1 || ld < 3LL * channels || ld_out < channels || num_rows > 65535) PYLON_REFUSE("min_gru: %d channels, rows %lld / %lld apart, %d rows", channels, ld, ld_out, num_rows);
  const GruParams p{proj, ld, bias, state, q_start, slots, out, ld_out, channels, factor};
  const size_t pair = dtype == PYLON_DTYPE_F32 ? 8 : 4;
  const bool pairs = channels % 2 == 0 && ld % 2 == 0 && ld_out % 2 == 0 && (uintptr_t)proj % pair == 0 && (uintptr_t)out % pair == 0;
  if (dtype == PYLON_DTYPE_F32) return pairs ? launch_min_gru<float, 2>(p, num_rows, max_q, stream) : launch_min_gru<float, 1>(p, num_rows, max_q, stream);
  if (dtype == PYLON_DTYPE_BF16) return pairs ? launch_min_gru<__nv_bfloat16, 2>(p, num_rows, max_q, stream) : launch_min_gru<__nv_bfloat16, 1>(p, num_rows, max_q, stream);
  PYLON_REFUSE("min_gru: unknown dtype %d", dtype);
}
