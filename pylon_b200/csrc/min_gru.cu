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
//                     the product A of its (1 - z) is the factor on what enters it: S_out = A S_in + B.  A thread-block cluster takes
//                     a row's 32 V channels; a warp takes TOKENS neighbouring tokens of them, a block 8 neighbouring warps' pieces,
//                     the cluster its blocks' pieces one after the other.  Every thread reads its tokens' gates and candidates once
//                     and keeps them in registers; pieces meet through shared memory inside the block and through the other blocks'
//                     shared memory across it (one cluster barrier per 8 x 8 x TOKENS tokens); then every thread walks its tokens again
//                     from the state that really enters them.  The row is read once and written once.
#include "common.cuh"

namespace pylon {

constexpr int GRU_WARPS = 8, GRU_CLUSTER = 8;

// The hardware's exponential and division (relative errors of a few 2^-23 for the sizes met here) for bfloat16 rows, the library's for
// float32 rows.
template <typename T> __device__ __forceinline__ float gru_sigmoid(float x);
template <> __device__ __forceinline__ float gru_sigmoid<float>(float x) { return 1.f / (1.f + expf(-x)); }
template <> __device__ __forceinline__ float gru_sigmoid<__nv_bfloat16>(float x) { return __fdividef(1.f, 1.f + __expf(-x)); }

template <typename T>
__device__ __forceinline__ float gru_candidate(float u) { return u >= 0.f ? u + 0.5f : gru_sigmoid<T>(u); }

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
      s[v] = fmaf(gru_sigmoid<T>(z[v] + bz[v]), gru_candidate<T>(x[v] + bx[v]) - s[v], s[v]);
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

// Grid (channel groups x GRU_CLUSTER, rows).
template <typename T, int V, int TOKENS>
__global__ void __launch_bounds__(GRU_WARPS * 32) min_gru_cluster_kernel(const GruParams p) {
  constexpr int GROUP = 32 * V;                                   // channels of a cluster
  __shared__ float warp_parts[2][GRU_WARPS][2][GROUP];            // [round parity][warp][A, B][channel]: the warps' pieces
  __shared__ float block_parts[2][GRU_CLUSTER][2][GROUP];         // the cluster's blocks' pieces, sent by the blocks
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int rank = blockIdx.x % GRU_CLUSTER, c0 = blockIdx.x / GRU_CLUSTER * GROUP, row = blockIdx.y;
  const int mine = lane * V, c = c0 + mine;
  const bool real = c < p.channels;                               // V divides the channels: a lane has all of its channels or none
  grid_dependency_wait();
  allow_dependents();
  const int first = p.q_start[row], count = p.q_start[row + 1] - first;
  if (count <= 0) return;                                         // the whole cluster leaves: nobody waits for it
  const bool one_piece = count <= TOKENS;                         // a decoded row in a step that also brings portions: one warp has it all
  if (one_piece && (rank > 0 || warp > 0)) return;                // (the same for the whole cluster: no barrier is met)
  float* slot = p.state + (long long)p.slots[row] * p.channels + c;
  float carry[V], bz[V], bx[V];
#pragma unroll
  for (int v = 0; v < V; ++v) {
    carry[v] = real ? slot[v] : 0.f;
    bz[v] = real ? p.bias[c + v] : 0.f;
    bx[v] = real ? p.bias[p.channels + c + v] : 0.f;
  }
  if (!one_piece) gru_cluster_barrier();   // every block has started (its shared memory may be written) and has read the slot (rank 0 may write it)
  constexpr int BLOCK_TOKENS = GRU_WARPS * TOKENS, ROUND_TOKENS = GRU_CLUSTER * BLOCK_TOKENS;
  for (int round = 0, base = 0; base < count; ++round, base += ROUND_TOKENS) {
    const int parity = round & 1;
    const int begin = base + rank * BLOCK_TOKENS + warp * TOKENS;   // this warp's tokens: begin .. begin + TOKENS - 1, as far as the row goes
    const T* from = (const T*)p.proj + (long long)(first + begin) * p.ld + c;
    float z[TOKENS][V], cand[TOKENS][V], g[TOKENS][V];
#pragma unroll
    for (int n = 0; n < TOKENS; ++n) {
      if (real && begin + n < count) {
        gru_load<T, V>(z[n], from + n * p.ld);
        gru_load<T, V>(cand[n], from + n * p.ld + p.channels);
        gru_load<T, V>(g[n], from + n * p.ld + 2 * (long long)p.channels);
      } else {
#pragma unroll
        for (int v = 0; v < V; ++v) { z[n][v] = -INFINITY; cand[n][v] = 0.f; g[n][v] = 0.f; }   // a gate that is shut: the state passes unchanged
      }
    }
    float a[V], b[V];
#pragma unroll
    for (int v = 0; v < V; ++v) { a[v] = 1.f; b[v] = 0.f; }
#pragma unroll
    for (int n = 0; n < TOKENS; ++n)
#pragma unroll
      for (int v = 0; v < V; ++v) {
        z[n][v] = gru_sigmoid<T>(z[n][v] + bz[v]);
        cand[n][v] = gru_candidate<T>(cand[n][v] + bx[v]);
        b[v] = fmaf(z[n][v], cand[n][v] - b[v], b[v]);
        a[v] = fmaf(-z[n][v], a[v], a[v]);
      }
    float s[V];
    if (one_piece) {
#pragma unroll
      for (int v = 0; v < V; ++v) { s[v] = carry[v]; carry[v] = fmaf(a[v], carry[v], b[v]); }
    } else {
#pragma unroll
      for (int v = 0; v < V; ++v) { warp_parts[parity][warp][0][mine + v] = a[v]; warp_parts[parity][warp][1][mine + v] = b[v]; }
      __syncthreads();
      // The block's piece, a thread per channel, into every block of the cluster.
      if (threadIdx.x < GROUP) {
        float block_a = 1.f, block_b = 0.f;
#pragma unroll
        for (int w = 0; w < GRU_WARPS; ++w) {
          const float wa = warp_parts[parity][w][0][threadIdx.x];
          block_b = fmaf(wa, block_b, warp_parts[parity][w][1][threadIdx.x]);
          block_a *= wa;
        }
#pragma unroll
        for (int r = 0; r < GRU_CLUSTER; ++r) {
          gru_cluster_store(&block_parts[parity][rank][0][threadIdx.x], r, block_a);
          gru_cluster_store(&block_parts[parity][rank][1][threadIdx.x], r, block_b);
        }
      }
      // One barrier a round: the buffers of this round are written again two rounds on, behind the next round's barrier, which every block
      // reaches only after it has read them.
      gru_cluster_barrier();
#pragma unroll
      for (int v = 0; v < V; ++v) {
        float enters = carry[v];
#pragma unroll
        for (int r = 0; r < GRU_CLUSTER; ++r) {
          if (r == rank) s[v] = enters;
          enters = fmaf(block_parts[parity][r][0][mine + v], enters, block_parts[parity][r][1][mine + v]);
        }
        carry[v] = enters;   // what leaves the round
        for (int w = 0; w < warp; ++w) s[v] = fmaf(warp_parts[parity][w][0][mine + v], s[v], warp_parts[parity][w][1][mine + v]);
      }
    }
    T* to = (T*)p.out + (long long)(first + begin) * p.ld_out + c;
#pragma unroll
    for (int n = 0; n < TOKENS; ++n) {
      float y[V];
#pragma unroll
      for (int v = 0; v < V; ++v) {
        s[v] = fmaf(z[n][v], cand[n][v] - s[v], s[v]);
        y[v] = p.factor * s[v] * g[n][v] * gru_sigmoid<T>(g[n][v]);
      }
      if (real && begin + n < count) gru_store<T, V>(to + n * p.ld_out, y);
    }
  }
  if (rank == 0 && warp == 0 && real) {
#pragma unroll
    for (int v = 0; v < V; ++v) slot[v] = carry[v];
  }
}

template <typename T, int V>
static int launch_min_gru(const GruParams& p, int num_rows, int max_q, cudaStream_t stream) {
  constexpr int TOKENS = V == 2 ? 8 : 16;
  if (max_q <= TOKENS) {
    launch_dependent(min_gru_walk_kernel<T, V>, dim3((unsigned)((p.channels / V + 127) / 128), (unsigned)num_rows), dim3(128), 0, stream, p);
  } else {
    const int groups = (p.channels + 32 * V - 1) / (32 * V);
    launch_dependent_cluster(min_gru_cluster_kernel<T, V, TOKENS>, dim3((unsigned)(groups * GRU_CLUSTER), (unsigned)num_rows), dim3(GRU_WARPS * 32), 0, stream, GRU_CLUSTER, p);
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
