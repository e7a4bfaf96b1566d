// A mixture of experts: every token goes through `top` of `experts` small gated feed-forwards, chosen by a router.
//
//     z       = W_r h + b_r                       (float32, whatever the compute dtype)
//     chosen  = the `top` largest z (the lower index wins a tie),   share = softmax over the chosen z only
//     out     = sum over chosen e of share_e * W_down,e (act(W_gate,e h) * (W_up,e h))
//
// A second way of routing (RouteScored): the scores are s = sigmoid(z); the choice goes by s + correction (a learnt vector), and only
// among the experts of the `keep` best of `groups` equal groups of neighbours, a group's worth being the sum of its two largest choice
// scores (of its one, if it has one expert); share = s of the chosen (without the correction), divided by their sum plus share_eps.  The
// router matrix may have `extra` rows behind the experts': their logits leave as sigmoid(z) in extra_out [T, extra] (the gate of an
// expert that every token goes through, say).  An ungated expert is W_down act(W_up h): the first product applies act itself.
//
// The shares may also stay the plain scores (normalize 0), and a share may weigh what an expert reads instead of what it gives:
// out = sum of expert_e(share_e * h).  An expert's first product is linear, so its sums are multiplied by the slot's share before the
// unit (slot_share, written by the plan), and the rows are then added up as they are.  Activation 4 is the clamped gated unit:
// g = min(gate, limit), u = clamp(up, -limit, limit), g * sigmoid(alpha * g) * (u + 1).
//
// A third way (RouteScored.on 2): the scores are the softmax over all of the router's outputs; a group may be worth its largest choice
// score; the shares may be times a factor.  The router's last outputs may be experts that hand their input back: whoever chooses one gets
// chosen -1 and no slot, and same_share [T] receives the shares of those a token chose, for whoever adds share * h.  And behind the `top`
// choices every token may have `always` more, the pieces of an expert that every token goes through, with a share of one; their matrices
// lie behind the experts'.  A token's choices and shares then lie top + always apart.
//
// Nothing here needs the host to know how many tokens an expert got, so the step stays one sequence of launches (and
// can be captured): the (token, choice) pairs are sorted by expert into row tiles of ROWS slots, every expert's span
// padded to whole tiles, and the grouped products run over the most tiles there can be; a tile beyond the last one, and
// a slot of padding inside a tile, is skipped.
//
//   experts_route     router logits, the top choices, their shares: a block per token in a step of few tokens, else a block per four
//   experts_plan      one block: tokens per expert, the experts' first tiles, a slot for every pair
//   experts_product   a block per (row tile, column tile): rows gathered by slot, the expert's matrix, float32 sums in a
//                     fixed order of k; with GLU the gate and up tiles side by side and act(gate) * up written
//   experts_product_mma   the same on tensor cores (bfloat16, mma.sync m16n8k16), the matrices through a ring of cp.async stages
//   experts_stream    the products of a step of few tokens where the matrices' rows can be fetched by TMA: as experts_product_mma, the
//                     matrices as 64 x 64 boxes in a ring that TMA fills, the rows gathered into it beside them
//   experts_sort_rows the tokens' rows copied into the order of their slots, for a step of many tokens: its products are the
//                     grouped form of the tcgen05 kernel (gemm_tcgen05.cu) over row tiles of 128 slots
//   experts_gather    out[t] = sum_k share[t, k] * y[slot(t, k)], float32
// A row's sums do not depend on where in a tile it lies or what else is in the batch.
#include "common.cuh"
#include <cuda.h>

#include <mutex>
#include <unordered_map>

namespace pylon {

constexpr int EXPERT_ROWS = 32;   // slots to a row tile

__device__ __forceinline__ float expert_activation(float x, int kind) {
  if (kind == 0) return x / (1.f + expf(-x));
  if (kind == 1) return fmaxf(x, 0.f);
  if (kind == 3) return 0.5f * x * (1.f + erff(x * 0.7071067811865476f));   // gelu, exact form
  return 0.5f * x * (1.f + tanhf(0.7978845608028654f * (x + 0.044715f * x * x * x)));
}

// A gated unit: act(gate) * up, or (kind 4) the clamped one.
__device__ __forceinline__ float expert_unit(float g, float u, int kind, float limit, float alpha) {
  if (kind == 4) {
    g = fminf(g, limit);
    return g / (1.f + expf(-alpha * g)) * (fminf(fmaxf(u, -limit), limit) + 1.f);
  }
  return expert_activation(g, kind) * u;
}

// The row of w that holds column n of the gate (half 0) or of the up projection (half 1): the two halves one after the other, or
// (interleaved) alternating in groups of 8 rows, the layout the tcgen05 product's gated epilogue takes.
__device__ __forceinline__ long long glu_row(int n, int half, int n_out, int interleaved) {
  return interleaved ? ((long long)(n >> 3) << 4) + (half << 3) + (n & 7) : (long long)half * n_out + n;
}

// The `top` largest of a token's logits (the lower index wins a tie) and the softmax over just those; one warp.  logits is spoilt.
__device__ __forceinline__ void route_choose(float* logits, int* __restrict__ chosen, float* __restrict__ share, long long t, int experts, int top,
                                             int per, int lane) {
  float first = 0.f, total = 0.f;
  for (int k = 0; k < top; ++k) {
    float best = -INFINITY;
    int where = 0x7fffffff;
    for (int e = lane; e < experts; e += 32) {
      const float z = logits[e];
      if (z > best) { best = z; where = e; }   // strictly larger: a lane keeps its lowest index
    }
    for (int offset = 16; offset > 0; offset >>= 1) {
      const float other = __shfl_xor_sync(0xffffffffu, best, offset);
      const int other_where = __shfl_xor_sync(0xffffffffu, where, offset);
      if (other > best || (other == best && other_where < where)) { best = other; where = other_where; }
    }
    if (where == 0x7fffffff) where = 0;   // every logit was NaN or -inf: still a valid expert
    if (k == 0) first = best;
    const float weight = expf(best - first);
    total += weight;
    if (lane == 0) {
      chosen[t * per + k] = where;
      share[t * per + k] = weight;
      logits[where] = -INFINITY;
    }
    __syncwarp();
  }
  const float inv = 1.f / total;
  if (lane < top) share[t * per + lane] *= inv;
  for (int k = 32 + lane; k < top; k += 32) share[t * per + k] *= inv;
}

// How the scores are made and the choice is restricted; correction null: none; groups 0: no groups.
struct RouteScored {
  int on;                    // 0: the softmax form above, the rest is unused then; 1: sigmoids; 2: the softmax over all of the router's outputs
  const float* correction;   // [experts] or null
  int groups, keep;
  float share_eps;
  int normalize;             // 0: the shares are the scores as they are
  int extra;                 // rows of the router behind the experts'
  float* extra_out;          // [T, extra]
  int group_best;            // a group is worth its largest choice score instead of the sum of its two largest
  float share_scale;         // on the shares
  int real;                  // outputs from here on are experts that hand their input back: chosen is -1, the share joins same_share
  float* same_share;         // [T] or null
};

// One warp.  logits [experts + extra] holds z; choice [experts] and worth [groups] are scratch.
__device__ __forceinline__ void route_choose_scored(float* logits, float* choice, float* worth, int* __restrict__ chosen, float* __restrict__ share,
                                                    long long t, int experts, int top, int per, int lane, const RouteScored& mode) {
  for (int x = lane; x < mode.extra; x += 32) mode.extra_out[t * mode.extra + x] = 1.f / (1.f + expf(-logits[experts + x]));
  float largest = 0.f, over = 1.f;   // of the softmax over all
  if (mode.on == 2) {
    largest = -INFINITY;
    for (int e = lane; e < experts; e += 32) largest = fmaxf(largest, logits[e]);
    largest = warp_max(largest);
    over = 0.f;
    for (int e = lane; e < experts; e += 32) over += expf(logits[e] - largest);
    over = warp_sum(over);
  }
  for (int e = lane; e < experts; e += 32) {
    const float s = mode.on == 2 ? expf(logits[e] - largest) / over : 1.f / (1.f + expf(-logits[e]));
    logits[e] = s;
    choice[e] = s + (mode.correction != nullptr ? mode.correction[e] : 0.f);
  }
  __syncwarp();
  if (mode.groups > 0) {
    const int size = experts / mode.groups;
    for (int g = lane; g < mode.groups; g += 32) {
      float first = -INFINITY, second = -INFINITY;
      for (int i = 0; i < size; ++i) {
        const float c = choice[g * size + i];
        if (c > first) { second = first; first = c; }
        else if (c > second) second = c;
      }
      worth[g] = size > 1 && !mode.group_best ? first + second : first;
    }
    __syncwarp();
    for (int k = 0; k < mode.keep; ++k) {   // the best group not yet kept, the lower index on a tie; a kept group's worth becomes +inf
      float best = -INFINITY;
      int where = 0x7fffffff;
      for (int g = lane; g < mode.groups; g += 32) {
        const float w = worth[g];
        if (w != INFINITY && (w > best || where == 0x7fffffff)) { best = w; where = g; }
      }
      for (int offset = 16; offset > 0; offset >>= 1) {
        const float other = __shfl_xor_sync(0xffffffffu, best, offset);
        const int other_where = __shfl_xor_sync(0xffffffffu, where, offset);
        if (other_where != 0x7fffffff && (where == 0x7fffffff || other > best || (other == best && other_where < where))) { best = other; where = other_where; }
      }
      if (lane == 0 && where != 0x7fffffff) worth[where] = INFINITY;
      __syncwarp();
    }
    for (int e = lane; e < experts; e += 32)
      if (worth[e / size] != INFINITY) choice[e] = -INFINITY;
    __syncwarp();
  }
  float total = 0.f, handed_back = 0.f;
  for (int k = 0; k < top; ++k) {
    float best = -INFINITY;
    int where = 0x7fffffff;
    for (int e = lane; e < experts; e += 32) {
      const float c = choice[e];
      if (c > best) { best = c; where = e; }
    }
    for (int offset = 16; offset > 0; offset >>= 1) {
      const float other = __shfl_xor_sync(0xffffffffu, best, offset);
      const int other_where = __shfl_xor_sync(0xffffffffu, where, offset);
      if (other > best || (other == best && other_where < where)) { best = other; where = other_where; }
    }
    if (where == 0x7fffffff) where = 0;
    const float s = logits[where];
    const bool same = where >= mode.real;
    total += s;
    if (same) handed_back += s;
    if (lane == 0) {
      chosen[t * per + k] = same ? -1 : where;
      share[t * per + k] = mode.normalize ? s : s * mode.share_scale;
      choice[where] = -INFINITY;
    }
    __syncwarp();
  }
  const float inv = mode.normalize ? mode.share_scale / (total + mode.share_eps) : mode.share_scale;
  if (mode.same_share != nullptr && lane == 0) mode.same_share[t] = handed_back * inv;
  if (!mode.normalize) return;
  if (lane < top) share[t * per + lane] *= inv;
  for (int k = 32 + lane; k < top; k += 32) share[t * per + k] *= inv;
}

// h [T, width] in T; router float32 [experts, width]; bias float32 [experts] or null.  chosen int32 [T, top], share float32 [T, top].
// A block of four warps takes TOKENS tokens, so that a router value it has loaded serves all of them; a warp takes a quarter of the
// columns.  A thread takes V neighbouring columns at a time (V 4 where the rows are whole pieces of it, else 1; by the sizes alone): warp k's
// lane l adds up the columns V (128 i + 32 k + l) .. + V - 1 in order of i, its 32 lanes' sums are added by a butterfly, and the four warps'
// sums in order of k.  So a token's logits, and with them its choice, do not depend on how many tokens the step has.
// Shared memory: TOKENS * (4 * ROUTE_SIDE + what a token takes) floats.
template <typename T, int V>
__device__ __forceinline__ void route_load(float (&x)[V], const T* from) {
  if constexpr (V == 1) x[0] = to_float<T>(from[0]);
  else if constexpr (sizeof(T) == 4) {
    const float4 raw = *reinterpret_cast<const float4*>(from);
    x[0] = raw.x; x[1] = raw.y; x[2] = raw.z; x[3] = raw.w;
  } else {
    const uint2 raw = *reinterpret_cast<const uint2*>(from);
    const float2 low = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x)), high = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    x[0] = low.x; x[1] = low.y; x[2] = high.x; x[3] = high.y;
  }
}

constexpr int ROUTE_SIDE = 8;   // router rows side by side at most: the tokens' rows are read once per so many

// The logits of the block's tokens for router rows e0 .. e0 + SIDE - 1 (those below `rows`).
template <typename T, int TOKENS, int V, int SIDE>
__device__ __forceinline__ void route_logits(const T* __restrict__ h, long long ld, const float* __restrict__ router, const float* __restrict__ bias, float* parts,
                                             float* logits, int per_token, int t0, int num_tokens, int width, int e0, int rows, int experts) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float acc[TOKENS][SIDE];
#pragma unroll
  for (int i = 0; i < TOKENS; ++i)
#pragma unroll
    for (int j = 0; j < SIDE; ++j) acc[i][j] = 0.f;
#pragma unroll(TOKENS == 1 ? 4 : 2)
  for (int c = V * threadIdx.x; c < width; c += V * 128) {
    float x[TOKENS][V], r[SIDE][V];
#pragma unroll
    for (int i = 0; i < TOKENS; ++i) route_load<T, V>(x[i], h + (long long)(t0 + i < num_tokens ? t0 + i : t0) * ld + c);
#pragma unroll
    for (int j = 0; j < SIDE; ++j) route_load<float, V>(r[j], router + (long long)(e0 + j < rows ? e0 + j : e0) * width + c);
#pragma unroll
    for (int i = 0; i < TOKENS; ++i)
#pragma unroll
      for (int j = 0; j < SIDE; ++j)
#pragma unroll
        for (int v = 0; v < V; ++v) acc[i][j] = fmaf(x[i][v], r[j][v], acc[i][j]);
  }
#pragma unroll
  for (int i = 0; i < TOKENS; ++i)
#pragma unroll
    for (int j = 0; j < SIDE; ++j) {
      const float z = warp_sum(acc[i][j]);
      if (lane == 0) parts[(warp * TOKENS + i) * SIDE + j] = z;
    }
  __syncthreads();
  if (threadIdx.x < TOKENS * SIDE) {
    const int i = threadIdx.x / SIDE, j = threadIdx.x % SIDE;
    if (e0 + j < rows)
      logits[i * per_token + e0 + j] = ((parts[i * SIDE + j] + parts[(TOKENS + i) * SIDE + j]) + parts[(2 * TOKENS + i) * SIDE + j]) + parts[(3 * TOKENS + i) * SIDE + j] +
                                       (bias != nullptr && e0 + j < experts ? bias[e0 + j] : 0.f);
  }
  __syncthreads();
}

template <typename T, int TOKENS, int V>
__global__ void __launch_bounds__(128) experts_route_kernel(const T* __restrict__ h, long long ld, const float* __restrict__ router, const float* __restrict__ bias,
                                                            int* __restrict__ chosen, float* __restrict__ share, int width, int experts, int top, int num_tokens,
                                                            int always, RouteScored mode) {
  extern __shared__ float route_shared[];
  const int rows = experts + mode.extra;                                        // rows of the router
  const int per_token = rows + (mode.on ? experts + mode.groups : 0);           // logits, then with mode.on choice scores and the groups' worths
  float* parts = route_shared;                                                  // [4][TOKENS][ROUTE_SIDE]
  float* logits = route_shared + 4 * TOKENS * ROUTE_SIDE;                       // [TOKENS][per_token]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t0 = blockIdx.x * TOKENS;
  if (TOKENS == 1) {   // the router's rows are nobody's work: on their way to L2 before the wait for the kernel ahead
    const long long bytes = (long long)rows * width * 4;
    for (long long at = (long long)threadIdx.x * 128; at < bytes; at += 128 * 128) asm volatile("prefetch.global.L2 [%0];\n" ::"l"((const char*)router + at));
  }
  grid_dependency_wait();
  allow_dependents();
  int e0 = 0;
  for (; rows - e0 > ROUTE_SIDE / 2; e0 += ROUTE_SIDE)
    route_logits<T, TOKENS, V, ROUTE_SIDE>(h, ld, router, bias, parts, logits, per_token, t0, num_tokens, width, e0, rows, experts);
  if (e0 < rows && rows - e0 <= 2)        // the few rows that are left
    route_logits<T, TOKENS, V, 2>(h, ld, router, bias, parts, logits, per_token, t0, num_tokens, width, e0, rows, experts);
  else if (e0 < rows)
    route_logits<T, TOKENS, V, ROUTE_SIDE / 2>(h, ld, router, bias, parts, logits, per_token, t0, num_tokens, width, e0, rows, experts);
  for (int i = warp; i < TOKENS && t0 + i < num_tokens; i += 4) {
    float* mine = logits + i * per_token;
    const int per = top + always;
    if (mode.on) route_choose_scored(mine, mine + rows, mine + rows + experts, chosen, share, t0 + i, experts, top, per, lane, mode);
    else route_choose(mine, chosen, share, t0 + i, experts, top, per, lane);
    for (int k = lane; k < always; k += 32) {   // the pieces every token goes through lie behind the experts
      chosen[(long long)(t0 + i) * per + top + k] = mode.real + k;
      share[(long long)(t0 + i) * per + top + k] = 1.f;
    }
  }
}

// One block.  chosen [pairs], `per` to a token, -1: none; the last `always` experts are every token's.  slot_of [pairs] out; source [max_slots] out: the pair in a slot, or -1; tile_expert [max_tiles] out:
// the expert of a row tile of tile_rows slots, or -1; slot_share [max_slots] out, or null: the share of the pair in a slot.  Shared memory: 2 * experts + 1 ints.
__global__ void experts_plan_kernel(const int* __restrict__ chosen, int* __restrict__ slot_of, int* __restrict__ source,
                                    int* __restrict__ tile_expert, int pairs, int experts, int max_slots, int max_tiles, int tile_rows,
                                    const float* __restrict__ share, float* __restrict__ slot_share, int per, int always) {
  extern __shared__ int plan[];
  grid_dependency_wait();
  allow_dependents();
  int* count = plan;                 // tokens per expert, then the next free slot of each
  int* first = plan + experts;       // first slot of each expert, [experts + 1]
  for (int e = threadIdx.x; e < experts; e += blockDim.x) count[e] = 0;
  for (int s = threadIdx.x; s < max_slots; s += blockDim.x) {
    source[s] = -1;
    if (slot_share) slot_share[s] = 0.f;
  }
  for (int tile = threadIdx.x; tile < max_tiles; tile += blockDim.x) tile_expert[tile] = -1;
  __syncthreads();
  const int real = experts - always;   // the pieces every token goes through: their tokens in order, nothing to count
  for (int i = threadIdx.x; i < pairs; i += blockDim.x) {
    const int e = chosen[i];
    if (e >= 0 && e < real) atomicAdd(&count[e], 1);
  }
  for (int k = threadIdx.x; k < always; k += blockDim.x) count[real + k] = pairs / per;
  __syncthreads();
  if (threadIdx.x == 0) {
    int at = 0;
    for (int e = 0; e < experts; ++e) {
      first[e] = at;
      at += (count[e] + tile_rows - 1) / tile_rows * tile_rows;
    }
    first[experts] = at;
  }
  __syncthreads();
  for (int e = threadIdx.x; e < experts; e += blockDim.x) {
    for (int tile = first[e] / tile_rows; tile < first[e + 1] / tile_rows; ++tile) tile_expert[tile] = e;
    count[e] = first[e];
  }
  __syncthreads();
  for (int i = threadIdx.x; i < pairs; i += blockDim.x) {
    const int e = chosen[i];
    if (e < 0) {   // handed back: no slot
      slot_of[i] = -1;
      continue;
    }
    const int slot = e >= real ? first[e] + i / per : atomicAdd(&count[e], 1);   // the order inside an expert's span does not matter: rows do not see each other
    slot_of[i] = slot;
    source[slot] = i;
    if (slot_share) slot_share[slot] = share[i];
  }
}

// out[slot, n] = sum_k a[row(slot), k] * w[expert, n, k].  row(slot) = source[slot] / divide when `gathered`, else slot.
// GLU: w is [experts, 2 * n_out, k] (gate rows, then up rows) and out[slot, n] = act(gate) * up in T; else out is float32.
// Block 256 threads = 16 x 16; tile EXPERT_ROWS x 64; a thread owns 2 rows x 4 columns.
template <typename T, bool GLU>
__global__ void __launch_bounds__(256) experts_product_kernel(const T* __restrict__ a, long long lda, const T* __restrict__ w,
                                                              const int* __restrict__ source, const int* __restrict__ tile_expert,
                                                              int gathered, int divide, void* __restrict__ out_v, int n_out, int k_size,
                                                              int kind, int interleaved, int act_out,
                                                              const float* __restrict__ slot_share, float limit, float alpha) {
  constexpr int TN = 64, TK = 16;
  __shared__ float a_tile[EXPERT_ROWS][TK + 1];
  __shared__ float b_tile[GLU ? 2 : 1][TN][TK + 1];
  __shared__ int rows[EXPERT_ROWS];
  grid_dependency_wait();
  allow_dependents();
  const int tile = blockIdx.y;
  const int expert = tile_expert[tile];
  if (expert < 0) return;
  const int n0 = blockIdx.x * TN;
  if (threadIdx.x < EXPERT_ROWS) {
    const int pair = source[tile * EXPERT_ROWS + threadIdx.x];
    rows[threadIdx.x] = pair < 0 ? -1 : (gathered ? pair / divide : tile * EXPERT_ROWS + threadIdx.x);
  }
  __syncthreads();
  const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;
  const long long w_rows = GLU ? 2LL * n_out : n_out;
  const T* w_mine = w + (long long)expert * w_rows * k_size;
  float acc[GLU ? 2 : 1][2][4];
#pragma unroll
  for (int g = 0; g < (GLU ? 2 : 1); ++g)
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[g][i][j] = 0.f;
  for (int k0 = 0; k0 < k_size; k0 += TK) {
    for (int x = threadIdx.x; x < EXPERT_ROWS * TK; x += 256) {
      const int r = x / TK, c = x % TK;
      const int row = rows[r];
      a_tile[r][c] = (row >= 0 && k0 + c < k_size) ? to_float<T>(a[(long long)row * lda + k0 + c]) : 0.f;
    }
    for (int x = threadIdx.x; x < TN * TK; x += 256) {
      const int r = x / TK, c = x % TK;
      const bool inside = n0 + r < n_out && k0 + c < k_size;
      b_tile[0][r][c] = inside ? to_float<T>(w_mine[glu_row(n0 + r, 0, n_out, GLU && interleaved) * k_size + k0 + c]) : 0.f;
      if (GLU) b_tile[1][r][c] = inside ? to_float<T>(w_mine[glu_row(n0 + r, 1, n_out, interleaved) * k_size + k0 + c]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < TK; ++c) {
      float av[2], bv[GLU ? 2 : 1][4];
#pragma unroll
      for (int i = 0; i < 2; ++i) av[i] = a_tile[ty * 2 + i][c];
#pragma unroll
      for (int g = 0; g < (GLU ? 2 : 1); ++g)
#pragma unroll
        for (int j = 0; j < 4; ++j) bv[g][j] = b_tile[g][tx * 4 + j][c];
#pragma unroll
      for (int g = 0; g < (GLU ? 2 : 1); ++g)
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) acc[g][i][j] = fmaf(av[i], bv[g][j], acc[g][i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int r = ty * 2 + i;
    if (rows[r] < 0) continue;
    const long long slot = (long long)tile * EXPERT_ROWS + r;
    const float reads = GLU && slot_share ? slot_share[slot] : 1.f;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= n_out) continue;
      if (GLU) ((T*)out_v)[slot * n_out + n] = from_float<T>(expert_unit(reads * acc[0][i][j], reads * acc[GLU ? 1 : 0][i][j], kind, limit, alpha));
      else if (act_out) ((T*)out_v)[slot * n_out + n] = from_float<T>(expert_activation(acc[0][i][j], kind));   // an ungated expert's first product
      else ((float*)out_v)[slot * n_out + n] = acc[0][i][j];
    }
  }
}

// The same product on tensor cores for bfloat16: a block of four warps takes a row tile of 32 slots x 64 columns (with GLU: 64 gate and
// the 64 matching up columns); warp w owns columns 16 w .. 16 w + 15 of the tile, both 16-row halves.  Steps of 64 along k through a ring
// of four shared-memory stages that cp.async fills ahead of the products (a step of few tokens is bound by the experts' matrices
// coming from memory, so several steps' loads are kept in flight); rows padded by 8 elements so that fragment loads do not collide;
// k_size is a multiple of 8, the rest of a step and the rows of empty slots are filled with zeros.
constexpr int MMA_TN = 64, MMA_TK = 64, MMA_PAD = 8;
__host__ __device__ constexpr int mma_stages(bool) { return 4; }   // (six stages for the plain product, whose stages are half as large, were faster at width 2,048 and slower at 4,096)
__host__ __device__ constexpr int mma_stage_elements(bool glu) { return (EXPERT_ROWS + (glu ? 2 : 1) * MMA_TN) * (MMA_TK + MMA_PAD); }
constexpr size_t mma_shared_bytes(bool glu) { return (size_t)mma_stages(glu) * mma_stage_elements(glu) * sizeof(__nv_bfloat16); }

__device__ __forceinline__ void copy_16_or_zeros(void* shared, const void* global, bool real) {
  const unsigned target = (unsigned)__cvta_generic_to_shared(shared);
  const int bytes = real ? 16 : 0;   // what is not copied is written as zeros
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(target), "l"(global), "r"(bytes) : "memory");
}

template <bool GLU>
__global__ void __launch_bounds__(128) experts_product_mma_kernel(const __nv_bfloat16* __restrict__ a, long long lda,
                                                                  const __nv_bfloat16* __restrict__ w, const int* __restrict__ source,
                                                                  const int* __restrict__ tile_expert, int gathered, int divide,
                                                                  void* __restrict__ out_v, int n_out, int k_size, int kind, int interleaved, int act_out,
                                                                  const float* __restrict__ slot_share, float limit, float alpha,
                                                                  int k_each, long long part_stride) {
  constexpr int TN = MMA_TN, TK = MMA_TK, LD = MMA_TK + MMA_PAD, G = GLU ? 2 : 1, MMA_STAGES = mma_stages(GLU);
  constexpr int A_ELEMENTS = EXPERT_ROWS * LD, STAGE_ELEMENTS = mma_stage_elements(GLU);
  extern __shared__ __align__(16) unsigned char mma_shared[];
  __nv_bfloat16* ring = reinterpret_cast<__nv_bfloat16*>(mma_shared);
  __shared__ int rows[EXPERT_ROWS];
  grid_dependency_wait();
  allow_dependents();
  const int tile = blockIdx.y;
  const int expert = tile_expert[tile];
  if (expert < 0) return;
  const int n0 = blockIdx.x * TN;
  if (threadIdx.x < EXPERT_ROWS) {
    const int pair = source[tile * EXPERT_ROWS + threadIdx.x];
    rows[threadIdx.x] = pair < 0 ? -1 : (gathered ? pair / divide : tile * EXPERT_ROWS + threadIdx.x);
  }
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int group = lane >> 2, quad = lane & 3;
  const long long w_rows = GLU ? 2LL * n_out : n_out;
  const __nv_bfloat16* w_mine = w + (long long)expert * w_rows * k_size;
  float acc[G][2][2][4];   // [gate | up][row half][column eighth][fragment]
#pragma unroll
  for (int g = 0; g < G; ++g)
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int f = 0; f < 4; ++f) acc[g][i][j][f] = 0.f;
  const int k_first = blockIdx.z * k_each;                                            // this block's share of k (all of it for a gated product)
  const int k_last = k_first + k_each < k_size ? k_first + k_each : k_size;
  const int steps = (k_last - k_first + TK - 1) / TK;
  auto fill = [&](int step) {   // every thread commits one group a call, also an empty one, so that the groups count the steps
    if (step < steps) {
      const int k0 = k_first + step * TK;
      __nv_bfloat16* a_stage = ring + (size_t)(step % MMA_STAGES) * STAGE_ELEMENTS;
      __nv_bfloat16* b_stage = a_stage + A_ELEMENTS;
      for (int x = threadIdx.x; x < EXPERT_ROWS * (TK / 8); x += 128) {
        const int r = x / (TK / 8), c = (x % (TK / 8)) * 8;
        const int row = rows[r];
        const bool real = row >= 0 && k0 + c < k_last;
        copy_16_or_zeros(a_stage + r * LD + c, real ? a + (long long)row * lda + k0 + c : a, real);
      }
      for (int x = threadIdx.x; x < G * TN * (TK / 8); x += 128) {
        const int g = x / (TN * (TK / 8)), y = x % (TN * (TK / 8));
        const int r = y / (TK / 8), c = (y % (TK / 8)) * 8;
        const bool real = n0 + r < n_out && k0 + c < k_last;
        copy_16_or_zeros(b_stage + (g * TN + r) * LD + c, real ? w_mine + glu_row(n0 + r, g, n_out, GLU && interleaved) * k_size + k0 + c : w_mine, real);
      }
    }
    asm volatile("cp.async.commit_group;\n" ::: "memory");
  };
#pragma unroll
  for (int step = 0; step < MMA_STAGES - 1; ++step) fill(step);
  for (int step = 0; step < steps; ++step) {
    asm volatile("cp.async.wait_group %0;\n" ::"n"(MMA_STAGES - 2) : "memory");   // this step's stage has arrived (for this thread's copies)
    __syncthreads();                                                               // ... for everyone's; and the stage of the step before is free
    fill(step + MMA_STAGES - 1);
    const __nv_bfloat16* a_stage = ring + (size_t)(step % MMA_STAGES) * STAGE_ELEMENTS;
    const __nv_bfloat16* b_stage = a_stage + A_ELEMENTS;
#pragma unroll
    for (int kk = 0; kk < TK; kk += 16) {
      unsigned af[2][4];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        af[i][0] = *reinterpret_cast<const unsigned*>(a_stage + (16 * i + group) * LD + kk + 2 * quad);
        af[i][1] = *reinterpret_cast<const unsigned*>(a_stage + (16 * i + group + 8) * LD + kk + 2 * quad);
        af[i][2] = *reinterpret_cast<const unsigned*>(a_stage + (16 * i + group) * LD + kk + 2 * quad + 8);
        af[i][3] = *reinterpret_cast<const unsigned*>(a_stage + (16 * i + group + 8) * LD + kk + 2 * quad + 8);
      }
#pragma unroll
      for (int g = 0; g < G; ++g)
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          const int n = 16 * warp + 8 * j + group;
          const unsigned b0 = *reinterpret_cast<const unsigned*>(b_stage + (g * TN + n) * LD + kk + 2 * quad);
          const unsigned b1 = *reinterpret_cast<const unsigned*>(b_stage + (g * TN + n) * LD + kk + 2 * quad + 8);
#pragma unroll
          for (int i = 0; i < 2; ++i)
            asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                         : "+f"(acc[g][i][j][0]), "+f"(acc[g][i][j][1]), "+f"(acc[g][i][j][2]), "+f"(acc[g][i][j][3])
                         : "r"(af[i][0]), "r"(af[i][1]), "r"(af[i][2]), "r"(af[i][3]), "r"(b0), "r"(b1));
        }
    }
  }
  asm volatile("cp.async.wait_group 0;\n" ::: "memory");
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int r = 16 * i + group + 8 * half;
      if (rows[r] < 0) continue;
      const long long slot = (long long)tile * EXPERT_ROWS + r;
      const float reads = GLU && slot_share ? slot_share[slot] : 1.f;
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int n = n0 + 16 * warp + 8 * j + 2 * quad + e;
          if (n >= n_out) continue;
          const float value = acc[0][i][j][2 * half + e];
          if (GLU) ((__nv_bfloat16*)out_v)[slot * n_out + n] = __float2bfloat16_rn(expert_unit(reads * value, reads * acc[G - 1][i][j][2 * half + e], kind, limit, alpha));
          else if (act_out) ((__nv_bfloat16*)out_v)[slot * n_out + n] = __float2bfloat16_rn(expert_activation(value, kind));
          else ((float*)out_v)[blockIdx.z * part_stride + slot * n_out + n] = value;
        }
    }
}

// ---------------------------------------------------------------------------------------------
// The products of a step of few tokens, the matrices by TMA.  A block takes 64 weight rows of one expert (with GLU: 32 gate rows and their up
// rows, alternating in groups of 8) and a row tile of 32 slots.  Warp 0 fills a ring: its first lane asks TMA for the 64 x 64 box of the
// matrix (128-byte swizzle), every lane copies its own slot's 128 bytes beside it (cp.async, in the same swizzle), and both complete on the
// stage's one mbarrier (33 arrivals).  Four consumer warps, 16 weight rows each, multiply with mma.sync, the weights as the 16-row A operand,
// the slots as 8-column B operands - as many of them as the tile holds.  Rows of empty slots are never filled: a column of the product depends
// on its own slot alone, and theirs are not written.  Every wait is bounded (error word 1: the producer, 2: a consumer gave up); a block that
// gives up waits for the copies it asked for before it leaves.  Bound by the matrices coming from memory: 64 KB in flight a block, three to
// an SM.  (The ring of cp.async stages reaches 3.3 TB/s.)
// ---------------------------------------------------------------------------------------------
constexpr int ES_SLAB = 64, ES_BK = 64, ES_CONSUMERS = 4, ES_THREADS = 32 * (1 + ES_CONSUMERS), ES_STAGES = 5;
constexpr int ES_W_BYTES = ES_SLAB * ES_BK * 2, ES_STAGE_BYTES = ES_W_BYTES + EXPERT_ROWS * ES_BK * 2;
constexpr size_t ES_SMEM = (size_t)ES_STAGES * ES_STAGE_BYTES + 1024 /* alignment slack */ + 128 /* barriers */;
constexpr unsigned ES_WAIT_LIMIT = 1u << 22;
enum ExpertStreamForm { ES_SUMS = 0, ES_GATED = 1, ES_ACTIVATED = 2 };

__device__ __forceinline__ unsigned es_smem(const void* p) { return (unsigned)__cvta_generic_to_shared(p); }
__device__ __forceinline__ bool es_wait(uint64_t* bar, unsigned parity) {
  for (unsigned tries = 0; tries < ES_WAIT_LIMIT; ++tries) {
    unsigned done;
    asm volatile("{\n.reg .pred p;\nmbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\nselp.u32 %0, 1, 0, p;\n}\n"
                 : "=r"(done) : "r"(es_smem(bar)), "r"(parity) : "memory");
    if (done) return true;
  }
  return false;
}
__device__ __forceinline__ void es_ldmatrix(unsigned (&r)[4], unsigned address) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(address));
}
__device__ __forceinline__ void es_mma(float (&c)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// Grid (slabs of 64 weight rows, row tiles, parts of k).  map_w: the stacked matrices [experts * w_rows, k_size] in boxes of 64 x 64.
template <int FORM>
__global__ void __launch_bounds__(ES_THREADS, 3) experts_stream_kernel(const __grid_constant__ CUtensorMap map_w, const __nv_bfloat16* __restrict__ a, long long lda,
                                                                        const int* __restrict__ source, const int* __restrict__ tile_expert, int gathered, int divide,
                                                                        void* __restrict__ out_v, int n_out, int k_size, int w_rows, int kind,
                                                                        const float* __restrict__ slot_share, float limit, float alpha, int k_each, long long part_stride,
                                                                        int* __restrict__ error) {
  constexpr int TILES = EXPERT_ROWS / 8;
  extern __shared__ unsigned char es_shared[];
  unsigned char* stages = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(es_shared) + 1023) & ~(uintptr_t)1023);
  uint64_t* full = reinterpret_cast<uint64_t*>(stages + (size_t)ES_STAGES * ES_STAGE_BYTES);
  uint64_t* empty = full + ES_STAGES;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int tile = blockIdx.y, n0 = blockIdx.x * ES_SLAB;
  if (threadIdx.x == 0) {
#pragma unroll
    for (int s = 0; s < ES_STAGES; ++s) {
      asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;\n" ::"r"(es_smem(&full[s])), "r"(33));
      asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;\n" ::"r"(es_smem(&empty[s])), "r"(ES_CONSUMERS));
    }
    asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
  }
  __syncthreads();
  grid_dependency_wait();
  allow_dependents();
  const int expert = tile_expert[tile];
  if (expert < 0) return;
  const int pair = source[tile * EXPERT_ROWS + lane];   // every warp knows the tile's slots, one a lane; the filled ones come first
  const int filled = __popc(__ballot_sync(0xffffffffu, pair >= 0));
  const int k_first = blockIdx.z * k_each;
  const int k_last = k_first + k_each < k_size ? k_first + k_each : k_size;
  const int boxes = (k_last - k_first + ES_BK - 1) / ES_BK;

  if (warp == 0) {
    const __nv_bfloat16* row = pair < 0 ? nullptr : a + (long long)(gathered ? pair / divide : tile * EXPERT_ROWS + lane) * lda + k_first;
    unsigned stage = 0, phase = 0;
    for (int box = 0; box < boxes; ++box) {
      if (box >= ES_STAGES && !es_wait(&empty[stage], phase ^ 1)) {
        if (lane == 0) atomicExch(error, 1);
        break;
      }
      unsigned char* to = stages + (size_t)stage * ES_STAGE_BYTES;
      if (lane == 0) {
        asm volatile("fence.proxy.async.shared::cta;\n" ::: "memory");   // the consumers read the stage with ordinary loads: TMA is another proxy
        asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;\n" ::"r"(es_smem(&full[stage])), "r"(ES_W_BYTES) : "memory");
        asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4}], [%2];\n"
                     ::"r"(es_smem(to)), "l"((unsigned long long)&map_w), "r"(es_smem(&full[stage])), "r"(k_first + box * ES_BK), "r"(expert * w_rows + n0) : "memory");
      }
      if (row) {
        unsigned char* mine = to + ES_W_BYTES + lane * 128;
#pragma unroll
        for (int unit = 0; unit < 8; ++unit) {
          const int k = box * ES_BK + unit * 8;
          const bool real = k_first + k < k_last;
          copy_16_or_zeros(mine + ((unit ^ (lane & 7)) << 4), real ? row + k : row, real);
        }
      }
      asm volatile("cp.async.mbarrier.arrive.noinc.shared::cta.b64 [%0];\n" ::"r"(es_smem(&full[stage])) : "memory");
      if (++stage == ES_STAGES) { stage = 0; phase ^= 1; }
    }
    asm volatile("cp.async.wait_all;\n" ::: "memory");
    return;
  }

  // In the 128-byte swizzle the 16-byte unit u of row r sits at unit u ^ (r % 8).
  const int slab_row = (warp - 1) * 16 + (lane & 7) + 8 * ((lane >> 3) & 1);
  const unsigned w_row_offset = (unsigned)slab_row * 128, w_xor = (unsigned)(slab_row & 7);
  const unsigned x_row_offset = (unsigned)ES_W_BYTES + (unsigned)(lane & 7) * 128, x_xor = (unsigned)(lane & 7);
  float acc[TILES][2][4];   // per 8 slots: even and odd k-steps, two MMA chains
#pragma unroll
  for (int j = 0; j < TILES; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) acc[j][0][i] = acc[j][1][i] = 0.f;
  unsigned stage = 0, phase = 0;
  for (int box = 0; box < boxes; ++box) {
    if (!es_wait(&full[stage], phase)) {
      if (lane == 0) atomicExch(error, 2);
      return;
    }
    const unsigned here = es_smem(stages + (size_t)stage * ES_STAGE_BYTES);
#pragma unroll
    for (int half = 0; half < 2; ++half) {   // 32 k each
      unsigned w[2][4];
#pragma unroll
      for (int step = 0; step < 2; ++step)    // 16 k each
        es_ldmatrix(w[step], here + w_row_offset + ((((unsigned)(4 * half + 2 * step) + (lane >> 4)) ^ w_xor) << 4));
#pragma unroll
      for (int j = 0; j < TILES; ++j) {
        if (8 * j >= filled) break;            // the same for every lane
        unsigned x[4];                         // units 4 * half .. + 3 of slots 8j .. 8j + 7
        es_ldmatrix(x, here + (unsigned)(j * 8 * 128) + x_row_offset + ((((unsigned)(4 * half) + (lane >> 3)) ^ x_xor) << 4));
        es_mma(acc[j][0], w[0], x[0], x[1]);
        es_mma(acc[j][1], w[1], x[2], x[3]);
      }
    }
    __syncwarp();
    if (lane == 0) asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];\n" ::"r"(es_smem(&empty[stage])) : "memory");
    if (++stage == ES_STAGES) { stage = 0; phase ^= 1; }
  }

  // Accumulator element i of lane (group, quad): weight row group + 8 * (i / 2), slot 2 * quad + (i % 2) of its eight.
  const int group = lane >> 2, quad = lane & 3;
  const int row0 = n0 + (warp - 1) * 16 + group;
#pragma unroll
  for (int j = 0; j < TILES; ++j) {
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int m = j * 8 + 2 * quad + e;
      if (m >= filled) continue;
      const long long slot = (long long)tile * EXPERT_ROWS + m;
      const float low = acc[j][0][e] + acc[j][1][e], high = acc[j][0][2 + e] + acc[j][1][2 + e];
      if (FORM == ES_GATED) {   // rows row0 (gate) and row0 + 8 (its up row)
        const int n = (n0 + (warp - 1) * 16) / 2 + group;
        const float reads = slot_share ? slot_share[slot] : 1.f;
        if (n < n_out) ((__nv_bfloat16*)out_v)[slot * n_out + n] = __float2bfloat16_rn(expert_unit(reads * low, reads * high, kind, limit, alpha));
      } else if (FORM == ES_ACTIVATED) {
        if (row0 < n_out) ((__nv_bfloat16*)out_v)[slot * n_out + row0] = __float2bfloat16_rn(expert_activation(low, kind));
        if (row0 + 8 < n_out) ((__nv_bfloat16*)out_v)[slot * n_out + row0 + 8] = __float2bfloat16_rn(expert_activation(high, kind));
      } else {
        float* out = (float*)out_v + blockIdx.z * part_stride + slot * n_out;
        if (row0 < n_out) out[row0] = low;
        if (row0 + 8 < n_out) out[row0 + 8] = high;
      }
    }
  }
}

// share null: the rows are added up as they are.
// out[t, c] = sum_k share[t, k] * y[slot_of[t * top + k], c], the choices in their order; y in float32 or in the compute dtype.
// With `same` (rows in C, same_ld apart) and same_share (float32 [T]): + same_share[t] * same[t, c].  A slot of -1 is none.
// With `common` ([T, width] in C, an expert that every token goes through) and `gate` (float32 [T]): + gate[t] * common[t, c].
template <typename Y, typename C>
__global__ void experts_gather_kernel(const Y* __restrict__ y, const int* __restrict__ slot_of, const float* __restrict__ share,
                                      float* __restrict__ out, int width, int top, long long total, const C* __restrict__ common,
                                      const float* __restrict__ gate, int parts, long long part_stride, const C* __restrict__ same, long long same_ld,
                                      const float* __restrict__ same_share) {
  grid_dependency_wait();
  allow_dependents();
  const long long item = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (item >= total) return;
  const long long t = item / width;
  const int c = (int)(item % width);
  float acc = 0.f;
  for (int k = 0; k < top; ++k) {
    const int slot = slot_of[t * top + k];
    if (slot < 0) continue;
    const Y* row = y + (long long)slot * width + c;
    float value = to_float<Y>(row[0]);
    for (int part = 1; part < parts; ++part) value += to_float<Y>(row[part * part_stride]);
    acc = fmaf(share ? share[t * top + k] : 1.f, value, acc);
  }
  if (common != nullptr) acc = fmaf(gate[t], to_float<C>(common[item]), acc);
  if (same != nullptr) acc = fmaf(same_share[t], to_float<C>(same[t * same_ld + c]), acc);
  out[item] = acc;
}

// sorted[slot, :] = h[source[slot] / top, :], zeros in an empty slot: the tokens' rows in the order of their experts, for a product
// that takes whole row tiles from memory.  A thread moves 16 bytes; chunks = 16-byte pieces of a row.
__global__ void experts_sort_rows_kernel(const uint4* __restrict__ h, long long ld_chunks, const int* __restrict__ source, uint4* __restrict__ sorted,
                                         int chunks, int top, long long total) {
  grid_dependency_wait();
  allow_dependents();
  const long long item = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (item >= total) return;
  const long long slot = item / chunks;
  const int c = (int)(item % chunks);
  const int pair = source[slot];
  sorted[item] = pair < 0 ? make_uint4(0, 0, 0, 0) : h[(long long)(pair / top) * ld_chunks + c];
}

}  // namespace pylon

using namespace pylon;

extern "C" int pylon_experts_row_tile() { return EXPERT_ROWS; }

// scored 1: the sigmoid form, 2: the softmax over all (see RouteScored); router is then float32 [experts + extra, width].  `experts` counts the last
// `identity` outputs, experts that hand their input back; chosen and share are [T, top + always].
extern "C" int pylon_experts_route(const void* h, long long ld, const float* router, const float* bias, int* chosen, float* share, int width,
                                   int experts, int top, int num_tokens, int dtype, int scored, const float* correction, int groups, int keep,
                                   float share_eps, int normalize, int extra, float* extra_out, int group_best, float share_scale, int identity,
                                   float* same_share, int always, cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  if (experts < 1 || top < 1 || top > experts || experts > 2048) PYLON_REFUSE("experts_route: %d of %d experts (at most 2048)", top, experts);
  if (scored < 0 || scored > 2 || identity < 0 || identity >= experts || (identity > 0 && (!scored || !same_share)) || always < 0)
    PYLON_REFUSE("experts_route: form %d, %d experts that hand their input back of %d, %d pieces for every token", scored, identity, experts, always);
  if (!scored && (correction || groups || extra)) PYLON_REFUSE("experts_route: a correction, groups and extra rows go with the sigmoid form");
  if (scored && (groups < 0 || (groups > 0 && (experts % groups || keep < 1 || keep > groups || top > keep * (experts / groups))) || extra < 0 || extra > 64 ||
                 (extra > 0 && !extra_out)))
    PYLON_REFUSE("experts_route: %d groups of which %d are kept for %d of %d experts, %d extra rows", groups, keep, top, experts, extra);
  const RouteScored mode{scored, correction, groups, keep, share_eps, normalize, extra, extra_out, group_best, share_scale, experts - identity, same_share};
  const int per_token = experts + extra + (scored ? experts + groups : 0);
  const bool few = num_tokens < 512;   // a step of few tokens: a block each
  const size_t element = dtype == PYLON_DTYPE_F32 ? 4 : 2;
  const bool pieces = width % 4 == 0 && ld % 4 == 0 && (uintptr_t)h % (4 * element) == 0 && (uintptr_t)router % 16 == 0;
#define PYLON_ROUTE(T, TOKENS, V)                                                                                                            \
  launch_dependent(experts_route_kernel<T, TOKENS, V>, dim3((unsigned)((num_tokens + TOKENS - 1) / TOKENS)), dim3(128),                      \
                   (size_t)TOKENS * (4 * ROUTE_SIDE + per_token) * sizeof(float), stream, (const T*)h, ld, router, bias, chosen, share, width, experts, top, num_tokens, always, mode)
#define PYLON_ROUTE_SIZES(T)                                                                                                                 \
  if (few) { if (pieces) PYLON_ROUTE(T, 1, 4); else PYLON_ROUTE(T, 1, 1); }                                                                  \
  else { if (pieces) PYLON_ROUTE(T, 4, 4); else PYLON_ROUTE(T, 4, 1); }
  if (dtype == PYLON_DTYPE_F32) { PYLON_ROUTE_SIZES(float) }
  else if (dtype == PYLON_DTYPE_BF16) { PYLON_ROUTE_SIZES(__nv_bfloat16) }
  else PYLON_REFUSE("experts_route: unknown dtype %d", dtype);
#undef PYLON_ROUTE_SIZES
#undef PYLON_ROUTE
  PYLON_CHECK_LAUNCH("experts_route");
}

// tile_rows: the slots of a row tile (pylon_experts_row_tile() for the products of this file, 128 for the grouped tcgen05 product).
extern "C" int pylon_experts_plan(const int* chosen, int* slot_of, int* source, int* tile_expert, int pairs, int experts, int max_slots,
                                  int max_tiles, int tile_rows, const float* share, float* slot_share, int per, int always, cudaStream_t stream) {
  if (pairs <= 0) return 0;
  if (per < 1 || pairs % per || always < 0 || always >= experts || always >= per) PYLON_REFUSE("experts_plan: %d pairs, %d to a token, %d of %d experts every token's", pairs, per, always, experts);
  if (slot_share && !share) PYLON_REFUSE("experts_plan: shares per slot need the shares per choice");
  if (tile_rows < 1 || max_slots < pairs || (long long)max_tiles * tile_rows < max_slots)
    PYLON_REFUSE("experts_plan: %d slots in %d tiles of %d for %d pairs", max_slots, max_tiles, tile_rows, pairs);
  launch_dependent(experts_plan_kernel, dim3(1), dim3(1024), (size_t)(2 * experts + 1) * sizeof(int), stream, chosen, slot_of, source, tile_expert,
                   pairs, experts, max_slots, max_tiles, tile_rows, share, slot_share, per, always);
  PYLON_CHECK_LAUNCH("experts_plan");
}

typedef CUresult (*EncodeTiled)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

// The stacked matrices [rows, cols], contiguous, in boxes of 64 x 64 in the 128-byte swizzle.  Maps are kept by their arguments: a model
// multiplies by the same matrices at every step.
static bool stacked_map(CUtensorMap* map, const void* base, long long rows, long long cols) {
  struct Key {
    const void* base; long long rows, cols;
    bool operator==(const Key& o) const { return base == o.base && rows == o.rows && cols == o.cols; }
  };
  struct Hash {
    size_t operator()(const Key& k) const { return std::hash<const void*>()(k.base) ^ (size_t)(k.rows * 1315423911LL) ^ (size_t)(k.cols * 2654435761LL); }
  };
  static std::unordered_map<Key, CUtensorMap, Hash> known;
  static std::mutex mutex;
  std::lock_guard<std::mutex> guard(mutex);
  const Key key{base, rows, cols};
  auto found = known.find(key);
  if (found != known.end()) { *map = found->second; return true; }
  static EncodeTiled encode = [] {
    void* symbol = nullptr;
    cudaDriverEntryPointQueryResult result;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &symbol, cudaEnableDefault, &result) != cudaSuccess || result != cudaDriverEntryPointSuccess) symbol = nullptr;
    return (EncodeTiled)symbol;
  }();
  if (!encode) return false;
  cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows};
  cuuint64_t strides[1] = {(cuuint64_t)cols * 2};
  cuuint32_t box[2] = {(cuuint32_t)ES_BK, (cuuint32_t)ES_SLAB};
  cuuint32_t element_strides[2] = {1, 1};
  if (encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, element_strides, CU_TENSOR_MAP_INTERLEAVE_NONE,
             CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
    return false;
  if (known.size() >= 4096) known.clear();
  known.emplace(key, *map);
  return true;
}

template <int FORM>
static int launch_experts_stream(const CUtensorMap& map_w, const __nv_bfloat16* a, long long lda, const int* source, const int* tile_expert, int gathered, int divide,
                                 void* out, int n_out, int k_size, int w_rows, int max_tiles, int kind, const float* slot_share, float limit, float alpha, int k_parts,
                                 int* error, cudaStream_t stream) {
  static bool configured_on[pylon::MAX_DEVICES] = {};   // function attributes belong to a device
  bool& configured = configured_on[pylon::current_device_slot()];
  if (!configured) {
    cudaError_t err = cudaFuncSetAttribute(experts_stream_kernel<FORM>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)ES_SMEM);
    if (err != cudaSuccess) PYLON_REFUSE("experts_stream: %s", cudaGetErrorString(err));
    configured = true;
  }
  launch_dependent(experts_stream_kernel<FORM>, dim3((unsigned)((w_rows + ES_SLAB - 1) / ES_SLAB), (unsigned)max_tiles, (unsigned)k_parts), dim3(ES_THREADS), ES_SMEM, stream,
                   map_w, a, lda, source, tile_expert, gathered, divide, out, n_out, k_size, w_rows, kind, slot_share, limit, alpha, k_size / k_parts,
                   (long long)max_tiles * EXPERT_ROWS * n_out, error);
  PYLON_CHECK_LAUNCH("experts_stream");
}

template <bool GLU>
static void allow_mma_shared_memory() {
  static bool configured_on[pylon::MAX_DEVICES] = {};   // function attributes belong to a device
  bool& configured = configured_on[pylon::current_device_slot()];
  if (configured) return;
  cudaFuncSetAttribute(experts_product_mma_kernel<GLU>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)mma_shared_bytes(GLU));
  configured = true;
}

// a: [rows, lda] in dtype; w: [experts, (glu ? 2 : 1) * n_out, k] in dtype, contiguous (with glu an expert's gate rows, then its up rows;
// or, interleaved != 0, alternating in groups of 8); out: [max_tiles * EXPERT_ROWS, n_out], in dtype with glu, else float32.
// k_parts > 1 (a plain bfloat16 product): k in so many equal parts, out float32 [k_parts, max_tiles * EXPERT_ROWS, n_out] whose sum the product is.
// glu == 2: no gate, but the activation on the product itself, out in dtype (the first product of an ungated expert).
// experts: how many matrices w holds; error: one int that a kernel sets when a bounded wait of it ran out (the output is then void), or null: the
// form whose matrices come by TMA is then not taken.
extern "C" int pylon_experts_product(const void* a, long long lda, const void* w, const int* source, const int* tile_expert, int gathered,
                                     int divide, void* out, int n_out, int k_size, int max_tiles, int glu, int kind, int interleaved, int dtype,
                                     const float* slot_share, float limit, float alpha, int k_parts, int experts, int* error, cudaStream_t stream) {
  if (max_tiles <= 0) return 0;
  const int act_out = glu == 2 ? 1 : 0;
  if (act_out) glu = 0;
  if (n_out <= 0 || k_size <= 0 || divide < 1 || kind < 0 || kind > 4 || (kind == 4 && glu && !(limit > 0.f)) || (kind == 4 && act_out)) PYLON_REFUSE("experts_product: n %d, k %d, divide %d, activation %d", n_out, k_size, divide, kind);
  if (max_tiles > 65535) PYLON_REFUSE("experts_product: %d row tiles", max_tiles);
  if (interleaved && (!glu || n_out % 8)) PYLON_REFUSE("experts_product: interleaved rows need a gated product of a multiple of 8 columns, got %d", n_out);
  if (k_parts < 1 || k_parts > 16 || (k_parts > 1 && (glu || act_out || dtype != PYLON_DTYPE_BF16 || k_size % (64 * k_parts) || lda % 8 || (uintptr_t)a % 16 || (uintptr_t)w % 16)))
    PYLON_REFUSE("experts_product: k of %d in %d parts (a plain bfloat16 product over whole steps of 64 only)", k_size, k_parts);
  const dim3 grid((unsigned)((n_out + 63) / 64), (unsigned)max_tiles, (unsigned)k_parts);
  const int k_each = k_size / k_parts;
  const long long part_stride = (long long)max_tiles * EXPERT_ROWS * n_out;
  if (dtype == PYLON_DTYPE_F32) {
    if (glu) launch_dependent(experts_product_kernel<float, true>, grid, dim3(256), 0, stream, (const float*)a, lda, (const float*)w, source, tile_expert, gathered, divide, out, n_out, k_size, kind, interleaved, act_out, slot_share, limit, alpha);
    else launch_dependent(experts_product_kernel<float, false>, grid, dim3(256), 0, stream, (const float*)a, lda, (const float*)w, source, tile_expert, gathered, divide, out, n_out, k_size, kind, interleaved, act_out, slot_share, limit, alpha);
  } else if (dtype == PYLON_DTYPE_BF16) {
    const __nv_bfloat16* ab = (const __nv_bfloat16*)a;
    const __nv_bfloat16* wb = (const __nv_bfloat16*)w;
    const bool vectors = k_size % 8 == 0 && lda % 8 == 0 && (uintptr_t)a % 16 == 0 && (uintptr_t)w % 16 == 0;
    const int w_rows = glu ? 2 * n_out : n_out;
    if (vectors && error && experts > 0 && (!glu || interleaved) && (long long)experts * w_rows < 2147483647LL - ES_SLAB) {
      CUtensorMap map_w;
      if (!stacked_map(&map_w, w, (long long)experts * w_rows, k_size)) PYLON_REFUSE("experts_product: the tensor map of the matrices could not be made");
#define PYLON_STREAM(FORM) return launch_experts_stream<FORM>(map_w, ab, lda, source, tile_expert, gathered, divide, out, n_out, k_size, w_rows, max_tiles, kind, slot_share, limit, alpha, k_parts, error, stream)
      if (glu) PYLON_STREAM(ES_GATED);
      if (act_out) PYLON_STREAM(ES_ACTIVATED);
      PYLON_STREAM(ES_SUMS);
#undef PYLON_STREAM
    }
    if (vectors) {
      if (glu) {
        allow_mma_shared_memory<true>();
        launch_dependent(experts_product_mma_kernel<true>, grid, dim3(128), mma_shared_bytes(true), stream, ab, lda, wb, source, tile_expert, gathered, divide, out, n_out, k_size, kind, interleaved, act_out, slot_share, limit, alpha, k_each, part_stride);
      } else {
        allow_mma_shared_memory<false>();
        launch_dependent(experts_product_mma_kernel<false>, grid, dim3(128), mma_shared_bytes(false), stream, ab, lda, wb, source, tile_expert, gathered, divide, out, n_out, k_size, kind, interleaved, act_out, slot_share, limit, alpha, k_each, part_stride);
      }
    } else {
      if (glu) launch_dependent(experts_product_kernel<__nv_bfloat16, true>, grid, dim3(256), 0, stream, ab, lda, wb, source, tile_expert, gathered, divide, out, n_out, k_size, kind, interleaved, act_out, slot_share, limit, alpha);
      else launch_dependent(experts_product_kernel<__nv_bfloat16, false>, grid, dim3(256), 0, stream, ab, lda, wb, source, tile_expert, gathered, divide, out, n_out, k_size, kind, interleaved, act_out, slot_share, limit, alpha);
    }
  } else PYLON_REFUSE("experts_product: unknown dtype %d", dtype);
  PYLON_CHECK_LAUNCH("experts_product");
}

// h [T, ld] and sorted [max_slots, width] in a 16-bit or 32-bit dtype; rows of whole 16-byte pieces at 16-byte addresses.
extern "C" int pylon_experts_sort_rows(const void* h, long long ld, const int* source, void* sorted, int width, int top, int max_slots, int dtype,
                                       cudaStream_t stream) {
  if (max_slots <= 0) return 0;
  const int per_chunk = dtype == PYLON_DTYPE_F32 ? 4 : 8;
  if (top < 1 || width % per_chunk || ld % per_chunk || (uintptr_t)h % 16 || (uintptr_t)sorted % 16)
    PYLON_REFUSE("experts_sort_rows: rows of %d (stride %lld) are not whole 16-byte pieces at 16-byte addresses", width, ld);
  const int chunks = width / per_chunk;
  const long long total = (long long)max_slots * chunks;
  launch_dependent(experts_sort_rows_kernel, dim3((unsigned)((total + 255) / 256)), dim3(256), 0, stream, (const uint4*)h, ld / per_chunk, source, (uint4*)sorted,
                   chunks, top, total);
  PYLON_CHECK_LAUNCH("experts_sort_rows");
}

// parts > 1: y is float32 [parts, slots, width], the rows' partial sums.
// y: [slots, width] in float32 (y_dtype PYLON_DTYPE_F32) or bfloat16; out float32 [num_tokens, width].
// same (rows same_ld apart, in common_dtype) and same_share (float32 [num_tokens]): out += same_share[t] * same[t].
// common ([num_tokens, width] in common_dtype) and gate (float32 [num_tokens]), both or neither: out += gate[t] * common[t].
extern "C" int pylon_experts_gather(const void* y, const int* slot_of, const float* share, float* out, int num_tokens, int width, int top, int y_dtype,
                                    const void* common, const float* gate, int common_dtype, int parts, long long slots, const void* same, long long same_ld,
                                    const float* same_share, cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  if (parts < 1 || (parts > 1 && (y_dtype != PYLON_DTYPE_F32 || slots < 1))) PYLON_REFUSE("experts_gather: %d parts", parts);
  if ((common == nullptr) != (gate == nullptr)) PYLON_REFUSE("experts_gather: a common expert's output and its gate go together");
  const long long total = (long long)num_tokens * width;
  const dim3 grid((unsigned)((total + 255) / 256));
  if (common && same) PYLON_REFUSE("experts_gather: a common expert or experts that hand their input back, not both");
  const bool common_f32 = (common == nullptr && same == nullptr) || common_dtype == PYLON_DTYPE_F32;
#define PYLON_GATHER(Y, C) launch_dependent(experts_gather_kernel<Y, C>, grid, dim3(256), 0, stream, (const Y*)y, slot_of, share, out, width, top, total, (const C*)common, gate, parts, slots * width, (const C*)same, same_ld, same_share)
  if (y_dtype == PYLON_DTYPE_F32) { if (common_f32) PYLON_GATHER(float, float); else PYLON_GATHER(float, __nv_bfloat16); }
  else if (y_dtype == PYLON_DTYPE_BF16) { if (common_f32) PYLON_GATHER(__nv_bfloat16, float); else PYLON_GATHER(__nv_bfloat16, __nv_bfloat16); }
  else PYLON_REFUSE("experts_gather: unknown dtype %d", y_dtype);
#undef PYLON_GATHER
  PYLON_CHECK_LAUNCH("experts_gather");
}
