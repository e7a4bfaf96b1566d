// Paged causal attention, the plain form: one block per (token, query head), any key size
// up to 2,048 and value size up to 512, any page size, any group size, optional window or chunks of positions, optional soft
// cap on the scores, values of another width than the keys.  It is the attention of the
// true 32-bit path and the fall-back of the bfloat16 path for head sizes the tensor-core
// kernel is not built for.  Scores, softmax and the weighted sum are float32.
//
// Semantics (raun6k/Pylon: src/pylon/kv/cache.py:462-476 on the GPU, its exact restatement
// 483-491): a token at position p of its request attends the keys at positions j <= p of
// the same request (and j > p - window when a window is given); scale 1/sqrt(head size)
// unless another is passed; query head h reads KV head h / (nq / nkv).  With `chunk` > 0 a token sees
// only the keys of its own chunk of positions, j / chunk == p / chunk (chunks count from position 0 of
// the request); with `softcap` c > 0 a score s becomes c * tanh(s / c) before the softmax.  With `sinks`
// (one float32 per query head) the softmax's denominator also holds exp(sink): a key without a value
// whose score is the sink as it stands, neither scaled nor capped.  Key and value rows may lie
// `k_row_stride` / `v_row_stride` elements apart (0: their own widths), so that the values can be the first
// `dv` columns of the key rows themselves (one latent row per token, read by every head: nkv = 1).
// With `keep_first` n > 0 a window never hides the keys at positions j < n: a token sees j <= p with p - j < window or j < n.
// With `bias` (float32 [bias_rows, nq]) the scaled (and capped) score of the key d = p - j positions back gets
// bias[min(d, bias_rows - 1), h] added: a learnt function of the distance that is constant from bias_rows - 1 on.
//
// With `slopes` (float32 [nq]) that score loses slopes[h] for every position of distance.
//
// With `sigmoid` weights nothing is normalised: a visible key's weight is sigmoid(score + score_bias[h]) (score_bias float32 [nq] or
// null).  `gate` ([tokens, >= nq] in the compute dtype, or null): head h's output is multiplied by sigmoid(gate[t, h]), or with gate_elements
// ([tokens, >= nq * dv]) element e of it by sigmoid(gate[t, h * dv + e]); `factor` multiplies every output; the output's rows may lie
// out_stride elements apart.
//
// The keys of a token are walked in chunks of 128 positions aligned at position 0, so a
// token's result depends on its position only, not on how the step was cut or batched.
#include "common.cuh"

namespace pylon {

constexpr int SIMPLE_THREADS = 128;
constexpr int SIMPLE_MAX_DIMS_PER_THREAD = 4;  // head size <= 512

template <typename T>
__global__ void __launch_bounds__(SIMPLE_THREADS) paged_attention_simple_kernel(
    const T* __restrict__ q, long long q_token_stride, const T* __restrict__ k_pages,
    const T* __restrict__ v_pages, T* __restrict__ out, const int* __restrict__ positions,
    const int* __restrict__ token_row, const int* __restrict__ block_table, int table_width, int page_size,
    int num_pages, int nq, int nkv, int d, int dv, int window, int chunk, float softcap, float scale,
    const float* __restrict__ sinks, long long k_row_stride, long long v_row_stride, int keep_first, const float* __restrict__ bias,
    int bias_rows, int sigmoid, const float* __restrict__ score_bias, const T* __restrict__ gate, long long gate_stride, float factor,
    long long out_stride, const float* __restrict__ slopes, int gate_elements) {
  extern __shared__ long long shared[];
  long long* offsets = shared;                                      // [128] cache rows of the keys (page, head, slot), -1: none
  float* probs = reinterpret_cast<float*>(offsets + SIMPLE_THREADS);  // [128]
  float* scratch = probs + SIMPLE_THREADS;                          // [33]
  float* qs = scratch + 34;                                         // [d]

  const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  const int kv_head = h / (nq / nkv);
  const int pos = positions[t];
  const int row = token_row[t];
  if (row < 0) return;   // a padding token of a step padded to a captured size: it belongs to no request, its output is never read
  const int* table = block_table + (size_t)row * table_width;
  const T* qrow = q + (size_t)t * q_token_stride + (size_t)h * d;
  for (int e = tid; e < d; e += SIMPLE_THREADS) qs[e] = to_float<T>(qrow[e]) * scale;

  int lo = window > 0 ? (pos - window + 1 > 0 ? pos - window + 1 : 0) : 0;
  if (chunk > 0 && (pos / chunk) * chunk > lo) lo = (pos / chunk) * chunk;
  float acc[SIMPLE_MAX_DIMS_PER_THREAD];
#pragma unroll
  for (int k = 0; k < SIMPLE_MAX_DIMS_PER_THREAD; ++k) acc[k] = 0.f;
  // a sink is a key of score sinks[h] and value zero, met before all others
  float running_max = sinks ? sinks[h] : -INFINITY, running_sum = sinks ? 1.f : 0.f;
  __syncthreads();

  const int kept = keep_first < lo ? keep_first : lo;   // the keys before the window that stay visible: [0, kept)
  for (int c0 = kept > 0 ? 0 : (lo / SIMPLE_THREADS) * SIMPLE_THREADS; c0 <= pos; c0 += SIMPLE_THREADS) {
    if (c0 >= kept && c0 + SIMPLE_THREADS <= lo) continue;   // a chunk between the kept keys and the window (the same for all threads)
    const int j = c0 + tid;
    float score = -INFINITY;
    long long offset = -1;
    if ((j >= lo || j < kept) && j <= pos) {
      const int page = table[j / page_size];
      if (page >= 0 && page < num_pages) {
        offset = ((long long)page * nkv + kv_head) * page_size + j % page_size;
        const T* krow = k_pages + offset * k_row_stride;
        float dot = 0.f;
        for (int e = 0; e < d; ++e) dot = fmaf(qs[e], to_float<T>(krow[e]), dot);
        score = softcap > 0.f ? softcap * tanhf(dot / softcap) : dot;
        if (bias) score += bias[(size_t)(pos - j < bias_rows ? pos - j : bias_rows - 1) * nq + h];
        if (slopes) score -= slopes[h] * (float)(pos - j);
      }
    }
    offsets[tid] = offset;
    float rescale = 1.f;
    if (sigmoid) {
      probs[tid] = offset >= 0 ? 1.f / (1.f + expf(-(score + (score_bias ? score_bias[h] : 0.f)))) : 0.f;
      __syncthreads();
    } else {
      const float chunk_max = block_max(score, scratch);
      const float new_max = fmaxf(running_max, chunk_max);
      // new_max is finite: the chunk holds at least key `pos` (or an earlier chunk did).
      const float p = offset >= 0 ? expf(score - new_max) : 0.f;
      probs[tid] = p;
      const float chunk_sum = block_sum(p, scratch);  // also orders probs/offsets writes
      rescale = running_max == -INFINITY ? 0.f : expf(running_max - new_max);
      running_sum = running_sum * rescale + chunk_sum;
      running_max = new_max;
    }
    const int valid = pos - c0 + 1 < SIMPLE_THREADS ? pos - c0 + 1 : SIMPLE_THREADS;
#pragma unroll
    for (int k = 0; k < SIMPLE_MAX_DIMS_PER_THREAD; ++k) {
      const int e = tid + k * SIMPLE_THREADS;
      if (e < dv) {
        float a = acc[k] * rescale;
        for (int i = 0; i < valid; ++i) {
          const long long off = offsets[i];
          if (off >= 0) a = fmaf(probs[i], to_float<T>(v_pages[off * v_row_stride + e]), a);
        }
        acc[k] = a;
      }
    }
    __syncthreads();
  }
  T* orow = out + (size_t)t * out_stride + (size_t)h * dv;
  float inv = sigmoid ? 1.f : (running_sum > 0.f ? 1.f / running_sum : 0.f);
  inv *= factor;
  if (gate && !gate_elements) inv *= 1.f / (1.f + expf(-to_float<T>(gate[(size_t)t * gate_stride + h])));
#pragma unroll
  for (int k = 0; k < SIMPLE_MAX_DIMS_PER_THREAD; ++k) {
    const int e = tid + k * SIMPLE_THREADS;
    if (e >= dv) continue;
    const float open = gate && gate_elements ? 1.f / (1.f + expf(-to_float<T>(gate[(size_t)t * gate_stride + (size_t)h * dv + e]))) : 1.f;
    orow[e] = from_float<T>(acc[k] * inv * open);
  }
}

}  // namespace pylon

using namespace pylon;

extern "C" int pylon_paged_attention_simple(const void* q, long long q_token_stride, const void* k_pages,
                                            const void* v_pages, void* out, const int* positions,
                                            const int* token_row, const int* block_table, int table_width,
                                            int page_size, int num_pages, int nq, int nkv, int d, int dv, int window,
                                            int chunk, float softcap, float scale, const float* sinks,
                                            long long k_row_stride, long long v_row_stride, int num_tokens, int dtype,
                                            int keep_first, const float* bias, int bias_rows, int sigmoid, const float* score_bias,
                                            const void* gate, long long gate_stride, float factor, long long out_stride, const float* slopes, int gate_elements,
                                            cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  if (d < 1 || d > 2048) PYLON_REFUSE("paged_attention_simple: head size %d is outside 1..2048", d);
  if (k_row_stride == 0) k_row_stride = d;
  if (v_row_stride == 0) v_row_stride = dv;
  if (k_row_stride < d || v_row_stride < dv) PYLON_REFUSE("paged_attention_simple: rows of %d / %d elements cannot lie %lld / %lld apart", d, dv, k_row_stride, v_row_stride);
  if (dv < 1 || dv > SIMPLE_THREADS * SIMPLE_MAX_DIMS_PER_THREAD)
    PYLON_REFUSE("paged_attention_simple: value size %d is outside 1..%d", dv, SIMPLE_THREADS * SIMPLE_MAX_DIMS_PER_THREAD);
  if (chunk < 0 || softcap < 0.f) PYLON_REFUSE("paged_attention_simple: chunk %d, soft cap %f", chunk, softcap);
  if (keep_first < 0 || (keep_first > 0 && chunk > 0)) PYLON_REFUSE("paged_attention_simple: %d kept first keys (not with chunks)", keep_first);
  if (bias && bias_rows < 1) PYLON_REFUSE("paged_attention_simple: a bias table of %d rows", bias_rows);
  if (out_stride == 0) out_stride = (long long)nq * dv;
  if (out_stride < (long long)nq * dv || (score_bias && !sigmoid) || (sigmoid && (sinks || slopes))) PYLON_REFUSE("paged_attention_simple: output rows %lld apart, a number per head on the scores without sigmoid weights, or a sink with them", out_stride);
  if (nkv < 1 || nq < 1 || nq % nkv) PYLON_REFUSE("paged_attention_simple: %d query heads over %d KV heads", nq, nkv);
  if (nq > 65535) PYLON_REFUSE("paged_attention_simple: %d query heads", nq);
  if (page_size < 1 || table_width < 1 || window < 0)
    PYLON_REFUSE("paged_attention_simple: page size %d, table width %d, window %d", page_size, table_width, window);
  const size_t smem = (size_t)(d + SIMPLE_THREADS + 34) * sizeof(float) + SIMPLE_THREADS * sizeof(long long) + 8;
  dim3 grid(num_tokens, nq);
  if (dtype == PYLON_DTYPE_F32)
    paged_attention_simple_kernel<float><<<grid, SIMPLE_THREADS, smem, stream>>>(
        (const float*)q, q_token_stride, (const float*)k_pages, (const float*)v_pages, (float*)out, positions,
        token_row, block_table, table_width, page_size, num_pages, nq, nkv, d, dv, window, chunk, softcap, scale, sinks, k_row_stride, v_row_stride,
        keep_first, bias, bias_rows, sigmoid, score_bias, (const float*)gate, gate_stride, factor, out_stride, slopes, gate_elements);
  else if (dtype == PYLON_DTYPE_BF16)
    paged_attention_simple_kernel<__nv_bfloat16><<<grid, SIMPLE_THREADS, smem, stream>>>(
        (const __nv_bfloat16*)q, q_token_stride, (const __nv_bfloat16*)k_pages, (const __nv_bfloat16*)v_pages,
        (__nv_bfloat16*)out, positions, token_row, block_table, table_width, page_size, num_pages, nq, nkv, d, dv,
        window, chunk, softcap, scale, sinks, k_row_stride, v_row_stride, keep_first, bias, bias_rows, sigmoid, score_bias,
        (const __nv_bfloat16*)gate, gate_stride, factor, out_stride, slopes, gate_elements);
  else
    PYLON_REFUSE("paged_attention_simple: unknown dtype %d", dtype);
  PYLON_CHECK_LAUNCH("paged_attention_simple");
}
