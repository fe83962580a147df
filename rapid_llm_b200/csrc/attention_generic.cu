// Paged causal attention for any head size (steps of 16 up to 256; up to 640 in a second build of the
// kernel with more registers, for cached latent rows wider than the tensor-core tiles take), any number of heads
// and groups, any page size, with an optional window or chunks; one warp per (token, query head).
//
// This is the kernel of the float32 path and the fallback of the bfloat16 path for head
// sizes the tensor-core kernels are not instantiated for.  Every token of the step is a
// query row of its own: a portion of a prompt and a single decoded token differ only in
// how many rows a request contributes.  Keys and values are read from the cache through
// the request's block table, so the rows of this step must have been written before.
//
// Formula (rapid_llm/kernels/ops/attention/flashattention2_nopad.py:85,141-168 and
// rapid_llm/kernels/ops/attention/flashdecoding.py:223-230): kv head = q head // group;
// s_j = (q . k_j) * scale over the cached positions j <= p of the same request (and
// j > p - window when a window is set: the query's own position counts, as in
// rapid_llm/engine/kv_cache_spec.py:204,221-224; and j of the chunk p lies in when a chunk size is set); softmax over j; o = sum_j P_j v_j.
// With slopes, slope[head] * (p - j) is taken off the score (after a cap).  Scores, running maximum and sum, and the
// output accumulator are float32.
#include "common.cuh"

namespace rl {

constexpr int kGenericWarps = 4;
constexpr int kGenericMaxD = 256;
constexpr int kGenericWideD = 640;

template <typename T, int kMaxD>
__global__ void attention_generic_kernel(
    const T* __restrict__ q,            // [tokens, hq, d]
    const T* __restrict__ cache,        // [num_pages, kv_planes (2, or 1: values are the keys' rows), hkv, page_size, d]
    T* out,                             // [tokens, hq, d], rows out_stride apart
    int out_stride,
    const T* gate, int gate_stride,     // [tokens, hq] or null: head outputs are multiplied by its sigmoid
    const int* __restrict__ positions,  // [tokens]
    const int* __restrict__ token_slot, // [tokens]
    const int* __restrict__ block_table,  // [slots, max_pages]
    int tokens, int hq, int hkv, int d, int page_size, int num_pages, int max_pages, int slots,
    int window, int chunk, float scale, float softcap, const float* __restrict__ sink,
    const float* __restrict__ slopes, int kv_planes, int* __restrict__ fault) {
  __shared__ float q_staged[kGenericWarps][kMaxD];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long item = static_cast<long long>(blockIdx.x) * kGenericWarps + warp;
  if (item >= static_cast<long long>(tokens) * hq) return;
  const int t = static_cast<int>(item / hq);
  const int head = static_cast<int>(item - static_cast<long long>(t) * hq);
  const int kv_head = head / (hq / hkv);
  const int pos = positions[t];
  const int slot = token_slot[t];
  T* o = out + static_cast<size_t>(t) * out_stride + static_cast<size_t>(head) * d;
  if (slot < 0 || slot >= slots || pos < 0 || pos >= max_pages * page_size) {
    if (lane == 0) atomicOr(fault, slot < 0 || slot >= slots ? kFaultSlot : kFaultPosition);
    for (int i = lane; i < d; i += 32) o[i] = from_float<T>(0.0f);
    return;
  }
  const int* table = block_table + static_cast<size_t>(slot) * max_pages;

  float* qs = q_staged[warp];
  const T* qr = q + (static_cast<size_t>(t) * hq + head) * d;
  for (int i = lane; i < d; i += 32) qs[i] = to_float(qr[i]) * scale;
  __syncwarp();

  const float slope = slopes != nullptr ? slopes[head] : 0.0f;
  const int first = first_visible(pos, window, chunk);
  const size_t head_stride = static_cast<size_t>(page_size) * d;
  // K plane -> V plane; a cache of one plane keeps rows that are keys and values at once
  const size_t v_offset = kv_planes == 2 ? static_cast<size_t>(hkv) * head_stride : 0;

  float running_max = -INFINITY, running_sum = 0.0f;
  float acc[kMaxD / 32];
#pragma unroll
  for (int i = 0; i < kMaxD / 32; ++i) acc[i] = 0.0f;

  for (int base = first; base <= pos; base += 32) {
    const int j = base + lane;
    const bool valid = j <= pos;
    long long k_row = -1;  // element offset of key row j in the cache
    float score = -INFINITY;
    if (valid) {
      const int page = table[j / page_size];
      if (page < 0 || page >= num_pages) {
        atomicOr(fault, kFaultPageId);
      } else {
        k_row = static_cast<long long>(
            ((static_cast<size_t>(page) * kv_planes * hkv + kv_head) * page_size + (j % page_size)) * d);
        const T* kr = cache + k_row;
        float dot = 0.0f;
        for (int i = 0; i < d; i += 8) {
          float kv[8];
          load8(kr + i, kv);
#pragma unroll
          for (int e = 0; e < 8; ++e) dot = fmaf(qs[i + e], kv[e], dot);
        }
        // squashed scores: cap * tanh(s / cap) of the scaled score, where the mixer has a cap
        score = softcap > 0.0f ? softcap * tanhf(dot / softcap) : dot;
        score -= slope * static_cast<float>(pos - j);
      }
    }
    const float chunk_max = warp_max(score);
    const float new_max = fmaxf(running_max, chunk_max);
    if (new_max == -INFINITY) continue;  // every key of this chunk was unreadable
    const float p = (k_row >= 0) ? expf(score - new_max) : 0.0f;
    const float correction = expf(running_max - new_max);
    running_sum = running_sum * correction + warp_sum(p);
    running_max = new_max;
#pragma unroll
    for (int i = 0; i < kMaxD / 32; ++i) acc[i] *= correction;
    const int count = min(32, pos - base + 1);
    for (int jj = 0; jj < count; ++jj) {
      const float pj = __shfl_sync(0xffffffffu, p, jj);
      const long long row = __shfl_sync(0xffffffffu, k_row, jj);
      if (row < 0) continue;
      const T* vr = cache + row + v_offset;
#pragma unroll
      for (int i = 0; i < kMaxD / 32; ++i) {
        const int col = lane + 32 * i;
        if (col < d) acc[i] = fmaf(pj, to_float(vr[col]), acc[i]);
      }
    }
  }
  float inv_sum = running_sum > 0.0f ? 1.0f / running_sum : 0.0f;
  if (sink != nullptr) {
    // one more term exp(sink[head]) in the denominator, without a key or a value; it is neither scaled nor capped
    const float s = sink[head];
    const float top = fmaxf(running_max, s);
    const float keys = running_max == -INFINITY ? 0.0f : expf(running_max - top);
    inv_sum = keys / (running_sum * keys + expf(s - top));
  }
  inv_sum *= head_gate(gate, gate_stride, t, head);
#pragma unroll
  for (int i = 0; i < kMaxD / 32; ++i) {
    const int col = lane + 32 * i;
    if (col < d) o[col] = from_float<T>(acc[i] * inv_sum);
  }
}

}  // namespace rl

extern "C" int rl_attention_generic(int dtype, const void* q, const void* cache, void* out, int out_stride,
                                    const void* gate, int gate_stride,
                                    const int* positions, const int* token_slot,
                                    const int* block_table, int tokens, int hq, int hkv, int d,
                                    int page_size, int num_pages, int max_pages, int slots,
                                    int window, int chunk, float scale, float softcap, const float* sink, const float* slopes, int kv_planes,
                                    int* fault, cudaStream_t stream) {
  if (tokens == 0) return 0;
  if (d <= 0 || d % 16 != 0 || d > rl::kGenericWideD || hkv <= 0 || hq % hkv != 0 ||
      page_size <= 0 || window < 0 || chunk < 0 || (window > 0 && chunk > 0) || softcap < 0.0f ||
      out_stride < hq * d || (gate != nullptr && gate_stride < hq) || kv_planes < 1 || kv_planes > 2)
    return static_cast<int>(cudaErrorInvalidValue);
  const long long items = static_cast<long long>(tokens) * hq;
  const unsigned blocks =
      static_cast<unsigned>((items + rl::kGenericWarps - 1) / rl::kGenericWarps);
  RL_DISPATCH_DTYPE(dtype, {
    auto kernel = d <= rl::kGenericMaxD ? rl::attention_generic_kernel<scalar_t, rl::kGenericMaxD>
                                        : rl::attention_generic_kernel<scalar_t, rl::kGenericWideD>;
    kernel<<<blocks, rl::kGenericWarps * 32, 0, stream>>>(
        static_cast<const scalar_t*>(q), static_cast<const scalar_t*>(cache),
        static_cast<scalar_t*>(out), out_stride, static_cast<const scalar_t*>(gate), gate_stride, positions, token_slot, block_table, tokens, hq, hkv, d,
        page_size, num_pages, max_pages, slots, window, chunk, scale, softcap, sink, slopes, kv_planes, fault);
  });
  return rl::launch_status();
}
