// What the grouped-attention kernels share: which keys a query sees, and the extra term of the softmax.
//
// Cache layout (one page of one cache entry), the one of the differential attention with one key map
// (DiffCache with kd = dim):
//   keys   [kv_head][position in page][dim]    at offset 0
//   values [kv_head][position in page][vd]     at offset nkv * page_size * dim
//
// Mask.  The query at position p sees key j when j <= p and (p - j < window or j < keep_first); window <= 0:
// every j <= p.  With chunk > 0 it sees only keys of its own run of `chunk` positions (counted from position 0) beside
// those of keep_first.  The seen keys are two ranges of positions: the kept first ones [0, head_end) with
// head_end = min(keep_first, lo), and the recent ones [lo, p] with lo the larger of max(0, p - window + 1) and the
// run's first position; lo never falls as p grows.
//
// Softmax.  With has_sink the denominator holds one more term exp(sink) that has no value row:
//   w_j = exp(s_j) / (exp(sink) + sum_i exp(s_i)).
#pragma once
#include "diff_attention.cuh"

struct GqaMask {
    int window, keep_first, chunk;
};

__device__ __forceinline__ int gqa_lo(int pos, const GqaMask& m) {
    const int lo = m.window > 0 ? max(0, pos - m.window + 1) : 0;
    return m.chunk > 0 ? max(lo, pos - pos % m.chunk) : lo;
}
__device__ __forceinline__ bool gqa_limited(const GqaMask& m) { return m.window > 0 || m.chunk > 0; }
__device__ __forceinline__ int gqa_head_end(int lo, const GqaMask& m) { return min(m.keep_first, lo); }
// lo: gqa_lo of the query's position
__device__ __forceinline__ bool gqa_seen(int key, int pos, int lo, const GqaMask& m) {
    return key <= pos && (key >= lo || key < m.keep_first);
}

// What is done to a head's result before it is stored: times out_scale, and, with gate, times
// sigmoid(gate[token * gate_ld + head * vd + e]) (gate logits as a product left them, in the storage type), or, with
// gate_heads, times sigmoid(gate[token * gate_ld + head]): one number for the whole head.
// sinks: with has_sink, the extra term's logit of every head (float [heads]); null: the one `sink` for all heads.
struct GqaEpilogue {
    const void* gate;
    long long gate_ld;
    float out_scale;
    const float* sinks;
    int gate_heads;
};

__device__ __forceinline__ float sigmoidf_(float z) { return 1.f / (1.f + expf(-z)); }
