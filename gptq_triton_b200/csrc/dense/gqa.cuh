// Launchers of the grouped-query attention kernels (one or two softmax maps per head).
#pragma once

#include "dense.cuh"

namespace gptq {

using GqaArgs = dense_gqa_t;

constexpr float GQ_LOG2E = 1.4426950408889634f;

// Queries are stored times scale / cap (or times scale * log2(e) without a cap), so that a product with a key is the argument of
// the tanh (or the score in base 2).
__host__ __device__ __forceinline__ float gqa_query_factor(const GqaArgs &p) { return p.cap > 0.f ? p.scale / p.cap : p.scale * GQ_LOG2E; }
// score in base 2 from that product
__device__ __forceinline__ float gqa_score(float v, float cap2) { return cap2 > 0.f ? cap2 * tanhf(v) : v; }

int gqa_append_launch(const GqaArgs &p, int dtype, cudaStream_t stream);
bool gqa_attend_ok(int maps, int dim, int vdim);
int gqa_splits(int M, int heads, int kv_heads, int maps, int max_seq, int dtype);
int gqa_attend_launch(const GqaArgs &p, int dtype, cudaStream_t stream);
int gqa_prefill_maps(int maps, int dim, int vdim);      // maps per CTA of the prompt kernel: 2 (writes out), 1 (writes partials), 0: does not fit
int gqa_prefill_launch(const GqaArgs &p, int start, cudaStream_t stream);
int gqa_merge_launch(const GqaArgs &p, int dtype, cudaStream_t stream);

}   // namespace gptq
