// What the tensor-core attention kernels for prompts share.
#pragma once

#include "../tcgen05.cuh"
#include "dense.cuh"

namespace gptq {

int dense_tensor_map(const void *base, long long rows, long long cols, long long ld, int box_rows, int box_cols, CUtensorMap *out);

constexpr uint32_t ATTN_SPIN = 1u << 24;          // polls of a bounded wait

__device__ __forceinline__ float ex2(float x) {
	float r;
	asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
	return r;
}
// One poll inline; the bounded loop (and the look at the abort flag) out of line, so that the code of a wait that is already
// over stays short.
static __device__ __noinline__ bool wait_slow(uint32_t bar, uint32_t parity, volatile int *abort_flag) {
	return !*abort_flag && mbar_wait_bounded(bar, parity, ATTN_SPIN);
}
__device__ __forceinline__ bool wait_fast(uint32_t bar, uint32_t parity, volatile int *abort_flag) {
	return mbar_try_wait(bar, parity) || wait_slow(bar, parity, abort_flag);
}
// registers loaded by tcgen05.ld may be used only behind the wait: tie them to it
template <int N>
__device__ __forceinline__ void tmem_settle(float (&v)[N]) {
#pragma unroll
	for (int i = 0; i < N; ++i) asm volatile("" : "+f"(v[i]));
}

}   // namespace gptq
