// Launchers of the state-space recurrence kernels.
#pragma once

#include "dense.cuh"

namespace gptq {

using SsmArgs = dense_ssm_t;

constexpr int SS_MAX_STATE = 256, SS_MAX_TAPS = 16, SS_CHUNK = DENSE_SSM_CHUNK;

__device__ __forceinline__ float ssm_softplus(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }

int ssm_step_launch(const SsmArgs &p, cudaStream_t stream);
int ssm_conv_launch(const SsmArgs &p, int dtype, cudaStream_t stream);
int ssm_scan_launch(const SsmArgs &p, cudaStream_t stream);
bool ssm_tc_ok(const SsmArgs &p);
int ssm_tc_launch(const SsmArgs &p, cudaStream_t stream);      // a launch per sequence
int ssm_chunk_launch(const SsmArgs &p, cudaStream_t stream);

}   // namespace gptq
