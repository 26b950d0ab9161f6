// Launchers of the latent-attention kernels.
#pragma once

#include "dense.cuh"

namespace gptq {

using LatentArgs = dense_latent_t;               // sizes are the padded ones; kv_width is what the RMS norm averages over
using LatentPrefill = dense_latent_prefill_t;

int latent_absorb_launch(const LatentArgs &p, bool queries, int dtype, cudaStream_t stream);
bool latent_attend_ok(int kv_rank, int rot_dim);
int latent_splits(int M, int heads, int max_seq, int dtype);
int latent_attend_launch(const LatentArgs &p, int dtype, cudaStream_t stream);
int latent_value_launch(const LatentArgs &p, int dtype, cudaStream_t stream);
bool latent_prefill_ok(int dim, int rot_dim, int vdim);
int latent_prefill_launch(const LatentPrefill &p, cudaStream_t stream);

}   // namespace gptq
