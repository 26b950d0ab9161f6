// Decode-regime projection (M <= 8 rows) over dense weights [N, K], HBM-bound: every weight is read once with 16-byte loads
// straight into registers, double-buffered so that loads are always in flight across tile boundaries.
//
// A CTA of 8 warps owns tiles of 16 weight rows (strided over the grid) and splits K over its warps.  bf16: the weight rows
// are the A operand of mma.m16n8k16 and the activations the B operand.  A dot product does not care about the order of k, so
// lane (gid, tig) feeds the eight consecutive k that its 16-byte loads deliver for rows gid and gid + 8 and the same eight k
// of activation row gid: two MMAs per pair of loads, no shuffle.  fp32: the same layout on the FMA units.
// Few tiles (a narrow projection) leave most SMs idle: then a cluster of CTAs shares a tile's K, the partial sums meet in the first
// CTA's shared memory.
// The prologue optionally prepares the rows itself (embedding lookup, residual, norm), the epilogue applies what
// follows the projection (rotary queries / raw latent / gates, act(gate) * up, scaled logits with the greedy choice).
#include <algorithm>

#include "dense.cuh"

namespace gptq {

namespace {

constexpr int SK_M = 8, SK_U = 4, SK_REDLD = 17, SK_PARTS = 8;
constexpr size_t SK_STATIC = (2 * DN_WARPS * SK_M * SK_REDLD + RP_SMEM) * sizeof(float) + 64;
constexpr size_t SK_SMEM_MAX = 227 * 1024 - SK_STATIC - 1024;

template <typename T, bool SPLIT>
__global__ void __launch_bounds__(DN_THREADS, 2) dense_skinny_kernel(const DenseArgs p, int kparts) {
	constexpr int E = 16 / sizeof(T);            // elements per 16-byte load
	constexpr int STEP = 4 * E;                  // k per step of a warp
	extern __shared__ __align__(16) unsigned char sk_smem[];
	__shared__ float s_red[2][DN_WARPS][SK_M][SK_REDLD];
	__shared__ float s_norm[RP_SMEM];
	__shared__ int s_last;
	__shared__ float2 s_part[SPLIT ? SK_PARTS : 1][SPLIT ? 8 * SK_M : 1];
	if (SPLIT) cluster_arrive();                 // (every CTA of the cluster runs before its shared memory is written)
	const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gid = lane >> 2, tig = lane & 3;
	const int xs = p.K * (int)sizeof(T) + 16;    // bytes per staged row
	const int rank = SPLIT ? (int)cluster_rank() : 0, tile0 = SPLIT ? (int)blockIdx.x / kparts : (int)blockIdx.x, stride = SPLIT ? (int)gridDim.x / kparts : (int)gridDim.x;
	const int slots = DN_WARPS * (SPLIT ? kparts : 1);
	const int nsteps = (p.K + STEP - 1) / STEP, spw = (nsteps + slots - 1) / slots;
	const int s0 = min((rank * DN_WARPS + warp) * spw, nsteps), s1 = min(s0 + spw, nsteps);
	const int nbatch = (spw + SK_U - 1) / SK_U;
	const int ntiles = (p.N + 15) >> 4;
	const int mytiles = (ntiles - tile0 + stride - 1) / stride;          // (SPLIT: one)
	const int total = mytiles * nbatch;
	const T *w = reinterpret_cast<const T *>(p.w);

	uint4 wa[2][SK_U], wb[2][SK_U];
	auto load = [&](int it, uint4 (&a)[SK_U], uint4 (&b)[SK_U]) {
		const int ti = it / nbatch, bi = it - ti * nbatch;
		const int row = (tile0 + ti * stride) * 16 + gid;
		const T *pa = w + (size_t)min(row, p.N - 1) * p.ldw, *pb = w + (size_t)min(row + 8, p.N - 1) * p.ldw;
#pragma unroll
		for (int u = 0; u < SK_U; ++u) {
			const int s = s0 + bi * SK_U + u, k = s * STEP + tig * E;
			if (s < s1 && k < p.K) {
				a[u] = ld_nc_v4(pa + k);
				b[u] = ld_nc_v4(pb + k);
			} else {
				a[u] = make_uint4(0u, 0u, 0u, 0u);
				b[u] = a[u];
			}
		}
	};
	load(0, wa[0], wb[0]);                       // weights do not depend on earlier kernels
	pdl_wait();
	pdl_trigger();

	// ---- stage the rows -------------------------------------------------------------------------------------------
	if (p.prep) {
		for (int m = 0; m < p.M; ++m) {
			if (m) __syncthreads();
			prepare_row<T>(p.rp, m, reinterpret_cast<T *>(sk_smem + (size_t)m * xs), p.rp.x_out != nullptr && blockIdx.x == 0, s_norm);
		}
	} else {
		const int units = p.K / E;
		for (int m = 0; m < p.M; ++m) {
			const uint4 *src = reinterpret_cast<const uint4 *>(reinterpret_cast<const T *>(p.x) + (size_t)m * p.ldx);
			for (int u = tid; u < units; u += DN_THREADS) *reinterpret_cast<uint4 *>(sk_smem + (size_t)m * xs + u * 16) = __ldcg(src + u);
		}
	}
	__syncthreads();

	float d[4] = {0.f, 0.f, 0.f, 0.f};           // bf16 accumulators
	float f[2][SK_M];                            // fp32 accumulators: rows gid, gid + 8 by activation row
#pragma unroll
	for (int m = 0; m < SK_M; ++m) f[0][m] = f[1][m] = 0.f;
	const unsigned char *xrow = sk_smem + (size_t)min(gid, p.M - 1) * xs;
	const bool live = gid < p.M;
	unsigned long long best = 0ull;              // LOGITS: running candidate of thread (m = tid / 8)

	float part_a = 0.f, part_b = 0.f;            // SPLIT: this CTA's share of the results of threads below 8 M
	auto finish = [&](int m, int j, int tile, float va, float vb) {
		if (p.e.mode == DENSE_EPI_GATED) {
			Elem<T>::store(reinterpret_cast<T *>(p.e.out) + (size_t)m * p.e.ldo + tile * 8 + j, activation(p.e.act, va) * vb);
			return;
		}
		const int n = tile * 16 + 2 * j;
		epi_pair<T>(p.e, m, n, va, vb);
		if (p.e.mode == DENSE_EPI_LOGITS) {
			if (n < p.N) best = max(best, argmax_key(va * p.e.scale, n));
			if (n + 1 < p.N) best = max(best, argmax_key(vb * p.e.scale, n + 1));
		}
	};
	auto compute = [&](int it, uint4 (&a)[SK_U], uint4 (&b)[SK_U]) {
		const int ti = it / nbatch, bi = it - ti * nbatch;
#pragma unroll
		for (int u = 0; u < SK_U; ++u) {
			const int s = s0 + bi * SK_U + u, k = min(s * STEP + tig * E, p.K - E);      // beyond the range the weights are zero
			if (sizeof(T) == 2) {
				uint4 x = make_uint4(0u, 0u, 0u, 0u);
				if (live) x = *reinterpret_cast<const uint4 *>(xrow + k * 2);
				mma16816_bf16(d, a[u].x, b[u].x, a[u].y, b[u].y, x.x, x.y);
				mma16816_bf16(d, a[u].z, b[u].z, a[u].w, b[u].w, x.z, x.w);
			} else {
#pragma unroll
				for (int m = 0; m < SK_M; ++m) {
					if (m < p.M) {
						const float4 x = *reinterpret_cast<const float4 *>(sk_smem + (size_t)m * xs + k * 4);
						f[0][m] = fmaf(__uint_as_float(a[u].x), x.x, fmaf(__uint_as_float(a[u].y), x.y, fmaf(__uint_as_float(a[u].z), x.z, fmaf(__uint_as_float(a[u].w), x.w, f[0][m]))));
						f[1][m] = fmaf(__uint_as_float(b[u].x), x.x, fmaf(__uint_as_float(b[u].y), x.y, fmaf(__uint_as_float(b[u].z), x.z, fmaf(__uint_as_float(b[u].w), x.w, f[1][m]))));
					}
				}
			}
		}
		if (bi != nbatch - 1) return;
		// ---- end of a tile: sum the warps' K slices (fixed order), epilogue ----------------------------------------
		float(*red)[SK_M][SK_REDLD] = s_red[ti & 1];
		if (sizeof(T) == 2) {
			const int c = 2 * tig;
			if (c < p.M) {
				red[warp][c][gid] = d[0];
				red[warp][c][gid + 8] = d[2];
			}
			if (c + 1 < p.M) {
				red[warp][c + 1][gid] = d[1];
				red[warp][c + 1][gid + 8] = d[3];
			}
			d[0] = d[1] = d[2] = d[3] = 0.f;
		} else {
#pragma unroll
			for (int m = 0; m < SK_M; ++m) {
				if (m < p.M) {
#pragma unroll
					for (int r = 0; r < 2; ++r) {
						float v = f[r][m];
						v += __shfl_xor_sync(0xffffffffu, v, 1);
						v += __shfl_xor_sync(0xffffffffu, v, 2);
						if (tig == 0) red[warp][m][gid + 8 * r] = v;
						f[r][m] = 0.f;
					}
				}
			}
		}
		__syncthreads();                         // the buffer is written again two tiles later, behind the next tile's barrier
		if (tid < 8 * p.M) {
			const int m = tid >> 3, j = tid & 7, tile = tile0 + ti * stride;
			const bool gated = p.e.mode == DENSE_EPI_GATED;
			const int ra = gated ? j : 2 * j, rb = gated ? j + 8 : 2 * j + 1;
			float va = 0.f, vb = 0.f;
#pragma unroll
			for (int i = 0; i < DN_WARPS; ++i) {
				va += red[i][m][ra];
				vb += red[i][m][rb];
			}
			if (SPLIT) {
				part_a = va;
				part_b = vb;
			} else {
				finish(m, j, tile, va, vb);
			}
		}
	};
#pragma unroll 1
	for (int it = 0; it < total; it += 2) {
		if (it + 1 < total) load(it + 1, wa[1], wb[1]);
		compute(it, wa[0], wb[0]);
		if (it + 2 < total) load(it + 2, wa[0], wb[0]);
		if (it + 1 < total) compute(it + 1, wa[1], wb[1]);
	}

	if (SPLIT) {
		__syncwarp();
		cluster_wait();
		if (tid < 8 * p.M) cluster_store2(cluster_map(smem_u32(&s_part[rank][tid]), 0), part_a, part_b);
		__syncwarp();
		cluster_arrive();
		cluster_wait();
		if (rank == 0 && tid < 8 * p.M) {
			float va = 0.f, vb = 0.f;
			for (int i = 0; i < kparts; ++i) {
				va += s_part[i][tid].x;
				vb += s_part[i][tid].y;
			}
			finish(tid >> 3, tid & 7, tile0, va, vb);
		}
		return;
	}
	if (p.e.mode != DENSE_EPI_LOGITS || !p.e.best) return;
	// ---- greedy choice: one candidate per CTA and row, the last CTA writes token and position ----------------------------
	if (tid < 8 * SK_M) {                        // whole warps
#pragma unroll
		for (int s = 1; s < 8; s <<= 1) best = max(best, __shfl_xor_sync(0xffffffffu, best, s));
		if (tid < 8 * p.M && (tid & 7) == 0) atomicMax(p.e.best + (tid >> 3), best);
	}
	__syncthreads();
	if (tid == 0) {
		unsigned t;
		asm volatile("atom.acq_rel.gpu.global.add.u32 %0, [%1], 1;" : "=r"(t) : "l"(p.e.ticket) : "memory");
		s_last = t == gridDim.x - 1;
		if (s_last) *p.e.ticket = 0u;
	}
	__syncthreads();
	if (s_last && tid < p.M) {
		const unsigned long long b = atomicExch(p.e.best + tid, 0ull);
		p.e.tok[tid] = (int64_t)(uint32_t)~(uint32_t)b;
		p.e.pos_inout[tid] += 1;
	}
}

template <typename T>
int launch(const DenseArgs &a, cudaStream_t stream) {
	const size_t smem = (size_t)a.M * ((size_t)a.K * sizeof(T) + 16);
	const int ntiles = (a.N + 15) / 16, slots = dn_sm_count() * (smem + SK_STATIC > 110 * 1024 ? 1 : 2);
	// few tiles with long rows: a cluster per tile, as long as every warp of it has a step of K (with shorter rows the launch of a
	// cluster costs more than it saves)
	int kparts = a.K * (int)sizeof(T) > 8192 ? SK_PARTS : 1;
	while (kparts > 1 && (ntiles * kparts > dn_sm_count() || a.K < kparts * DN_WARPS * 64 / (int)sizeof(T))) kparts >>= 1;
	if (kparts > 1 && !a.e.best && smem <= 160 * 1024) return dn_launch_as(kparts, -1, dense_skinny_kernel<T, true>, dim3(ntiles * kparts), dim3(DN_THREADS), smem, stream, a, kparts);
	const int waves = (ntiles + slots - 1) / slots;
	return dn_launch(dense_skinny_kernel<T, false>, dim3((ntiles + waves - 1) / waves), dim3(DN_THREADS), smem, stream, a, 1);
}

}   // namespace

bool dense_skinny_ok(int M, int K, int dtype) { return M >= 1 && M <= SK_M && (size_t)M * ((size_t)K * (dtype ? 4 : 2) + 16) <= SK_SMEM_MAX; }

int dense_skinny_launch(const DenseArgs &a, int dtype, cudaStream_t stream) {
	return dtype ? launch<float>(a, stream) : launch<bf16>(a, stream);
}

// ---- the same row preparation as a kernel of its own (prompts, and many rows) -------------------------------------------
template <typename T>
__global__ void __launch_bounds__(DN_THREADS) dense_rows_kernel(const RowPrep p, T *h, long long ldh) {
	__shared__ float s_norm[RP_SMEM];
	pdl_wait();
	pdl_trigger();
	prepare_row<T>(p, blockIdx.x, h + (size_t)blockIdx.x * ldh, p.x_out != nullptr, s_norm);
}

int dense_rows_launch(const RowPrep &p, int M, void *h, long long ldh, int dtype, cudaStream_t stream) {
	if (dtype) return dn_launch(dense_rows_kernel<float>, dim3(M), dim3(DN_THREADS), 0, stream, p, reinterpret_cast<float *>(h), ldh);
	return dn_launch(dense_rows_kernel<bf16>, dim3(M), dim3(DN_THREADS), 0, stream, p, reinterpret_cast<bf16 *>(h), ldh);
}

}   // namespace gptq
