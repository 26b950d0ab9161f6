// Prompt-regime projection over dense bf16 weights on the 5th-generation tensor cores: C[M, N] = X[M, K] W[N, K]^T with fp32
// accumulation in tensor memory.
//
// Persistent, one CTA per SM, output tiles of 128 rows x BN columns, K in blocks of 64:
//   warp 0      TMA producer (one thread): X tile and W tile of a K-block into a ring of stages, 128-byte swizzle
//   warp 1      tensor-memory owner and MMA issuer (one thread): four tcgen05.mma of K = 16 per block
//   warps 2-9   epilogue, two warps per lane quarter and half the columns each: tcgen05.ld of the accumulators, then the fused
//               epilogue of the projection
// The accumulators are double-buffered in tensor memory, so the epilogue of a tile runs under the MMAs of the next one.
// Every wait is bounded; one that runs out sets the status word and the kernel unwinds.
#include <algorithm>
#include <mutex>

#include "../tcgen05.cuh"
#include "dense.cuh"

namespace gptq {

int dense_tensor_map(const void *base, long long rows, long long cols, long long ld, int box_rows, int box_cols, CUtensorMap *out);

namespace {

constexpr int TD_BM = 128, TD_BK = 64, TD_EPI = 256, TD_THREADS = 64 + TD_EPI;
constexpr int TD_A_BYTES = TD_BM * TD_BK * 2;
constexpr uint32_t TD_SPIN = 1u << 24;
constexpr size_t TD_SMEM = 226 * 1024;

template <int BN> struct TdShape {
	static constexpr int STAGE = TD_A_BYTES + BN * TD_BK * 2;
	static constexpr int S = (int)((TD_SMEM - 2048) / STAGE) > 8 ? 8 : (int)((TD_SMEM - 2048) / STAGE);
	static constexpr size_t SMEM = (size_t)S * STAGE + 2048;      // 1 KB of alignment slack, 1 KB of barriers
	static constexpr uint32_t TMEM = 2 * BN < 32 ? 32 : 2 * BN;
};

template <int BN>
__global__ void __launch_bounds__(TD_THREADS, 1) dense_tc_kernel(const __grid_constant__ CUtensorMap tmx, const __grid_constant__ CUtensorMap tmw, const DenseArgs p,
																 int mt, int nt) {
	extern __shared__ unsigned char td_raw[];
	using Sh = TdShape<BN>;
	constexpr int S = Sh::S;
	constexpr uint32_t IDESC = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(BN >> 3) << 17) | ((uint32_t)(TD_BM >> 4) << 24);   // D fp32, A/B bf16 K-major
	unsigned char *smem = td_raw + ((1024u - (smem_u32(td_raw) & 1023u)) & 1023u);
	uint64_t *bars = reinterpret_cast<uint64_t *>(smem + (size_t)S * Sh::STAGE);
	const uint32_t bar_full = smem_u32(bars), bar_empty = smem_u32(bars + S), bar_acc = smem_u32(bars + 2 * S), bar_free = smem_u32(bars + 2 * S + 2);
	uint32_t *s_tmem = reinterpret_cast<uint32_t *>(bars + 2 * S + 4);
	volatile int *s_abort = reinterpret_cast<volatile int *>(s_tmem + 1);
	const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
	const int nkb = (p.K + TD_BK - 1) / TD_BK, ntiles = mt * nt;

	if (tid == 0) {
		for (int s = 0; s < S; ++s) {
			mbar_init(bar_full + 8 * s, 1);
			mbar_init(bar_empty + 8 * s, 1);
		}
		for (int s = 0; s < 2; ++s) {
			mbar_init(bar_acc + 8 * s, 1);
			mbar_init(bar_free + 8 * s, TD_EPI);
		}
		*s_abort = 0;
		fence_mbar_init();
		tma_prefetch_desc(&tmx);
		tma_prefetch_desc(&tmw);
	}
	if (warp == 1) {
		tmem_alloc(smem_u32(s_tmem), Sh::TMEM);
		tmem_relinquish();
	}
	tc_fence_before();
	__syncthreads();
	tc_fence_after();
	const uint32_t tmem = *s_tmem;
	auto fail = [&]() {
		*s_abort = 1;
		atomicExch(p.status, 3);
	};
	pdl_wait();
	pdl_trigger();

	if (warp == 0) {
		if (lane == 0) {
			int it = 0;
			for (int t = blockIdx.x; t < ntiles && !*s_abort; t += gridDim.x) {
				const int m0 = (t % mt) * TD_BM, n0 = (t / mt) * BN;
				for (int kb = 0; kb < nkb; ++kb, ++it) {
					const int s = it % S;
					if (*s_abort || !mbar_wait_bounded(bar_empty + 8 * s, ((it / S) & 1) ^ 1, TD_SPIN)) { fail(); break; }
					mbar_arrive_expect_tx(bar_full + 8 * s, Sh::STAGE);
					unsigned char *st = smem + (size_t)s * Sh::STAGE;
					tma_load_2d(smem_u32(st), &tmx, kb * TD_BK, m0, bar_full + 8 * s);              // rows and columns outside are zero-filled
					tma_load_2d(smem_u32(st + TD_A_BYTES), &tmw, kb * TD_BK, n0, bar_full + 8 * s);
				}
			}
			// leave only when every copy has landed (also after an abort): the stages' memory is freed at exit
			for (int i = max(0, it - S); i < it; ++i) mbar_wait_bounded(bar_full + 8 * (i % S), (i / S) & 1, TD_SPIN);
		}
	} else if (warp == 1) {
		if (lane == 0) {
			int it = 0, lt = 0;
			for (int t = blockIdx.x; t < ntiles && !*s_abort; t += gridDim.x, ++lt) {
				const int b = lt & 1;
				if (!mbar_wait_bounded(bar_free + 8 * b, ((lt >> 1) & 1) ^ 1, TD_SPIN)) { fail(); break; }
				tc_fence_after();
				for (int kb = 0; kb < nkb; ++kb, ++it) {
					const int s = it % S;
					if (*s_abort || !mbar_wait_bounded(bar_full + 8 * s, (it / S) & 1, TD_SPIN)) { fail(); break; }
					tc_fence_after();
					const uint32_t a = smem_u32(smem + (size_t)s * Sh::STAGE), w = a + TD_A_BYTES;
#pragma unroll
					for (int k = 0; k < TD_BK / 16; ++k)
						umma_f16(tmem + b * BN, smem_desc_sw128(a + k * 32), smem_desc_sw128(w + k * 32), IDESC, (kb > 0 || k > 0) ? 1u : 0u);
					umma_commit(bar_empty + 8 * s);
				}
				umma_commit(bar_acc + 8 * b);
			}
			// drain: the last commits of both buffers, before tensor memory goes back
			for (int i = max(0, lt - 2); i < lt; ++i) mbar_wait_bounded(bar_acc + 8 * (i & 1), (i >> 1) & 1, TD_SPIN);
		}
		__syncwarp();
	} else {
		const int q = warp & 3, half = (warp - 2) >> 2;
		int lt = 0;
		bool ok = true;
		for (int t = blockIdx.x; t < ntiles && ok; t += gridDim.x, ++lt) {
			const int b = lt & 1, m = (t % mt) * TD_BM + q * 32 + lane, n0 = (t / mt) * BN;
			ok = !*s_abort && mbar_wait_bounded(bar_acc + 8 * b, (lt >> 1) & 1, TD_SPIN);
			ok = __all_sync(0xffffffffu, ok);
			if (!ok) {
				fail();
				break;
			}
			tc_fence_after();
			const uint32_t t0 = tmem + b * BN + ((uint32_t)(q * 32) << 16);
#pragma unroll 1
			for (int c = 32 * half; c < BN; c += 64) {
				float v[2][16];
				tmem_ld16(t0 + c, v[0]);
				tmem_ld16(t0 + c + 16, v[1]);
				tmem_ld_wait();
#pragma unroll
				for (int i = 0; i < 16; ++i) asm volatile("" : "+f"(v[0][i]), "+f"(v[1][i]));
				if (m < p.M) {
					if (n0 + c < p.N) epi_16<bf16>(p.e, m, n0 + c, v[0]);
					if (n0 + c + 16 < p.N) epi_16<bf16>(p.e, m, n0 + c + 16, v[1]);
				}
			}
			tc_fence_before();
			mbar_arrive(bar_free + 8 * b);
		}
	}
	tc_fence_before();
	__syncthreads();
	if (warp == 1) tmem_dealloc(tmem, Sh::TMEM);
}

// ---- narrow outputs: a cluster of CTAs shares the K range of one output tile -------------------------------------------------------
// Every CTA accumulates its K blocks in its own tensor memory; then each gets a share of the tile's columns from all of them
// through distributed shared memory (the ring's stages, idle by then), adds the parts in rank order and runs the epilogue.
constexpr int TK_BN = 256, TK_STAGE = TD_A_BYTES + TK_BN * TD_BK * 2, TK_S = 4;
constexpr size_t TK_SMEM = (size_t)TK_S * TK_STAGE + 2048;

__global__ void __launch_bounds__(TD_THREADS, 1) dense_tc_cluster_kernel(const __grid_constant__ CUtensorMap tmx, const __grid_constant__ CUtensorMap tmw, const DenseArgs p,
																		 int mt, int parts) {
	extern __shared__ unsigned char tk_raw[];
	constexpr uint32_t IDESC = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(TK_BN >> 3) << 17) | ((uint32_t)(TD_BM >> 4) << 24);
	unsigned char *smem = tk_raw + ((1024u - (smem_u32(tk_raw) & 1023u)) & 1023u);
	uint64_t *bars = reinterpret_cast<uint64_t *>(smem + (size_t)TK_S * TK_STAGE);
	const uint32_t bar_full = smem_u32(bars), bar_empty = smem_u32(bars + TK_S), bar_acc = smem_u32(bars + 2 * TK_S);
	uint32_t *s_tmem = reinterpret_cast<uint32_t *>(bars + 2 * TK_S + 1);
	volatile int *s_abort = reinterpret_cast<volatile int *>(s_tmem + 1);
	const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, rank = (int)cluster_rank(), tile = blockIdx.x / parts;
	const int m0 = (tile % mt) * TD_BM, n0 = (tile / mt) * TK_BN;
	const int nkb = (p.K + TD_BK - 1) / TD_BK, k_lo = rank * nkb / parts, n = (rank + 1) * nkb / parts - k_lo;      // (nkb >= parts)
	if (tid == 0) {
		for (int s = 0; s < TK_S; ++s) {
			mbar_init(bar_full + 8 * s, 1);
			mbar_init(bar_empty + 8 * s, 1);
		}
		mbar_init(bar_acc, 1);
		*s_abort = 0;
		fence_mbar_init();
		tma_prefetch_desc(&tmx);
		tma_prefetch_desc(&tmw);
	}
	if (warp == 1) {
		tmem_alloc(smem_u32(s_tmem), TK_BN);
		tmem_relinquish();
	}
	tc_fence_before();
	__syncthreads();
	tc_fence_after();
	const uint32_t tmem = *s_tmem;
	auto fail = [&]() {
		*s_abort = 1;
		atomicExch(p.status, 3);
	};
	pdl_wait();
	pdl_trigger();
	if (warp == 0) {
		if (lane == 0) {
			int it = 0;
			for (; it < n; ++it) {
				const int s = it % TK_S;
				if (*s_abort || !mbar_wait_bounded(bar_empty + 8 * s, ((it / TK_S) & 1) ^ 1, TD_SPIN)) { fail(); break; }
				mbar_arrive_expect_tx(bar_full + 8 * s, TK_STAGE);
				unsigned char *st = smem + (size_t)s * TK_STAGE;
				tma_load_2d(smem_u32(st), &tmx, (k_lo + it) * TD_BK, m0, bar_full + 8 * s);              // rows and columns outside are zero-filled
				tma_load_2d(smem_u32(st + TD_A_BYTES), &tmw, (k_lo + it) * TD_BK, n0, bar_full + 8 * s);
			}
			for (int i = max(0, it - TK_S); i < it; ++i) mbar_wait_bounded(bar_full + 8 * (i % TK_S), (i / TK_S) & 1, TD_SPIN);
		}
		__syncwarp();
	} else if (warp == 1) {
		if (lane == 0) {
			for (int it = 0; it < n; ++it) {
				const int s = it % TK_S;
				if (*s_abort || !mbar_wait_bounded(bar_full + 8 * s, (it / TK_S) & 1, TD_SPIN)) { fail(); break; }
				tc_fence_after();
				const uint32_t a = smem_u32(smem + (size_t)s * TK_STAGE), w = a + TD_A_BYTES;
#pragma unroll
				for (int k = 0; k < TD_BK / 16; ++k) umma_f16(tmem, smem_desc_sw128(a + k * 32), smem_desc_sw128(w + k * 32), IDESC, (it > 0 || k > 0) ? 1u : 0u);
				umma_commit(bar_empty + 8 * s);
			}
			umma_commit(bar_acc);
		}
		__syncwarp();
	}
	// every warp waits for the CTA's own products; then the ring may be overwritten, here and (behind the barrier) by the others
	const bool ok = __all_sync(0xffffffffu, mbar_wait_bounded(bar_acc, 0, TD_SPIN)) && !*s_abort;
	if (!ok) fail();
	tc_fence_after();
	__syncwarp();
	cluster_arrive();
	cluster_wait();
	const int cols = TK_BN / parts, ld = cols + 4;                   // columns per rank; padded rows
	if (warp >= 2) {
		const int q = warp & 3, half = (warp - 2) >> 2, row = q * 32 + lane;
		const uint32_t src = smem_u32(smem) + (uint32_t)(rank * TD_BM + row) * ld * 4;
#pragma unroll 1
		for (int c = half * (TK_BN / 2); c < (half + 1) * (TK_BN / 2); c += 16) {
			float v[16];
			tmem_ld16(tmem + ((uint32_t)(q * 32) << 16) + c, v);
			tmem_ld_wait();
#pragma unroll
			for (int i = 0; i < 16; ++i) asm volatile("" : "+f"(v[i]));
			const int to = c / cols;
			const uint32_t dst = cluster_map(src + (uint32_t)(c - to * cols) * 4, (uint32_t)to);
#pragma unroll
			for (int i = 0; i < 4; ++i) cluster_store4(dst + 16 * i, v[4 * i], v[4 * i + 1], v[4 * i + 2], v[4 * i + 3]);
		}
	}
	__syncwarp();
	cluster_arrive();
	cluster_wait();
	if (warp >= 2 && ok) {
		const int t = tid - 64, row = t & (TD_BM - 1);
		for (int c = (t >> 7) * 16; c < cols; c += 32) {
			float v[16] = {};
			for (int r = 0; r < parts; ++r) {
				const float4 *f = reinterpret_cast<const float4 *>(reinterpret_cast<const float *>(smem) + (size_t)(r * TD_BM + row) * ld + c);
#pragma unroll
				for (int i = 0; i < 4; ++i) {
					const float4 x = f[i];
					v[4 * i] += x.x;
					v[4 * i + 1] += x.y;
					v[4 * i + 2] += x.z;
					v[4 * i + 3] += x.w;
				}
			}
			const int col = n0 + rank * cols + c;
			if (m0 + row < p.M && col < p.N) epi_16<bf16>(p.e, m0 + row, col, v);
		}
	}
	tc_fence_before();
	__syncthreads();
	if (warp == 1) tmem_dealloc(tmem, TK_BN);
}

int launch_cluster(const CUtensorMap &tmx, const DenseArgs &a, int parts, cudaStream_t stream) {
	alignas(64) CUtensorMap tmw;
	if (int rc = dense_tensor_map(a.w, a.N, a.K, a.ldw, TK_BN, TD_BK, &tmw)) return rc;
	const int mt = (a.M + TD_BM - 1) / TD_BM, nt = (a.N + TK_BN - 1) / TK_BN;
	return dn_launch_as(parts, -1, dense_tc_cluster_kernel, dim3(mt * nt * parts), dim3(TD_THREADS), TK_SMEM, stream, tmx, tmw, a, mt, parts);
}

template <int BN>
int launch(const CUtensorMap &tmx, const DenseArgs &a, cudaStream_t stream) {
	alignas(64) CUtensorMap tmw;
	if (int rc = dense_tensor_map(a.w, a.N, a.K, a.ldw, BN, TD_BK, &tmw)) return rc;
	const int mt = (a.M + TD_BM - 1) / TD_BM, nt = (a.N + BN - 1) / BN;
	return dn_launch(dense_tc_kernel<BN>, dim3(std::min(mt * nt, dn_sm_count())), dim3(TD_THREADS), TdShape<BN>::SMEM, stream, tmx, tmw, a, mt, nt);
}

}   // namespace

static EncodeTiledFn encoder() {
	static EncodeTiledFn fn = nullptr;
	static std::once_flag once;
	std::call_once(once, [] {
		void *ptr = nullptr;
		cudaDriverEntryPointQueryResult q;
		if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &ptr, cudaEnableDefault, &q) == cudaSuccess && q == cudaDriverEntryPointSuccess)
			fn = reinterpret_cast<EncodeTiledFn>(ptr);
	});
	return fn;
}

// bf16 matrix [rows, cols] with row stride ld (elements), boxes of box_rows x box_cols (box_cols * 2 <= 128 bytes), 128-byte swizzle
int dense_tensor_map(const void *base, long long rows, long long cols, long long ld, int box_rows, int box_cols, CUtensorMap *out) {
	EncodeTiledFn enc = encoder();
	if (!enc) return GPTQ_ERR_CUDA;
	cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows};
	cuuint64_t strides[1] = {(cuuint64_t)ld * 2};
	cuuint32_t box[2] = {(cuuint32_t)box_cols, (cuuint32_t)box_rows};
	cuuint32_t estr[2] = {1, 1};
	CUresult r = enc(out, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void *>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
					 CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
	if (r != CUDA_SUCCESS) {
		g_last_cuda_error = (int)r;
		return GPTQ_ERR_CUDA;
	}
	return GPTQ_OK;
}

int dense_tc_launch(const DenseArgs &a, cudaStream_t stream) {
	alignas(64) CUtensorMap tmx;
	if (int rc = dense_tensor_map(a.x, a.M, a.K, a.ldx, TD_BM, TD_BK, &tmx)) return rc;
	// column tile: whole waves of tiles, each costing its columns plus a fixed part (smaller tiles feed the tensor cores worse)
	const int sms = dn_sm_count(), mt = (a.M + TD_BM - 1) / TD_BM;
	// an output of few wide tiles and a long K: clusters that share K read the rows once instead of once per narrow tile
	const int wide = mt * ((a.N + TK_BN - 1) / TK_BN);
	if (a.N <= 2 * TK_BN && a.K >= 1024 && wide * 2 <= sms) {
		int parts = 8;
		while (wide * parts > sms) parts >>= 1;
		return launch_cluster(tmx, a, parts, stream);
	}
	const int bns[4] = {256, 128, 64, 32};
	int pick = 0;
	double best = 1e30;
	for (int i = 0; i < 4; ++i) {
		const long long tiles = (long long)mt * ((a.N + bns[i] - 1) / bns[i]), waves = (tiles + sms - 1) / sms;
		const double c = (double)waves * (bns[i] + (i ? 64 : 32));
		if (c < best) {
			best = c;
			pick = i;
		}
	}
	switch (pick) {
		case 0: return launch<256>(tmx, a, stream);
		case 1: return launch<128>(tmx, a, stream);
		case 2: return launch<64>(tmx, a, stream);
		default: return launch<32>(tmx, a, stream);
	}
}

}   // namespace gptq
