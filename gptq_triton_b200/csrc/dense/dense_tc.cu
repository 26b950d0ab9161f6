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

template <int BN, bool SPLIT>
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
	const int nkb = (p.K + TD_BK - 1) / TD_BK, parts = SPLIT ? p.parts : 1, ntiles = mt * nt * parts;
	auto k_first = [&](int t) { return SPLIT ? t % parts * nkb / parts : 0; };          // (SPLIT: consecutive CTAs share a tile)
	auto k_last = [&](int t) { return SPLIT ? (t % parts + 1) * nkb / parts : nkb; };

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
				const int tile = t / parts, m0 = (tile % mt) * TD_BM, n0 = (tile / mt) * BN;
				for (int kb = k_first(t); kb < k_last(t); ++kb, ++it) {
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
				const int k0 = k_first(t);
				for (int kb = k0; kb < k_last(t); ++kb, ++it) {
					const int s = it % S;
					if (*s_abort || !mbar_wait_bounded(bar_full + 8 * s, (it / S) & 1, TD_SPIN)) { fail(); break; }
					tc_fence_after();
					const uint32_t a = smem_u32(smem + (size_t)s * Sh::STAGE), w = a + TD_A_BYTES;
#pragma unroll
					for (int k = 0; k < TD_BK / 16; ++k)
						umma_f16(tmem + b * BN, smem_desc_sw128(a + k * 32), smem_desc_sw128(w + k * 32), IDESC, (kb > k0 || k > 0) ? 1u : 0u);
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
			const int tile = t / parts, b = lt & 1, m = (tile % mt) * TD_BM + q * 32 + lane, n0 = (tile / mt) * BN;
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
				if (SPLIT) {
					const int n16 = (p.N + 15) & ~15;
					float *ws = p.ws + ((size_t)(t % parts) * p.M + m) * n16 + n0 + c;
#pragma unroll
					for (int h = 0; h < 2; ++h)
						if (m < p.M && n0 + c + 16 * h < p.N) {
							Elem<float>::store8(ws + 16 * h, v[h]);
							Elem<float>::store8(ws + 16 * h + 8, v[h] + 8);
						}
				} else if (m < p.M) {
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

// ---- narrow outputs: the K range of a tile split over CTAs, fp32 parts in scratch memory, summed in order by a second kernel ---------
__global__ void __launch_bounds__(DN_THREADS) dense_finish_kernel(const DenseArgs p, int n16) {
	const int groups = n16 >> 4, i = blockIdx.x * DN_THREADS + threadIdx.x, m = i / groups, n = (i - m * groups) * 16;
	pdl_wait();
	pdl_trigger();
	if (m >= p.M) return;
	float v[16] = {};
	for (int r = 0; r < p.parts; ++r) {
		const float4 *f = reinterpret_cast<const float4 *>(p.ws + ((size_t)r * p.M + m) * n16 + n);
#pragma unroll
		for (int k = 0; k < 4; ++k) {
			const float4 x = __ldcg(f + k);
			v[4 * k] += x.x;
			v[4 * k + 1] += x.y;
			v[4 * k + 2] += x.z;
			v[4 * k + 3] += x.w;
		}
	}
	epi_16<bf16>(p.e, m, n, v);
}

template <int BN, bool SPLIT = false>
int launch(const CUtensorMap &tmx, const DenseArgs &a, cudaStream_t stream) {
	alignas(64) CUtensorMap tmw;
	if (int rc = dense_tensor_map(a.w, a.N, a.K, a.ldw, BN, TD_BK, &tmw)) return rc;
	const int mt = (a.M + TD_BM - 1) / TD_BM, nt = (a.N + BN - 1) / BN;
	return dn_launch(dense_tc_kernel<BN, SPLIT>, dim3(std::min(mt * nt * (SPLIT ? a.parts : 1), dn_sm_count())), dim3(TD_THREADS), TdShape<BN>::SMEM, stream, tmx, tmw, a, mt, nt);
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

// An MMA with its first operand in shared memory takes as long for 32 columns as for 256, so a narrow output wants wide tiles and a
// split K: parts per tile, 1 where the plain kernel is better.
int dense_tc_parts(int M, int K, int N) {
	const int wide = (M + TD_BM - 1) / TD_BM * ((N + 255) / 256), most = std::min(dn_sm_count() / std::max(1, wide), K / (16 * TD_BK));
	return N <= 512 && most >= 2 ? std::min(most, 8) : 1;
}

int dense_tc_launch(const DenseArgs &a, cudaStream_t stream) {
	alignas(64) CUtensorMap tmx;
	if (int rc = dense_tensor_map(a.x, a.M, a.K, a.ldx, TD_BM, TD_BK, &tmx)) return rc;
	// column tile: whole waves of tiles, each costing its columns plus a fixed part (smaller tiles feed the tensor cores worse)
	const int sms = dn_sm_count(), mt = (a.M + TD_BM - 1) / TD_BM;
	if (a.ws && dense_tc_parts(a.M, a.K, a.N) > 1) {
		DenseArgs d = a;
		d.parts = dense_tc_parts(a.M, a.K, a.N);
		if (int rc = launch<256, true>(tmx, d, stream)) return rc;
		const int n16 = (a.N + 15) / 16 * 16;
		return dn_launch(dense_finish_kernel, dim3((unsigned)(((long long)a.M * (n16 / 16) + DN_THREADS - 1) / DN_THREADS)), dim3(DN_THREADS), 0, stream, d, n16);
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
