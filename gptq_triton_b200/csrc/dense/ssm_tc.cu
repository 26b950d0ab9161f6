// The chunked recurrence (see ssm_chunk.cu for the arithmetic) on the 5th-generation tensor cores, one kernel per prompt portion: a CTA
// owns up to 64 value entries of one head and walks the chunks of 128 tokens, the state stays in tensor memory from the first to
// the last.  Per chunk, with s_i the prefix sums of a * dt (base 2), w_j = log2(dt_j) - s_j, all fp32:
//   G  = C B^T                                  128 x 128, in tensor memory
//   M  = G_ij 2^(s_i + w_j), j <= i             written over G as bf16 high parts and remainders
//   Ya = M X,  Yi = C S                         S as two bf16 parts in shared memory
//   y  = 2^s_i Yi + Ya + d x, times silu(z)
//   S <- 2^s_last S + sum_j B_j (2^(s_last - s_j) dt_j x_j)^T     accumulates in tensor memory; the scaled inputs as two bf16 parts
// Differences of prefix sums must stay exact behind tokens that decay by orders of magnitude, so the sums are formed in fp64 and kept as
// an fp32 value hi and a remainder lo; log2(dt_j) joins the remainder of the second one.
//   warps 0-7   scale the inputs, split and decay S, form M, write y        warp 8   TMA: C, B, X tiles, two stages
//   warp 10     step sizes and prefix sums of the next chunk                 warp 9   MMA
// B and C are operands in both roles (rows of tokens as rows, and as the summed dimension); shared memory holds them once, in the
// 128-byte-swizzled layout that serves both.  The two parts of S are one operand of twice the width, their products are added when
// y is formed.  An MMA whose first operand comes from shared memory costs about 120 cycles however narrow it is, so the products
// of a chunk take about as long as the other warps' work; these prepare the next chunk between forming M and reading y.
// Outputs pass through the input tile, which nobody needs any more, so that global memory sees whole rows.  Every wait is bounded.
#include <algorithm>

#include "prefill_common.cuh"
#include "ssm.cuh"

namespace gptq {

namespace {

constexpr int ST_L = SS_CHUNK, ST_P = 64;
constexpr int ST_CHUNK = ST_L * 128;                    // bytes of a 128 x 64 bf16 tile
constexpr int ST_WORK = 256, ST_THREADS = ST_WORK + 96;
constexpr uint32_t T_G = 0, T_YI = 128, T_YA = 384, T_S = 448;      // tensor memory columns: G / M, two buffers of Yi (both parts of S), Ya, S

struct StPlan {
	int nc;                                             // 64-column tiles of C
	uint32_t stage;
	size_t smem;
};
__host__ __device__ inline StPlan st_plan(int state) {
	StPlan pl;
	pl.nc = (state + 63) / 64;
	pl.stage = (uint32_t)(pl.nc + 2 + 1) * ST_CHUNK;      // C, B (always two tiles: 128 rows of S), X
	pl.smem = 2 * (size_t)pl.stage + 4 * ST_CHUNK + 2 * ST_L * (2 * sizeof(float) + sizeof(bf16)) + 128;
	return pl;
}

// operand whose other dimension is contiguous: 64-column tiles ST_CHUNK apart, groups of 8 rows of 128 bytes
__device__ __forceinline__ uint64_t desc_rows(uint32_t addr) {
	uint64_t d = 0;
	d |= (uint64_t)((addr & 0x3FFFFu) >> 4);
	d |= (uint64_t)(ST_CHUNK >> 4) << 16;
	d |= (uint64_t)(1024 >> 4) << 32;
	d |= (uint64_t)1 << 46;
	d |= (uint64_t)2 << 61;
	return d;
}
__device__ __forceinline__ void st_split(float a, float b, uint32_t &hi, uint32_t &lo) {
	hi = pack_bf16(a, b);
	lo = pack_bf16(a - __uint_as_float(hi << 16), b - __uint_as_float(hi & 0xFFFF0000u));
}

__global__ void __launch_bounds__(ST_THREADS, 1) ssm_tc_kernel(const __grid_constant__ CUtensorMap tmu, const SsmArgs p, int seq) {
	extern __shared__ __align__(1024) unsigned char st_smem[];
	const StPlan pl = st_plan(p.state);
	const uint32_t base = smem_u32(st_smem), sxs = base + 2 * pl.stage, sst = sxs + 2 * ST_CHUNK;      // scaled inputs, S: high parts, remainders
	// prefix sums: hi, log2(dt) - lo, lo (bf16 is enough for it); two stages each
	float *s_hi = reinterpret_cast<float *>(st_smem + 2 * (size_t)pl.stage + 4 * ST_CHUNK), *s_w = s_hi + 2 * ST_L;
	bf16 *s_lo = reinterpret_cast<bf16 *>(s_w + 2 * ST_L);
	uint64_t *bars = reinterpret_cast<uint64_t *>(s_lo + 2 * ST_L);
	const uint32_t b0 = smem_u32(bars);
	const uint32_t bar_full = b0, bar_empty = b0 + 16, bar_g = b0 + 32, bar_r = b0 + 48, bar_m = b0 + 56, bar_y = b0 + 64, bar_u = b0 + 72, bar_end = b0 + 80;
	uint32_t *s_tmem = reinterpret_cast<uint32_t *>(bars + 11);
	volatile int *s_abort = reinterpret_cast<volatile int *>(s_tmem + 1);
	const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
	const int slices = (p.vdim + ST_P - 1) / ST_P, head = blockIdx.x / slices, p0 = (blockIdx.x - head * slices) * ST_P;
	const int np = min(ST_P, p.vdim - p0), g = head / (p.heads / p.groups), inner = p.heads * p.vdim;
	const int T = p.rows_per_seq, n = (T + ST_L - 1) / ST_L;
	if (base & 1023u) {                                 // (dynamic shared memory starts on a 1 KB boundary when there is no other)
		if (tid == 0) atomicExch(p.status, 2);
		return;
	}
	if (tid == 0) {
		for (int s = 0; s < 2; ++s) {
			mbar_init(bar_full + 8 * s, 1 + 32);
			mbar_init(bar_empty + 8 * s, ST_WORK + 1);
		}
		mbar_init(bar_g, 1);
		mbar_init(bar_r, ST_WORK);
		mbar_init(bar_m, ST_WORK);
		mbar_init(bar_y, 1);
		mbar_init(bar_u, 1);
		mbar_init(bar_end, 1);
		*s_abort = 0;
		fence_mbar_init();
	}
	if (warp == 9) {
		tmem_alloc(smem_u32(s_tmem), 512);
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
	auto wait_one = [&](uint32_t bar, int k) {            // one thread
		if (wait_fast(bar, k & 1, s_abort)) return true;
		fail();
		return false;
	};
	auto wait_warp = [&](uint32_t bar, int k) {           // a whole warp, one answer
		const bool got = wait_fast(bar, k & 1, s_abort);
		if (__all_sync(0xffffffffu, got)) return true;
		fail();
		return false;
	};
	pdl_wait();
	pdl_trigger();
	const int start = __ldcg(p.pos + (size_t)seq * T);

	if (warp == 8) {
		if (lane == 0) {
			int done = 0;
			for (int c = 0; c < n; ++c) {
				const int s = c & 1;
				if (*s_abort || !wait_one(bar_empty + 8 * s, (c >> 1) + 1)) break;
				const uint32_t dst = base + s * pl.stage;
				mbar_arrive_expect_tx(bar_full + 8 * s, pl.stage);
				for (int i = 0; i < pl.nc; ++i) tma_load_2d(dst + i * ST_CHUNK, &tmu, inner + (p.groups + g) * p.state + 64 * i, c * ST_L, bar_full + 8 * s);
				for (int i = 0; i < 2; ++i) tma_load_2d(dst + (pl.nc + i) * ST_CHUNK, &tmu, inner + g * p.state + 64 * i, c * ST_L, bar_full + 8 * s);
				tma_load_2d(dst + (pl.nc + 2) * ST_CHUNK, &tmu, head * p.vdim + p0, c * ST_L, bar_full + 8 * s);
				done = c + 1;
			}
			// no copy may be in flight when the CTA ends
			for (int c = max(0, done - 2); c < done; ++c) mbar_wait_bounded(bar_full + 8 * (c & 1), (c >> 1) & 1, ATTN_SPIN);
		}
		__syncwarp();
	} else if (warp == 10) {
		const float bias = __ldg(p.dt_bias + head), a = __ldg(p.a + head) * 1.4426950408889634f;
		constexpr int PER = ST_L / 32;
		const float *src = p.dt + (size_t)seq * T * p.dt_ld + head;
		for (int c = 0; c < n; ++c) {
			float dt[PER];
			double run = 0.0;
#pragma unroll
			for (int i = 0; i < PER; ++i) {
				const int t = c * ST_L + lane * PER + i;
				dt[i] = t < T ? __ldcg(src + (size_t)t * p.dt_ld) : 0.f;
			}
#pragma unroll
			for (int i = 0; i < PER; ++i) {
				dt[i] = c * ST_L + lane * PER + i < T ? ssm_softplus(dt[i] + bias) : 0.f;      // behind the end: no input, no decay
				run += (double)(a * dt[i]);
			}
			double before = run;
#pragma unroll
			for (int d = 1; d < 32; d <<= 1) {
				const double v = __shfl_up_sync(0xffffffffu, before, d);
				if (lane >= d) before += v;
			}
			before -= run;
			if (!wait_warp(bar_empty + 8 * (c & 1), (c >> 1) + 1)) break;
#pragma unroll
			for (int i = 0; i < PER; ++i) {
				before += (double)(a * dt[i]);
				const int at = (c & 1) * ST_L + lane * PER + i;
				const float hi = (float)before;
				const bf16 lo = __float2bfloat16_rn((float)(before - (double)hi));
				s_hi[at] = hi;
				s_lo[at] = lo;
				s_w[at] = log2f(dt[i]) - __bfloat162float(lo);          // dt = 0: weight 2^-inf = 0
			}
			mbar_arrive(bar_full + 8 * (c & 1));
		}
	} else if (warp == 9) {
		if (lane == 0) {
			const uint32_t fmt = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(ST_L >> 4) << 24);          // D fp32, A/B bf16, M = 128
			const uint32_t wide = (uint32_t)(ST_L >> 3) << 17, at_n = (uint32_t)((np + 15) / 16 * 2) << 17;
			const uint32_t id_g = fmt | wide, id_i = fmt | wide | (1u << 16), id_y = fmt | at_n | (1u << 16), id_u = id_y | (1u << 15);
			const int steps = p.state >> 4;
			const uint64_t d_c = smem_desc_sw128(base), d_bk = smem_desc_sw128(base + pl.nc * ST_CHUNK), d_bm = desc_rows(base + pl.nc * ST_CHUNK),
						   d_x = desc_rows(base + (pl.nc + 2) * ST_CHUNK), d_xs = desc_rows(sxs), d_s = desc_rows(sst);
			const uint32_t stage16 = pl.stage >> 4;
			constexpr uint32_t C16 = ST_CHUNK >> 4;
			auto issue_g = [&](int c) {                   // C and B tiles have arrived
				uint64_t a = d_c + (c & 1) * stage16, b = d_bk + (c & 1) * stage16;
#pragma unroll 1
				for (int k = 0; k < steps; ++k) {
					umma_f16(tmem + T_G, a, b, id_g, k ? 1u : 0u);
					const uint32_t next = (k & 3) == 3 ? C16 - 6 : 2;          // 16 entries further: 32 bytes, or the next tile
					a += next;
					b += next;
				}
				umma_commit(bar_g);
			};
			bool ok = wait_one(bar_full, 0);
			tc_fence_after();
			if (ok) issue_g(0);
			for (int c = 0; c < n && ok; ++c) {
				const uint32_t so = (c & 1) * stage16;
				if (!(ok = wait_one(bar_r, c))) break;
				tc_fence_after();
				const uint64_t bm = d_bm + so, x = d_x + so;
				uint64_t a = d_c + so, b = d_s;
#pragma unroll 1
				for (int k = 0; k < steps; ++k) {
					umma_f16(tmem + T_YI + (c & 1) * 2 * ST_P, a, b, id_i, k ? 1u : 0u);
					a += (k & 3) == 3 ? C16 - 6 : 2;
					b += 128;                                              // 16 rows of 128 bytes
				}
#pragma unroll
				for (int part = 0; part < 2; ++part)
#pragma unroll
					for (int k = 0; k < ST_L / 16; ++k) umma_f16(tmem + T_S, bm + 128 * k, d_xs + part * C16 + 128 * k, id_u, 1u);
				umma_commit(bar_u);
				if (!(ok = wait_one(bar_m, c))) break;
				tc_fence_after();
#pragma unroll
				for (int part = 0; part < 2; ++part)
#pragma unroll
					for (int k = 0; k < ST_L / 16; ++k) umma_f16_ts(tmem + T_YA, tmem + T_G + (k >> 1) * 32 + part * 16 + (k & 1) * 8, x + 128 * k, id_y, part | k ? 1u : 0u);
				umma_commit(bar_y);
				umma_commit(bar_empty + 8 * (c & 1));
				if (c + 1 < n) {
					if (!(ok = wait_one(bar_full + 8 * ((c + 1) & 1), (c + 1) >> 1))) break;
					tc_fence_after();
					issue_g(c + 1);
				}
			}
			umma_commit(bar_end);                         // every MMA has completed before tensor memory goes back
			mbar_wait_bounded(bar_end, 0, ATTN_SPIN);
		}
		__syncwarp();
	} else {
		const int q = warp & 3, h = warp >> 2, row = q * 32 + lane;          // token of the chunk, or state entry
		const uint32_t lanes = (uint32_t)(q * 32) << 16;
		const bool cols = 32 * h < np;                                       // this half of the value entries exists
		const float d = __ldg(p.d + head);
		// ---- state of the sequence into tensor memory: row = state entry, column = value entry ----
		float *state = p.s + ((size_t)seq * p.heads + head) * p.vdim * p.state + (size_t)p0 * p.state;
		if (cols) {
			uint32_t v[32];
#pragma unroll
			for (int i = 0; i < 32; ++i) v[i] = start > 0 && row < p.state && 32 * h + i < np ? __float_as_uint(__ldcg(state + (size_t)(32 * h + i) * p.state + row)) : 0u;
			tmem_st32(tmem + T_S + lanes + 32 * h, v);
			tmem_st_wait();
		}
		// a warp's part of z and y: 32 tokens x 64 bytes; four lanes per row where they meet global memory (rows lie far apart there)
		const int cr = q * 32 + (lane >> 2), cu = lane & 3;
		const bool ccol = 32 * h + 8 * cu < np;
		const bf16 *zg = reinterpret_cast<const bf16 *>(p.raw) + (size_t)seq * T * p.raw_ld + p.z_at + head * p.vdim + p0 + 32 * h + 8 * cu;
		bf16 *og = reinterpret_cast<bf16 *>(p.out) + (size_t)seq * T * p.out_ld + head * p.vdim + p0 + 32 * h + 8 * cu;
		auto input_tile = [&](int c) { return st_smem + (size_t)(c & 1) * pl.stage + (size_t)(pl.nc + 2) * ST_CHUNK; };
		// operands of chunk c that follow from the state and the inputs (both operands of chunk c - 1 have been read)
		auto prepare = [&](int c) {
			const unsigned char *xt = input_tile(c);
			const float *hi_j = s_hi + (c & 1) * ST_L, *w = s_w + (c & 1) * ST_L;
			const float end = hi_j[ST_L - 1], end_lo = __bfloat162float(s_lo[(c & 1) * ST_L + ST_L - 1]);
			// inputs times step size and decay to the chunk's end: element by element, so the tile's layout does not matter
			const int trow = tid >> 1;                                  // two threads per token, half a row each
			const float fx = ex2((end - hi_j[trow]) + (end_lo + w[trow]));
#pragma unroll
			for (int i = 0; i < 4; ++i) {
				const uint32_t off = (uint32_t)trow * 128 + (uint32_t)(((tid & 1) * 4 + i + trow) & 7) * 16;      // (rotated against bank conflicts)
				const uint4 x = *reinterpret_cast<const uint4 *>(xt + off);
				const uint32_t xs[4] = {x.x, x.y, x.z, x.w};
				uint32_t hi[4], lo[4];
#pragma unroll
				for (int j = 0; j < 4; ++j) st_split(__uint_as_float(xs[j] << 16) * fx, __uint_as_float(xs[j] & 0xFFFF0000u) * fx, hi[j], lo[j]);
				unsigned char *dst = st_smem + 2 * (size_t)pl.stage + off;
				*reinterpret_cast<uint4 *>(dst) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
				*reinterpret_cast<uint4 *>(dst + ST_CHUNK) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
			}
			// S in two parts for Yi, then decayed
			if (cols) {
				float v[32];
				tmem_ld32(tmem + T_S + lanes + 32 * h, v);
				tmem_ld_wait();
				tmem_settle(v);
				unsigned char *dst = st_smem + 2 * (size_t)pl.stage + 2 * ST_CHUNK + row * 128;
#pragma unroll
				for (int i = 0; i < 4; ++i) {
					uint32_t hi[4], lo[4];
#pragma unroll
					for (int j = 0; j < 4; ++j) st_split(v[8 * i + 2 * j], v[8 * i + 2 * j + 1], hi[j], lo[j]);
					const int unit = ((4 * h + i) ^ (row & 7)) * 16;
					*reinterpret_cast<uint4 *>(dst + unit) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
					*reinterpret_cast<uint4 *>(dst + ST_CHUNK + unit) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
				}
				const float f = ex2(end + end_lo);
				uint32_t o[32];
#pragma unroll
				for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(v[i] * f);
				tmem_st32(tmem + T_S + lanes + 32 * h, o);
				tmem_st_wait();
			}
			fence_proxy_async();
			tc_fence_before();
			mbar_arrive(bar_r);
		};
		bool ok = wait_warp(bar_full, 0);
		if (ok) prepare(0);
		for (int c = 0; c < n && ok; ++c) {
			const int s = c & 1, t0 = c * ST_L;
			const float *hi_j = s_hi + s * ST_L, *w = s_w + s * ST_L;
			uint4 z[4];                                                      // gates, requested early
#pragma unroll
			for (int i = 0; i < 4; ++i)
				z[i] = ccol && t0 + cr + 8 * i < T ? __ldcg(reinterpret_cast<const uint4 *>(zg + (size_t)(t0 + cr + 8 * i) * p.raw_ld)) : make_uint4(0u, 0u, 0u, 0u);
			// ---- M over G: this thread's row, half of the columns ----
			if (!(ok = wait_warp(bar_g, c))) break;
			tc_fence_after();
			const float si = hi_j[row], si_lo = __bfloat162float(s_lo[s * ST_L + row]);
			// left of the diagonal's 32 x 32 blocks the factor splits at the block's first row r: 2^(s_i - s_r) * 2^(s_r - s_j) dt_j, both at
			// most of the order of one; a lane computes the second one for one column
			const float rh = hi_j[q * 32], rl = __bfloat162float(s_lo[s * ST_L + q * 32]), from_r = ex2((si - rh) + (si_lo - rl));
#pragma unroll 1
			for (int b = 0; b < 2; ++b) {
				const int j0 = 64 * h + 32 * b;
				const uint32_t at = tmem + T_G + lanes + j0;
				uint32_t out[32];
				if (j0 > q * 32) {                                          // above the diagonal
#pragma unroll
					for (int i = 0; i < 32; ++i) out[i] = 0u;
				} else {
					float v[32];
					tmem_ld32(at, v);
					const float wl = w[j0 + lane], hl = hi_j[j0 + lane];
					if (j0 < q * 32) {
						const float to_r = ex2((rh - hl) + (rl + wl));
						tmem_ld_wait();
						tmem_settle(v);
#pragma unroll
						for (int i = 0; i < 32; ++i) v[i] *= from_r * __shfl_sync(0xffffffffu, to_r, i);
					} else {
						tmem_ld_wait();
						tmem_settle(v);
#pragma unroll
						for (int i = 0; i < 32; ++i) {
							const float f = ex2((si - __shfl_sync(0xffffffffu, hl, i)) + (si_lo + __shfl_sync(0xffffffffu, wl, i)));
							v[i] = i <= lane ? v[i] * f : 0.f;
						}
					}
#pragma unroll
					for (int i = 0; i < 16; ++i) st_split(v[2 * i], v[2 * i + 1], out[i], out[16 + i]);
				}
				tmem_st32(at, out);
			}
			tmem_st_wait();
			tc_fence_before();
			mbar_arrive(bar_m);
			// ---- what does not depend on the products: gates, inputs of this row ----
			unsigned char *xt = input_tile(c), *own = xt + row * 128;
			auto unit = [&](int r, int u) { return ((4 * h + u) ^ (r & 7)) * 16; };
#pragma unroll
			for (int i = 0; i < 4; ++i) asm volatile("" : "+r"(z[i].x), "+r"(z[i].y), "+r"(z[i].z), "+r"(z[i].w));      // not to be waited for any earlier
			uint4 x[4];
			float gate[32];
			if (cols) {
#pragma unroll
				for (int u = 0; u < 4; ++u) {
					x[u] = *reinterpret_cast<const uint4 *>(own + unit(row, u));
					const uint32_t zs[4] = {z[u].x, z[u].y, z[u].z, z[u].w};
#pragma unroll
					for (int j = 0; j < 4; ++j) {
						gate[8 * u + 2 * j] = silu_fast(__uint_as_float(zs[j] << 16));
						gate[8 * u + 2 * j + 1] = silu_fast(__uint_as_float(zs[j] & 0xFFFF0000u));
					}
				}
			}
			if (c + 1 < n) {
				if (!(ok = wait_warp(bar_full + 8 * (s ^ 1), (c + 1) >> 1)) || !(ok = wait_warp(bar_u, c))) break;
				tc_fence_after();
				prepare(c + 1);
			}
			// ---- y ----
			if (!(ok = wait_warp(bar_y, c))) break;
			tc_fence_after();
			if (cols) {
				const float e = ex2(si + si_lo);
				const uint32_t yi = tmem + T_YI + s * 2 * ST_P + lanes + 32 * h, ya = tmem + T_YA + lanes + 32 * h;
#pragma unroll
				for (int b = 0; b < 2; ++b) {
					float y0[16], y1[16], y2[16];
					tmem_ld16(yi + 16 * b, y0);
					tmem_ld16(yi + ST_P + 16 * b, y1);
					tmem_ld16(ya + 16 * b, y2);
					tmem_ld_wait();
					tmem_settle(y0);
					tmem_settle(y1);
					tmem_settle(y2);
#pragma unroll
					for (int u = 0; u < 2; ++u) {
						const uint4 xv = x[2 * b + u];
						const uint32_t xs[4] = {xv.x, xv.y, xv.z, xv.w};
						uint32_t o[4];
#pragma unroll
						for (int j = 0; j < 4; ++j) {
							const int i = 8 * u + 2 * j;
							const float a0 = fmaf(d, __uint_as_float(xs[j] << 16), fmaf(e, y0[i] + y1[i], y2[i]));
							const float a1 = fmaf(d, __uint_as_float(xs[j] & 0xFFFF0000u), fmaf(e, y0[i + 1] + y1[i + 1], y2[i + 1]));
							o[j] = pack_bf16(a0, a1);
						}
						*reinterpret_cast<uint4 *>(own + unit(row, 2 * b + u)) = make_uint4(o[0], o[1], o[2], o[3]);
					}
				}
				__syncwarp();
#pragma unroll
				for (int i = 0; i < 4; ++i) {
					const uint4 yv = *reinterpret_cast<const uint4 *>(xt + (cr + 8 * i) * 128 + unit(cr + 8 * i, cu));
					const uint32_t ys[4] = {yv.x, yv.y, yv.z, yv.w};
					uint32_t o[4];
#pragma unroll
					for (int j = 0; j < 4; ++j) o[j] = pack_bf16(__uint_as_float(ys[j] << 16) * gate[8 * i + 2 * j], __uint_as_float(ys[j] & 0xFFFF0000u) * gate[8 * i + 2 * j + 1]);
					if (ccol && t0 + cr + 8 * i < T) *reinterpret_cast<uint4 *>(og + (size_t)(t0 + cr + 8 * i) * p.out_ld) = make_uint4(o[0], o[1], o[2], o[3]);
				}
				fence_proxy_async();                          // the tile is written by a copy next
			}
			tc_fence_before();
			mbar_arrive(bar_empty + 8 * s);
		}
		if (ok && cols && wait_warp(bar_u, n - 1)) {
			tc_fence_after();
			float v[32];
			tmem_ld32(tmem + T_S + lanes + 32 * h, v);
			tmem_ld_wait();
			tmem_settle(v);
#pragma unroll
			for (int i = 0; i < 32; ++i)
				if (row < p.state && 32 * h + i < np) state[(size_t)(32 * h + i) * p.state + row] = v[i];
		}
		// ---- the convolution's last inputs ----
		const int last = min(T, p.taps);
		const bool shared = p0 == 0 && head % (p.heads / p.groups) == 0;
		const int count = np + (shared ? 2 * p.state : 0);
		const bf16 *in = reinterpret_cast<const bf16 *>(p.raw) + (size_t)seq * T * p.raw_ld + p.conv_at;
		float *ring = p.ring + (size_t)seq * p.taps * p.conv_ld;
		for (int i = tid; i < last * count; i += ST_WORK) {
			const int tt = T - last + i / count, e = i % count;
			const int ch = e < np ? head * p.vdim + p0 + e : e < np + p.state ? inner + g * p.state + e - np : inner + (p.groups + g) * p.state + e - np - p.state;
			ring[(size_t)((start + tt) % p.taps) * p.conv_ld + ch] = Elem<bf16>::ldcg(in + (size_t)tt * p.raw_ld + ch);
		}
	}
	tc_fence_before();
	__syncthreads();
	if (warp == 9) tmem_dealloc(tmem, 512);
}

}   // namespace

bool ssm_tc_ok(const SsmArgs &p) { return p.vdim % 16 == 0 && p.state % 16 == 0 && p.state <= 128 && p.out_ld % 8 == 0; }

int ssm_tc_launch(const SsmArgs &p, cudaStream_t stream) {
	const int T = p.rows_per_seq, seqs = p.M / T, slices = (p.vdim + ST_P - 1) / ST_P;
	for (int b = 0; b < seqs; ++b) {
		alignas(64) CUtensorMap tmu;
		const bf16 *u = reinterpret_cast<const bf16 *>(p.u) + (size_t)b * T * p.conv_ld;
		if (int rc = dense_tensor_map(u, T, p.conv_ld, p.conv_ld, ST_L, 64, &tmu)) return rc;
		if (int rc = dn_launch(ssm_tc_kernel, dim3(p.heads * slices), dim3(ST_THREADS), st_plan(p.state).smem, stream, tmu, p, b)) return rc;
	}
	return GPTQ_OK;
}

}   // namespace gptq
