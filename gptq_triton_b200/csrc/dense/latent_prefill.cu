// Latent attention of a prompt portion on the 5th-generation tensor cores, expanded form: the caller has multiplied the cached
// latents with W_uk and W_uv (keys [S, heads * dim], values transposed [heads * vdim, S]); the rotated key part that all heads
// share comes straight from the cache rows.
//
// A CTA serves one head and NQ tiles of 128 query rows against key tiles of 128:
//   softmax warps     eight per query tile, a thread owns half a query row (64 keys): scores from tensor memory, causal mask
//                     where the tile crosses the diagonal, online softmax in fp32 base 2 (the halves exchange their maxima),
//                     weights back to tensor memory; at the end the division by the sum, the head's gate and the bf16 store
//   TMA warp          Q once, then key and value tiles through rings of stages (128-byte swizzle)
//   MMA warps         one per query tile: S = Q K^T (operands in shared memory), O += P V (P in tensor memory, V^T in shared
//                     memory).  A wait costs the issuing thread as much as several MMAs even when it is over already, so one
//                     thread for both tiles would leave the tensor core idle more than half the time
// The weights are kept at more than bf16 precision: P is split into a bf16 high part and a bf16 remainder, which together take
// exactly the columns of the fp32 scores they replace (32 keys at a time: 16 columns of high parts, 16 of remainders, so that
// every thread overwrites only scores that it has read); both parts multiply the same V tile.  The running output stays in
// tensor memory; it is rescaled only when a row's maximum has grown by more than 2^8 since the last rescale (the weights are
// then at most 2^8 and the result is the same, the reference point of a softmax cancels).
// With NQ = 2 the MMAs of one query tile run under the softmax of the other.  Every wait is bounded.
#include <algorithm>

#include "latent.cuh"
#include "prefill_common.cuh"

namespace gptq {

namespace {

constexpr int LP_T = 128;                               // query rows and keys per tile
constexpr int LP_CHUNK = LP_T * 128;                    // bytes of a 128 x 64 bf16 operand chunk
constexpr int LP_TILE_THREADS = 2 * LP_T;               // softmax threads per query tile
constexpr size_t LP_SMEM = 227 * 1024 - 4 * 2 * LP_T * sizeof(float);      // what a CTA may have, less the exchanged maxima

struct LpPlan {
	int nd, nr, sk, sv;                                   // chunks of the unrotated / rotated part, stages of K and V
	size_t smem;
};

template <int NQ>
__global__ void __launch_bounds__(NQ * (LP_TILE_THREADS + 32) + 32, 1) latent_prefill_kernel(const __grid_constant__ CUtensorMap tmq, const __grid_constant__ CUtensorMap tmk,
																		 const __grid_constant__ CUtensorMap tmr, const __grid_constant__ CUtensorMap tmv,
																		 const LatentPrefill p, const LpPlan pl, uint32_t tmem_cols) {
	extern __shared__ unsigned char lp_raw[];
	__shared__ float s_mx[2][NQ][2][LP_T];          // [parity of the key tile][query tile][half][row]
	unsigned char *smem = lp_raw + ((1024u - (smem_u32(lp_raw) & 1023u)) & 1023u);
	const int nch = pl.nd + pl.nr;
	const uint32_t k_bytes = nch * LP_CHUNK, v_bytes = 2u * p.vdim * 128u;
	const uint32_t sq = smem_u32(smem), sk = sq + NQ * k_bytes, sv = sk + pl.sk * k_bytes;
	uint64_t *bars = reinterpret_cast<uint64_t *>(smem + (size_t)(NQ + pl.sk) * k_bytes + (size_t)pl.sv * v_bytes);
	const uint32_t b0 = smem_u32(bars);
	const uint32_t bar_q = b0, bar_fk = b0 + 16, bar_ek = b0 + 32, bar_fv = b0 + 48, bar_ev = b0 + 64;      // two slots each for K, V
	const uint32_t bar_s = b0 + 80, bar_p = b0 + 96, bar_o = b0 + 112, bar_drain = b0 + 128;                                                          // one per query tile
	uint32_t *s_tmem = reinterpret_cast<uint32_t *>(bars + 18);
	volatile int *s_abort = reinterpret_cast<volatile int *>(s_tmem + 1);
	const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
	const int nqb = (p.t + NQ * LP_T - 1) / (NQ * LP_T);
	const int head = blockIdx.x % p.heads, q0 = (nqb - 1 - (int)blockIdx.x / p.heads) * NQ * LP_T;          // the longest rows first
	const int hd = p.dim + p.rot_dim;
	auto tiles_of = [&](int i) {
		const int first = q0 + i * LP_T;
		return first >= p.t ? 0 : (p.start + min(first + LP_T, p.t) - 1) / LP_T + 1;
	};
	int ntile[2] = {tiles_of(0), NQ > 1 ? tiles_of(1) : 0};
	const int nmax = max(ntile[0], ntile[1]);

	if (tid == 0) {
		mbar_init(bar_q, 1);
		for (int s = 0; s < 2; ++s) {
			mbar_init(bar_fk + 8 * s, 1);
			mbar_init(bar_ek + 8 * s, NQ);          // every query tile releases a stage
			mbar_init(bar_fv + 8 * s, 1);
			mbar_init(bar_ev + 8 * s, NQ);
			mbar_init(bar_s + 8 * s, 1);
			mbar_init(bar_p + 8 * s, LP_TILE_THREADS);
			mbar_init(bar_o + 8 * s, 1);
			mbar_init(bar_drain + 8 * s, 1);
		}
		*s_abort = 0;
		fence_mbar_init();
	}
	constexpr int W_TMA = NQ * 8, W_MMA = NQ * 8 + 1;
	if (warp == W_MMA) {
		tmem_alloc(smem_u32(s_tmem), tmem_cols);
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

	if (warp == W_TMA) {
		if (lane == 0) {
			mbar_arrive_expect_tx(bar_q, NQ * k_bytes);
			for (int i = 0; i < NQ; ++i)
				for (int c = 0; c < nch; ++c)
					tma_load_2d(sq + i * k_bytes + c * LP_CHUNK, &tmq, head * hd + (c < pl.nd ? 64 * c : p.dim + 64 * (c - pl.nd)), q0 + i * LP_T, bar_q);
			int jk = 0, jv = 0;
			for (int j = 0; j < nmax; ++j) {
				const int a = j % pl.sk, b = j % pl.sv;
				if (*s_abort || !mbar_wait_bounded(bar_ek + 8 * a, ((j / pl.sk) & 1) ^ 1, ATTN_SPIN)) { fail(); break; }
				mbar_arrive_expect_tx(bar_fk + 8 * a, k_bytes);
				for (int c = 0; c < nch; ++c) {
					const uint32_t dst = sk + a * k_bytes + c * LP_CHUNK;
					if (c < pl.nd) tma_load_2d(dst, &tmk, head * p.dim + 64 * c, j * LP_T, bar_fk + 8 * a);
					else tma_load_2d(dst, &tmr, p.kv_rank + 64 * (c - pl.nd), j * LP_T, bar_fk + 8 * a);
				}
				jk = j + 1;
				if (*s_abort || !mbar_wait_bounded(bar_ev + 8 * b, ((j / pl.sv) & 1) ^ 1, ATTN_SPIN)) { fail(); break; }
				mbar_arrive_expect_tx(bar_fv + 8 * b, v_bytes);
				for (int c = 0; c < 2; ++c) tma_load_2d(sv + b * v_bytes + c * (v_bytes / 2), &tmv, j * LP_T + 64 * c, head * p.vdim, bar_fv + 8 * b);
				jv = j + 1;
			}
			// no copy may be in flight when the CTA ends
			mbar_wait_bounded(bar_q, 0, ATTN_SPIN);
			for (int j = max(0, jk - pl.sk); j < jk; ++j) mbar_wait_bounded(bar_fk + 8 * (j % pl.sk), (j / pl.sk) & 1, ATTN_SPIN);
			for (int j = max(0, jv - pl.sv); j < jv; ++j) mbar_wait_bounded(bar_fv + 8 * (j % pl.sv), (j / pl.sv) & 1, ATTN_SPIN);
		}
		__syncwarp();
	} else if (warp >= W_MMA) {
		if (lane == 0) {
			const int i = warp - W_MMA, n = ntile[i];
			const uint32_t base = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(LP_T >> 4) << 24);       // D fp32, A/B bf16 K-major, M = 128
			const uint32_t id_qk = base | ((uint32_t)(LP_T >> 3) << 17), id_pv = base | ((uint32_t)(p.vdim >> 3) << 17);
			auto wait = [&](uint32_t bar, int k) {
				if (!wait_fast(bar, k & 1, s_abort)) { fail(); return false; }
				tc_fence_after();
				return true;
			};
			auto wait_k = [&](int j) { return wait(bar_fk + 8 * (j % pl.sk), j / pl.sk); };
			auto wait_v = [&](int j) { return wait(bar_fv + 8 * (j % pl.sv), j / pl.sv); };
			auto qk = [&](int j) {
				if (!wait_k(j)) return false;
				uint32_t acc = 0;
				// a descriptor advances by 2 (32 bytes) per K step; one thread issues everything, so the loop must stay short
				uint64_t qd = smem_desc_sw128(sq + i * k_bytes), kd = smem_desc_sw128(sk + (j % pl.sk) * k_bytes);
				for (int c = 0; c < nch; ++c, qd += LP_CHUNK / 16, kd += LP_CHUNK / 16) {
					const int steps = (c < pl.nd ? p.dim - 64 * c : p.rot_dim - 64 * (c - pl.nd)) >> 4;
#pragma unroll
					for (int k = 0; k < 4; ++k)
						if (k < steps) {
							umma_f16(tmem + i * LP_T, qd + 2 * k, kd + 2 * k, id_qk, acc);
							acc = 1;
						}
				}
				umma_commit(bar_s + 8 * i);
				return true;
			};
			auto pv = [&](int j) {
				if (!wait_v(j) || !wait(bar_p + 8 * i, j)) return false;
				const uint32_t d = tmem + NQ * LP_T + i * p.vdim, pa = tmem + i * LP_T;
				const uint64_t vd = smem_desc_sw128(sv + (j % pl.sv) * v_bytes), vd1 = vd + (v_bytes >> 5);
				uint32_t acc = j ? 1u : 0u;
#pragma unroll
				for (int part = 0; part < 2; ++part)
#pragma unroll
					for (int k = 0; k < 8; ++k) {
						umma_f16_ts(d, pa + (k >> 1) * 32 + part * 16 + (k & 1) * 8, (k < 4 ? vd : vd1) + 2 * (k & 3), id_pv, acc);
						acc = 1;
					}
				umma_commit(bar_o + 8 * i);
				return true;
			};
			// A query tile whose keys have ended goes on releasing the stages that the other one uses, each only once it has been
			// filled: an arrival that came earlier would count for the phase before.
			bool ok = wait(bar_q, 0) && (n ? qk(0) : wait_k(0));
			umma_commit(bar_ek);
			for (int j = 0; j < nmax && ok; ++j) {
				ok = j < n ? pv(j) : wait_v(j);
				umma_commit(bar_ev + 8 * (j % pl.sv));
				if (ok && j + 1 < nmax) {
					ok = j + 1 < n ? qk(j + 1) : wait_k(j + 1);
					umma_commit(bar_ek + 8 * ((j + 1) % pl.sk));
				}
			}
			umma_commit(bar_drain + 8 * i);          // every MMA has completed before tensor memory goes back
			mbar_wait_bounded(bar_drain + 8 * i, 0, ATTN_SPIN);
		}
		__syncwarp();
	} else {
		const int i = warp >> 3, half = (warp >> 2) & 1, n = ntile[i];
		const int rl = (warp & 3) * 32 + lane, row = q0 + i * LP_T + rl, pos = p.start + row;
		const uint32_t lane_base = (uint32_t)((warp & 3) * 32) << 16;
		const uint32_t ts = tmem + i * LP_T + half * 64 + lane_base, to = tmem + NQ * LP_T + i * p.vdim + lane_base;
		const float sc = p.scale * 1.4426950408889634f;
		float ref = 0.f, sum = 0.f;
		bool ok = true;
		auto wait = [&](uint32_t bar, int k) {
			const bool got = wait_fast(bar, k & 1, s_abort);
			if (!__all_sync(0xffffffffu, got)) { fail(); return false; }
			tc_fence_after();
			return true;
		};
		auto pair_barrier = [&]() { asm volatile("bar.sync %0, %1;" ::"r"(1 + i), "n"(LP_TILE_THREADS) : "memory"); };
		for (int j = 0; j < n; ++j) {
			// (a wait that ran out does not leave the loop: both halves must keep meeting at the barrier)
			ok = ok && wait(bar_s + 8 * i, j);
			const int last = pos - j * LP_T - half * 64;                                     // last visible key of this half
			const bool edge = j * LP_T + half * 64 + 63 > p.start + q0 + i * LP_T + (warp & 3) * 32;      // this warp's first row does not see all of them
			float mx = -INFINITY;
			if (ok) {
				float s[2][32];
				tmem_ld32(ts, s[0]);
				tmem_ld32(ts + 32, s[1]);
				tmem_ld_wait();
				tmem_settle(s[0]);
				tmem_settle(s[1]);
				if (edge) {
#pragma unroll
					for (int k = 0; k < 64; ++k)
						if (k > last) s[k >> 5][k & 31] = -INFINITY;
				}
				float m0 = s[0][0], m1 = s[0][1], m2 = s[1][0], m3 = s[1][1];
#pragma unroll
				for (int k = 2; k < 32; k += 2) {
					m0 = fmaxf(m0, s[0][k]);
					m1 = fmaxf(m1, s[0][k + 1]);
					m2 = fmaxf(m2, s[1][k]);
					m3 = fmaxf(m3, s[1][k + 1]);
				}
				mx = fmaxf(fmaxf(m0, m1), fmaxf(m2, m3));
			}
			s_mx[j & 1][i][half][rl] = mx;
			pair_barrier();
			mx = fmaxf(mx, s_mx[j & 1][i][half ^ 1][rl]);
			// scaled maximum; a row below the diagonal of this tile sees none of its keys and keeps its reference point
			const float rm = mx == -INFINITY ? (j ? ref : 0.f) : mx * sc;
			if (j == 0) {
				ref = rm;
			} else if (__any_sync(0xffffffffu, rm > ref + 8.f)) {          // the same rows, so the same decision in both halves
				ok = ok && wait(bar_o + 8 * i, j - 1);
				const float nref = fmaxf(ref, rm), corr = ex2(ref - nref);
				ref = nref;
				sum *= corr;
				if (ok) {
#pragma unroll 1
					for (int c = half * 16; c < p.vdim; c += 32) {
						float o[16];
						tmem_ld16(to + c, o);
						tmem_ld_wait();
						tmem_settle(o);
#pragma unroll
						for (int k = 0; k < 16; ++k) o[k] *= corr;
						tmem_st16(to + c, o);
					}
					tmem_st_wait();
				}
			}
			if (ok) {
				float t0 = 0.f, t1 = 0.f;
#pragma unroll 1
				for (int c = 0; c < 2; ++c) {
					float s[32];
					uint32_t out[32];                // 16 columns of high parts, 16 of remainders
					tmem_ld32(ts + c * 32, s);
					tmem_ld_wait();
					tmem_settle(s);
					if (edge) {
#pragma unroll
						for (int k = 0; k < 32; ++k)
							if (c * 32 + k > last) s[k] = -INFINITY;
					}
#pragma unroll
					for (int k = 0; k < 16; ++k) {
						const float a = ex2(fmaf(s[2 * k], sc, -ref)), b = ex2(fmaf(s[2 * k + 1], sc, -ref));
						t0 += a;
						t1 += b;
						const uint32_t hi = pack_bf16(a, b);
						out[k] = hi;
						out[16 + k] = pack_bf16(a - __uint_as_float(hi << 16), b - __uint_as_float(hi & 0xFFFF0000u));
					}
					tmem_st32(ts + c * 32, out);
				}
				sum += t0 + t1;
				tmem_st_wait();
			}
			tc_fence_before();
			mbar_arrive(bar_p + 8 * i);
		}
		if (n) {
			s_mx[n & 1][i][half][rl] = sum;
			pair_barrier();
			sum += s_mx[n & 1][i][half ^ 1][rl];
			if (ok && wait(bar_o + 8 * i, n - 1)) {
				const float f = row < p.t ? (p.gate ? __ldcg(p.gate + (size_t)row * p.gate_ld + head) : 1.f) / sum : 0.f;
				bf16 *dst = reinterpret_cast<bf16 *>(p.out) + (size_t)row * p.out_ld + head * p.vdim;
#pragma unroll 1
				for (int c = half * 16; c < p.vdim; c += 32) {
					float o[16];
					tmem_ld16(to + c, o);
					tmem_ld_wait();
					tmem_settle(o);
					if (row < p.t) {
#pragma unroll
						for (int k = 0; k < 2; ++k)
							*reinterpret_cast<uint4 *>(dst + c + 8 * k) = make_uint4(pack_bf16(o[8 * k] * f, o[8 * k + 1] * f), pack_bf16(o[8 * k + 2] * f, o[8 * k + 3] * f),
																					 pack_bf16(o[8 * k + 4] * f, o[8 * k + 5] * f), pack_bf16(o[8 * k + 6] * f, o[8 * k + 7] * f));
					}
				}
			}
		}
	}
	tc_fence_before();
	__syncthreads();
	if (warp == W_MMA) tmem_dealloc(tmem, tmem_cols);
}

// stages for nq query tiles per CTA; false: does not fit
bool lp_plan(int nq, int dim, int rot_dim, int vdim, LpPlan *out) {
	LpPlan pl;
	pl.nd = (dim + 63) / 64;
	pl.nr = (rot_dim + 63) / 64;
	if (vdim > 256 || nq * (LP_T + vdim) > 512) return false;
	const size_t k = (size_t)(pl.nd + pl.nr) * LP_CHUNK, v = (size_t)vdim * 256;
	const int opts[4][2] = {{2, 2}, {1, 2}, {2, 1}, {1, 1}};      // V is needed sooner after its release than K
	for (auto &o : opts) {
		pl.sk = o[0];
		pl.sv = o[1];
		pl.smem = (nq + pl.sk) * k + pl.sv * v + 1024 + 256;
		if (pl.smem <= LP_SMEM) {
			*out = pl;
			return true;
		}
	}
	return false;
}

}   // namespace

bool latent_prefill_ok(int dim, int rot_dim, int vdim) {
	LpPlan pl;
	return lp_plan(1, dim, rot_dim, vdim, &pl);
}

int latent_prefill_launch(const LatentPrefill &p, cudaStream_t stream) {
	LpPlan pl;
	const bool two = p.t > LP_T && lp_plan(2, p.dim, p.rot_dim, p.vdim, &pl);
	if (!two && !lp_plan(1, p.dim, p.rot_dim, p.vdim, &pl)) return GPTQ_ERR_UNSUPPORTED;
	const int nq = two ? 2 : 1, hd = p.dim + p.rot_dim, R = p.kv_rank + p.rot_dim;
	alignas(64) CUtensorMap tmq, tmk, tmr, tmv;
	if (int rc = dense_tensor_map(p.q, p.t, (long long)p.heads * hd, (long long)p.heads * hd, LP_T, 64, &tmq)) return rc;
	if (int rc = dense_tensor_map(p.k, p.S, (long long)p.heads * p.dim, (long long)p.heads * p.dim, LP_T, 64, &tmk)) return rc;
	if (int rc = dense_tensor_map(p.cache, p.S, R, R, LP_T, 64, &tmr)) return rc;
	if (int rc = dense_tensor_map(p.vt, (long long)p.heads * p.vdim, p.S, p.ldv, p.vdim, 64, &tmv)) return rc;
	uint32_t cols = 32;
	while (cols < (uint32_t)(nq * (LP_T + p.vdim))) cols *= 2;
	const dim3 grid(p.heads * ((p.t + nq * LP_T - 1) / (nq * LP_T)));
	if (two) return dn_launch(latent_prefill_kernel<2>, grid, dim3(2 * (LP_TILE_THREADS + 32) + 32), pl.smem, stream, tmq, tmk, tmr, tmv, p, pl, cols);
	return dn_launch(latent_prefill_kernel<1>, grid, dim3(LP_TILE_THREADS + 64), pl.smem, stream, tmq, tmk, tmr, tmv, p, pl, cols);
}

}   // namespace gptq
