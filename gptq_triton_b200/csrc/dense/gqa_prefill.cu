// Grouped-query attention of a prompt portion on the 5th-generation tensor cores: queries normed and scaled beforehand, keys and
// values straight from the cache.
//
// A CTA serves one query head and 128 query rows against key tiles of 128.  With two maps it runs both of the head (MAPS = 2:
// their queries and keys differ, the value tile is loaded once) and combines them at the end; MAPS = 1 serves one map and leaves
// its normalised output to the merge kernel (a single map per head, or two whose values are too wide for tensor memory).
//   softmax warps     eight per map, a thread owns half a query row (64 keys): scores from tensor memory, soft cap, causal mask
//                     where the tile crosses the diagonal, online softmax in fp32 base 2 (the halves exchange their maxima),
//                     weights back to tensor memory
//   TMA warp          queries once, then key and value tiles through rings of stages (128-byte swizzle)
//   MMA warps         one per map: S = Q K^T (operands in shared memory), O += P V (P in tensor memory; V as it is cached, rows of
//                     keys, is an operand whose other dimension is contiguous, so it needs no transposed copy)
// The weights are split into a bf16 high part and a bf16 remainder, which together take the columns of the fp32 scores they
// replace; O is rescaled only when a row's maximum has grown by more than 2^8 (see latent_prefill.cu).
// Capped scores lie in [-cap, cap]: as long as 2^(cap * log2 e) and its inverse are far from the ends of the fp32 range (and of the
// bf16 range, which is the same), zero serves as the reference point of every softmax and there is no running maximum.  A larger
// cap, or none, takes the maximum (before the cap, which keeps the order) as above.
// tanh costs two special-function operations when it is built from an exponential and a reciprocal, which would make it three per
// score with the softmax's own; arguments of at most 1 take a polynomial on the FMA units instead, two scores per instruction.
// That arguments are small follows from the norm weights (`bound`), else a warp looks at its own.  Every wait is bounded.
#include <algorithm>

#include "gqa.cuh"
#include "prefill_common.cuh"

namespace gptq {

namespace {

constexpr int GP_T = 128;                               // query rows and keys per tile
constexpr int GP_CHUNK = GP_T * 128;                    // bytes of a 128 x 64 bf16 operand chunk
constexpr int GP_MAP_THREADS = 2 * GP_T;                // softmax threads per map
constexpr size_t GP_STATIC = (2 * 2 * 2 + 2 + 4) * GP_T * sizeof(float);
constexpr size_t GP_SMEM = 227 * 1024 - GP_STATIC;

struct GpPlan {
	int nd, nv, sk, sv;                                   // chunks of a query / key and of a value row, stages of K and V
	size_t smem;
};

// tanh(x) / x as a polynomial in x^2, |x| <= 1: interpolation of degree 5 in the Chebyshev points of [0, 1]; relative error 8e-7
__device__ __forceinline__ float tanh_small(float x) {
	const float u = x * x;
	float r = fmaf(u, -3.058229038e-03f, 1.672085518e-02f);
	r = fmaf(r, u, -5.158598840e-02f);
	r = fmaf(r, u, 1.328072065e-01f);
	r = fmaf(r, u, -3.332895137e-01f);
	r = fmaf(r, u, 9.999993948e-01f);
	return r * x;
}
// 1 - 2 / (1 + exp(2 x)); absolute error of a few 1e-7
__device__ __forceinline__ float tanh_any(float x) {
	float r;
	asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.f + ex2(2.f * GQ_LOG2E * x)));
	return fmaf(-2.f, r, 1.f);
}

// two fp32 operations per instruction
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pack2(float a, float b) {
	f32x2 r;
	asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
	return r;
}
__device__ __forceinline__ void unpack2(f32x2 v, float &a, float &b) { asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v)); }
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
	f32x2 r;
	asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
	return r;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
	f32x2 r;
	asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
	return r;
}
__device__ __forceinline__ f32x2 add2(f32x2 a, f32x2 b) {
	f32x2 r;
	asm("add.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
	return r;
}

enum { SCORE_PLAIN, SCORE_SMALL, SCORE_ANY };             // no cap, cap with small arguments, cap
template <int KIND>
__device__ __forceinline__ float gp_score(float v, float cap2) {
	return KIND == SCORE_PLAIN ? v : cap2 * (KIND == SCORE_SMALL ? tanh_small(v) : tanh_any(v));
}

// 32 scores of a row -> 16 columns of high parts, 16 of remainders; returns the sum of the weights
template <int KIND>
__device__ __forceinline__ float gp_weights(const float (&s)[32], uint32_t (&out)[32], float cap2, float ref, bool edge, int last) {
	float t0 = 0.f, t1 = 0.f;
#pragma unroll
	for (int k = 0; k < 16; ++k) {
		float a = ex2(gp_score<KIND>(s[2 * k], cap2) - ref), b = ex2(gp_score<KIND>(s[2 * k + 1], cap2) - ref);
		if (edge) {
			a = 2 * k > last ? 0.f : a;
			b = 2 * k + 1 > last ? 0.f : b;
		}
		t0 += a;
		t1 += b;
		const uint32_t hi = pack_bf16(a, b);
		out[k] = hi;
		out[16 + k] = pack_bf16(a - __uint_as_float(hi << 16), b - __uint_as_float(hi & 0xFFFF0000u));
	}
	return t0 + t1;
}

// The same with reference point zero.  SMALL: cap * tanh by the polynomial, its coefficients times the cap; else by the exponential.
template <bool SMALL>
__device__ __forceinline__ float gp_weights_fixed(const float (&s)[32], uint32_t (&out)[32], float cap2, bool edge, int last) {
	f32x2 total = pack2(0.f, 0.f);
	const float c0 = 9.999993948e-01f * cap2, c1 = -3.332895137e-01f * cap2, c2 = 1.328072065e-01f * cap2, c3 = -5.158598840e-02f * cap2, c4 = 1.672085518e-02f * cap2,
				c5 = -3.058229038e-03f * cap2;
#pragma unroll
	for (int k = 0; k < 16; ++k) {
		float a, b;
		if (SMALL) {
			const f32x2 x = pack2(s[2 * k], s[2 * k + 1]), u = mul2(x, x);
			f32x2 r = fma2(u, pack2(c5, c5), pack2(c4, c4));
			r = fma2(r, u, pack2(c3, c3));
			r = fma2(r, u, pack2(c2, c2));
			r = fma2(r, u, pack2(c1, c1));
			r = fma2(r, u, pack2(c0, c0));
			unpack2(mul2(r, x), a, b);
		} else {
			a = cap2 * tanh_any(s[2 * k]);
			b = cap2 * tanh_any(s[2 * k + 1]);
		}
		a = ex2(a);
		b = ex2(b);
		if (edge) {
			a = 2 * k > last ? 0.f : a;
			b = 2 * k + 1 > last ? 0.f : b;
		}
		const f32x2 ab = pack2(a, b);
		total = add2(total, ab);
		const uint32_t hi = pack_bf16(a, b);
		out[k] = hi;
		float la, lb;
		unpack2(fma2(pack2(__uint_as_float(hi << 16), __uint_as_float(hi & 0xFFFF0000u)), pack2(-1.f, -1.f), ab), la, lb);
		out[16 + k] = pack_bf16(la, lb);
	}
	float t0, t1;
	unpack2(total, t0, t1);
	return t0 + t1;
}

enum { MODE_PLAIN, MODE_CAP, MODE_FIXED };                // no cap; cap and running maximum; cap and reference point zero

// Descriptor of V as the B operand: the contiguous dimension is N (values).  Chunks of 64 value columns lie GP_CHUNK apart, a
// chunk holds rows of 128 bytes (one key each) in groups of 8 keys, 1024 bytes apart; 128-byte swizzle.
__device__ __forceinline__ uint64_t desc_values(uint32_t addr) {
	uint64_t d = 0;
	d |= (uint64_t)((addr & 0x3FFFFu) >> 4);
	d |= (uint64_t)(GP_CHUNK >> 4) << 16;               // leading byte offset: next 64 values
	d |= (uint64_t)(1024 >> 4) << 32;                   // stride byte offset: next 8 keys
	d |= (uint64_t)1 << 46;
	d |= (uint64_t)2 << 61;
	return d;
}

template <int MAPS, int MODE>
__global__ void __launch_bounds__(MAPS * (GP_MAP_THREADS + 32) + 32, 1) gqa_prefill_kernel(const __grid_constant__ CUtensorMap tmq, const __grid_constant__ CUtensorMap tmk,
																		   const __grid_constant__ CUtensorMap tmv, const GqaArgs p, int t, int start, const GpPlan pl,
																		   uint32_t tmem_cols) {
	extern __shared__ unsigned char gp_raw[];
	__shared__ float s_mx[2][MAPS][2][GP_T];          // [parity of the key tile][map][half][row]
	__shared__ float s_sum[2][GP_T], s_sq[4][GP_T];   // [map][row], [quarter of the values][row]
	unsigned char *smem = gp_raw + ((1024u - (smem_u32(gp_raw) & 1023u)) & 1023u);
	const uint32_t q_bytes = pl.nd * GP_CHUNK, k_bytes = MAPS * q_bytes, v_bytes = pl.nv * GP_CHUNK;
	const uint32_t sq = smem_u32(smem), sk = sq + MAPS * q_bytes, sv = sk + pl.sk * k_bytes;
	uint64_t *bars = reinterpret_cast<uint64_t *>(smem + (size_t)MAPS * q_bytes + (size_t)pl.sk * k_bytes + (size_t)pl.sv * v_bytes);
	const uint32_t b0 = smem_u32(bars);
	const uint32_t bar_q = b0, bar_fk = b0 + 16, bar_ek = b0 + 32, bar_fv = b0 + 48, bar_ev = b0 + 64;      // two slots each for K, V
	const uint32_t bar_s = b0 + 80, bar_p = b0 + 96, bar_o = b0 + 112, bar_drain = b0 + 128;              // one per map
	uint32_t *s_tmem = reinterpret_cast<uint32_t *>(bars + 18);
	volatile int *s_abort = reinterpret_cast<volatile int *>(s_tmem + 1);
	const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
	const int units = p.heads * (p.maps / MAPS), nqb = (t + GP_T - 1) / GP_T;          // MAPS = 1: a unit is one map of a head
	const int unit = blockIdx.x % units, q0 = (nqb - 1 - (int)blockIdx.x / units) * GP_T;          // the longest rows first
	const int head = unit * MAPS / p.maps, map0 = unit * MAPS - head * p.maps, kvh = head / (p.heads / p.kv_heads);
	const int n = (start + min(q0 + GP_T, t) - 1) / GP_T + 1;                         // key tiles

	if (tid == 0) {
		mbar_init(bar_q, 1);
		for (int s = 0; s < 2; ++s) {
			mbar_init(bar_fk + 8 * s, 1);
			mbar_init(bar_ek + 8 * s, MAPS);          // every map releases a stage
			mbar_init(bar_fv + 8 * s, 1);
			mbar_init(bar_ev + 8 * s, MAPS);
			mbar_init(bar_s + 8 * s, 1);
			mbar_init(bar_p + 8 * s, GP_MAP_THREADS);
			mbar_init(bar_o + 8 * s, 1);
			mbar_init(bar_drain + 8 * s, 1);
		}
		*s_abort = 0;
		fence_mbar_init();
	}
	constexpr int W_TMA = MAPS * 8, W_MMA = MAPS * 8 + 1;
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
			mbar_arrive_expect_tx(bar_q, MAPS * q_bytes);
			for (int i = 0; i < MAPS; ++i)
				for (int c = 0; c < pl.nd; ++c) tma_load_2d(sq + i * q_bytes + c * GP_CHUNK, &tmq, (head * p.maps + map0 + i) * p.dim + 64 * c, q0, bar_q);
			int jk = 0, jv = 0;
			for (int j = 0; j < n; ++j) {
				const int a = j % pl.sk, b = j % pl.sv;
				if (*s_abort || !mbar_wait_bounded(bar_ek + 8 * a, ((j / pl.sk) & 1) ^ 1, ATTN_SPIN)) { fail(); break; }
				mbar_arrive_expect_tx(bar_fk + 8 * a, k_bytes);
				for (int i = 0; i < MAPS; ++i)
					for (int c = 0; c < pl.nd; ++c)
						tma_load_2d(sk + a * k_bytes + i * q_bytes + c * GP_CHUNK, &tmk, (kvh * p.maps + map0 + i) * p.dim + 64 * c, j * GP_T, bar_fk + 8 * a);
				jk = j + 1;
				if (*s_abort || !mbar_wait_bounded(bar_ev + 8 * b, ((j / pl.sv) & 1) ^ 1, ATTN_SPIN)) { fail(); break; }
				mbar_arrive_expect_tx(bar_fv + 8 * b, v_bytes);
				for (int c = 0; c < pl.nv; ++c) tma_load_2d(sv + b * v_bytes + c * GP_CHUNK, &tmv, kvh * p.vdim + 64 * c, j * GP_T, bar_fv + 8 * b);
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
			const int i = warp - W_MMA;
			const uint32_t base = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(GP_T >> 4) << 24);       // D fp32, A/B bf16, M = 128
			const uint32_t id_qk = base | ((uint32_t)(GP_T >> 3) << 17), id_pv = base | (1u << 16) | ((uint32_t)(p.vdim >> 3) << 17);      // V: N contiguous
			auto wait = [&](uint32_t bar, int k) {
				if (!wait_fast(bar, k & 1, s_abort)) { fail(); return false; }
				tc_fence_after();
				return true;
			};
			auto qk = [&](int j) {
				if (!wait(bar_fk + 8 * (j % pl.sk), j / pl.sk)) return false;
				uint32_t acc = 0;
				// a descriptor advances by 2 (32 bytes) per K step; one thread issues everything, so the loop must stay short
				uint64_t qd = smem_desc_sw128(sq + i * q_bytes), kd = smem_desc_sw128(sk + (j % pl.sk) * k_bytes + i * q_bytes);
				for (int c = 0; c < pl.nd; ++c, qd += GP_CHUNK / 16, kd += GP_CHUNK / 16) {
					const int steps = (p.dim - 64 * c) >> 4;
#pragma unroll
					for (int k = 0; k < 4; ++k)
						if (k < steps) {
							umma_f16(tmem + i * GP_T, qd + 2 * k, kd + 2 * k, id_qk, acc);
							acc = 1;
						}
				}
				umma_commit(bar_s + 8 * i);
				return true;
			};
			auto pv = [&](int j) {
				if (!wait(bar_fv + 8 * (j % pl.sv), j / pl.sv) || !wait(bar_p + 8 * i, j)) return false;
				const uint32_t d = tmem + MAPS * GP_T + i * p.vdim, pa = tmem + i * GP_T;
				const uint64_t vd = desc_values(sv + (j % pl.sv) * v_bytes);
				uint32_t acc = j ? 1u : 0u;
#pragma unroll
				for (int part = 0; part < 2; ++part)
#pragma unroll
					for (int k = 0; k < 8; ++k) {          // 16 keys: 2048 bytes of a chunk
						umma_f16_ts(d, pa + (k >> 1) * 32 + part * 16 + (k & 1) * 8, vd + 128 * k, id_pv, acc);
						acc = 1;
					}
				umma_commit(bar_o + 8 * i);
				return true;
			};
			bool ok = wait(bar_q, 0) && qk(0);
			umma_commit(bar_ek);
			for (int j = 0; j < n && ok; ++j) {
				ok = pv(j);
				umma_commit(bar_ev + 8 * (j % pl.sv));
				if (ok && j + 1 < n) {
					ok = qk(j + 1);
					umma_commit(bar_ek + 8 * ((j + 1) % pl.sk));
				}
			}
			umma_commit(bar_drain + 8 * i);          // every MMA has completed before tensor memory goes back
			mbar_wait_bounded(bar_drain + 8 * i, 0, ATTN_SPIN);
		}
		__syncwarp();
	} else {
		const int i = warp >> 3, half = (warp >> 2) & 1;
		const int rl = (warp & 3) * 32 + lane, row = q0 + rl, pos = start + row;
		const uint32_t lane_base = (uint32_t)((warp & 3) * 32) << 16;
		const uint32_t ts = tmem + i * GP_T + half * 64 + lane_base, to = tmem + MAPS * GP_T + i * p.vdim + lane_base;
		const float cap2 = p.cap * GQ_LOG2E;
		constexpr bool CAP = MODE == MODE_CAP;
		const bool bounded = p.bound > 0.f && p.bound <= 0.98f;          // (queries and keys are rounded to bf16)
		float ref = 0.f, sum = 0.f;
		bool ok = true;
		auto wait = [&](uint32_t bar, int k) {
			const bool got = wait_fast(bar, k & 1, s_abort);
			if (!__all_sync(0xffffffffu, got)) { fail(); return false; }
			tc_fence_after();
			return true;
		};
		auto pair_barrier = [&]() { asm volatile("bar.sync %0, %1;" ::"r"(1 + i), "n"(GP_MAP_THREADS) : "memory"); };
		auto all_barrier = [&]() { asm volatile("bar.sync 3, %0;" ::"n"(MAPS * GP_MAP_THREADS) : "memory"); };
		for (int j = 0; j < n; ++j) {
			// (a wait that ran out does not leave the loop: both halves must keep meeting at the barrier)
			ok = ok && wait(bar_s + 8 * i, j);
			const int last = pos - j * GP_T - half * 64;                                     // last visible key of this half
			const bool edge = j * GP_T + half * 64 + 63 > start + q0 + (warp & 3) * 32;      // this warp's first row does not see all of them
			if (MODE == MODE_FIXED) {
				if (ok) {
#pragma unroll 1
					for (int c = 0; c < 2; ++c) {
						float s[32];
						uint32_t out[32];                // 16 columns of high parts, 16 of remainders
						tmem_ld32(ts + c * 32, s);
						tmem_ld_wait();
						tmem_settle(s);
						bool small = bounded;
						if (!bounded) {
							float g0 = fabsf(s[0]), g1 = fabsf(s[1]);
#pragma unroll
							for (int k = 2; k < 32; k += 2) {
								g0 = fmaxf(g0, fabsf(s[k]));
								g1 = fmaxf(g1, fabsf(s[k + 1]));
							}
							small = !__any_sync(0xffffffffu, fmaxf(g0, g1) > 1.f);
						}
						if (small) sum += gp_weights_fixed<true>(s, out, cap2, edge, last - 32 * c);
						else sum += gp_weights_fixed<false>(s, out, cap2, edge, last - 32 * c);
						tmem_st32(ts + c * 32, out);
					}
					tmem_st_wait();
				}
				tc_fence_before();
				mbar_arrive(bar_p + 8 * i);
				continue;
			}
			float mx = -INFINITY, big = 0.f;
			if (ok) {
				float s[2][32];
				tmem_ld32(ts, s[0]);
				tmem_ld32(ts + 32, s[1]);
				tmem_ld_wait();
				tmem_settle(s[0]);
				tmem_settle(s[1]);
				if (CAP) {
					float g0 = fabsf(s[0][0]), g1 = fabsf(s[0][1]), g2 = fabsf(s[1][0]), g3 = fabsf(s[1][1]);
#pragma unroll
					for (int k = 2; k < 32; k += 2) {
						g0 = fmaxf(g0, fabsf(s[0][k]));
						g1 = fmaxf(g1, fabsf(s[0][k + 1]));
						g2 = fmaxf(g2, fabsf(s[1][k]));
						g3 = fmaxf(g3, fabsf(s[1][k + 1]));
					}
					big = fmaxf(fmaxf(g0, g1), fmaxf(g2, g3));
				}
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
			const bool small = !__any_sync(0xffffffffu, big > 1.f);
			s_mx[j & 1][i][half][rl] = mx;
			pair_barrier();
			mx = fmaxf(mx, s_mx[j & 1][i][half ^ 1][rl]);
			// maximum in base 2; a row below the diagonal of this tile sees none of its keys and keeps its reference point
			const float rm = mx == -INFINITY ? (j ? ref : 0.f) : CAP ? cap2 * tanh_any(mx) : mx;
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
#pragma unroll 1
				for (int c = 0; c < 2; ++c) {
					float s[32];
					uint32_t out[32];                // 16 columns of high parts, 16 of remainders
					tmem_ld32(ts + c * 32, s);
					tmem_ld_wait();
					tmem_settle(s);
					if (!CAP) sum += gp_weights<SCORE_PLAIN>(s, out, cap2, ref, edge, last - 32 * c);
					else if (small) sum += gp_weights<SCORE_SMALL>(s, out, cap2, ref, edge, last - 32 * c);
					else sum += gp_weights<SCORE_ANY>(s, out, cap2, ref, edge, last - 32 * c);
					tmem_st32(ts + c * 32, out);
				}
				tmem_st_wait();
			}
			tc_fence_before();
			mbar_arrive(bar_p + 8 * i);
		}
		s_mx[n & 1][i][half][rl] = sum;
		pair_barrier();
		sum += s_mx[n & 1][i][half ^ 1][rl];
		ok = ok && wait(bar_o + 8 * i, n - 1);
		if (MAPS == 1) {
			if (ok) {
				const size_t slot = ((size_t)row * p.heads + head) * p.maps + map0;
				const float f = 1.f / sum;
				if (half == 0 && row < t) reinterpret_cast<float2 *>(p.part_ml)[slot] = make_float2(0.f, 1.f);
#pragma unroll 1
				for (int c = half * 16; c < p.vdim; c += 32) {
					float o[16];
					tmem_ld16(to + c, o);
					tmem_ld_wait();
					tmem_settle(o);
					if (row < t) {
#pragma unroll
						for (int k = 0; k < 4; ++k)
							*reinterpret_cast<float4 *>(p.part_acc + slot * p.vdim + c + 4 * k) = make_float4(o[4 * k] * f, o[4 * k + 1] * f, o[4 * k + 2] * f, o[4 * k + 3] * f);
					}
				}
			}
		} else {
			// both maps of a row: a quarter of the values (vdim <= 128: two groups of 16 at most) per thread
			if (half == 0) s_sum[i][rl] = sum;
			tc_fence_before();
			all_barrier();
			tc_fence_after();
			const int part = warp >> 2;
			const float f0 = 1.f / s_sum[0][rl], f1 = -p.lambda / s_sum[MAPS - 1][rl];
			float o[2][16], sq2 = 0.f;
#pragma unroll
			for (int g = 0; g < 2; ++g) {
				const int c = part * 16 + 64 * g;
				if (c < p.vdim && ok) {
					float b[16];
					const uint32_t at = tmem + MAPS * GP_T + lane_base + c;
					tmem_ld16(at, o[g]);
					tmem_ld16(at + p.vdim, b);
					tmem_ld_wait();
					tmem_settle(o[g]);
					tmem_settle(b);
#pragma unroll
					for (int k = 0; k < 16; ++k) {
						o[g][k] = fmaf(o[g][k], f0, b[k] * f1);
						sq2 = fmaf(o[g][k], o[g][k], sq2);
					}
				}
			}
			s_sq[part][rl] = sq2;
			all_barrier();
			float f = p.out_mul;
			if (p.out_norm) f /= sqrtf(((s_sq[0][rl] + s_sq[1][rl]) + (s_sq[2][rl] + s_sq[3][rl])) / (float)p.vdim_true + p.eps);
			if (row < t && ok) {
				bf16 *dst = reinterpret_cast<bf16 *>(p.out) + (size_t)row * p.out_ld + head * p.vdim;
#pragma unroll
				for (int g = 0; g < 2; ++g) {
					const int c = part * 16 + 64 * g;
					if (c < p.vdim) {
#pragma unroll
						for (int k = 0; k < 16; ++k) o[g][k] *= f;
						Elem<bf16>::store8(dst + c, o[g]);
						Elem<bf16>::store8(dst + c + 8, o[g] + 8);
					}
				}
			}
		}
	}
	tc_fence_before();
	__syncthreads();
	if (warp == W_MMA) tmem_dealloc(tmem, tmem_cols);
}

// stages for `maps` maps per CTA; false: does not fit
bool gp_plan(int maps, int dim, int vdim, GpPlan *out) {
	GpPlan pl;
	pl.nd = (dim + 63) / 64;
	pl.nv = (vdim + 63) / 64;
	if (vdim > 256 || maps * (GP_T + vdim) > 512) return false;
	const size_t q = (size_t)maps * pl.nd * GP_CHUNK, v = (size_t)pl.nv * GP_CHUNK;
	const int opts[4][2] = {{2, 2}, {1, 2}, {2, 1}, {1, 1}};      // V is needed sooner after its release than K
	for (auto &o : opts) {
		pl.sk = o[0];
		pl.sv = o[1];
		pl.smem = (1 + pl.sk) * q + pl.sv * v + 1024 + 256;
		if (pl.smem <= GP_SMEM) {
			*out = pl;
			return true;
		}
	}
	return false;
}

}   // namespace

int gqa_prefill_maps(int maps, int dim, int vdim) {
	GpPlan pl;
	if (maps == 2 && gp_plan(2, dim, vdim, &pl)) return 2;
	return gp_plan(1, dim, vdim, &pl) ? 1 : 0;
}

int gqa_prefill_launch(const GqaArgs &p, int start, cudaStream_t stream) {
	GpPlan pl;
	const int maps = gqa_prefill_maps(p.maps, p.dim, p.vdim), t = p.M, S = start + t;
	if (!maps || !gp_plan(maps, p.dim, p.vdim, &pl)) return GPTQ_ERR_UNSUPPORTED;
	alignas(64) CUtensorMap tmq, tmk, tmv;
	const long long qc = (long long)p.heads * p.maps * p.dim, kc = (long long)p.kv_heads * p.maps * p.dim, vc = (long long)p.kv_heads * p.vdim;
	if (int rc = dense_tensor_map(p.q_hi, t, qc, qc, GP_T, 64, &tmq)) return rc;
	if (int rc = dense_tensor_map(p.k_cache, S, kc, kc, GP_T, 64, &tmk)) return rc;
	if (int rc = dense_tensor_map(p.v_cache, S, vc, vc, GP_T, 64, &tmv)) return rc;      // keys behind S read as zero
	uint32_t cols = 32;
	while (cols < (uint32_t)(maps * (GP_T + p.vdim))) cols *= 2;
	const dim3 grid(p.heads * (p.maps / maps) * ((t + GP_T - 1) / GP_T)), block(maps * (GP_MAP_THREADS + 32) + 32);
	const int mode = p.cap <= 0.f ? MODE_PLAIN : p.cap * GQ_LOG2E <= 100.f ? MODE_FIXED : MODE_CAP;
	auto go = [&](auto kernel) { return dn_launch(kernel, grid, block, pl.smem, stream, tmq, tmk, tmv, p, t, start, pl, cols); };
	if (maps == 2) return mode == MODE_PLAIN ? go(gqa_prefill_kernel<2, MODE_PLAIN>) : mode == MODE_CAP ? go(gqa_prefill_kernel<2, MODE_CAP>) : go(gqa_prefill_kernel<2, MODE_FIXED>);
	return mode == MODE_PLAIN ? go(gqa_prefill_kernel<1, MODE_PLAIN>) : mode == MODE_CAP ? go(gqa_prefill_kernel<1, MODE_CAP>) : go(gqa_prefill_kernel<1, MODE_FIXED>);
}

}   // namespace gptq
