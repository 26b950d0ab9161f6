// Grouped-query attention with one or two softmax maps per head, for few query rows (decode steps, short portions) and, in
// fp32, for any number of them.
//
//   gqa_append    RMS norm of queries and keys (per head and map), cache rows
//   gqa_attend    scores, soft cap, online softmax in base 2, sum of p_j v_j over one range of the keys
//   gqa_merge     merges the ranges, combines a head's two maps, norm over the head's values
// A cached key row holds the maps of a key head next to each other.  In the bf16 kernel a CTA serves up to 16 (map, query head)
// rows of one key / value head: a row of map m is zero outside the m-th part, so one product with the whole key row gives every
// row its own map's score, and all rows share the values.  Queries and softmax weights are split into two bf16 values each (high part
// and remainder), so both keep about 16 bits of mantissa; scores, weights and sums are fp32.
#include <algorithm>

#include "gqa.cuh"

namespace gptq {

namespace {

constexpr int GQ_V = 4;                  // float4 units of a head vector per lane: dim, vdim <= 512
constexpr int GQ_SPLITS = 64;

// ---- norms and cache rows: LANES lanes per head vector, four entries per lane and unit ---------------------------------------------
// R: type of the raw rows (fp32, or bf16 for prompts), T: of the cache
template <typename R, typename T, int LANES, int UNITS>
__global__ void __launch_bounds__(DN_THREADS) gqa_append_kernel(const GqaArgs p) {
	constexpr int PER_CTA = DN_THREADS / LANES;
	const int nq = p.heads * p.maps, nk = p.kv_heads * p.maps, rows = nq + nk + p.kv_heads;
	const long long id = (long long)blockIdx.x * PER_CTA + threadIdx.x / LANES;
	const int lane = threadIdx.x % LANES;
	const int m = (int)(id / rows), r = (int)(id - (long long)m * rows);
	const bool value = r >= nq + nk, query = r < nq;
	const int n = value ? p.vdim : p.dim;
	const float *gain = value ? nullptr : query ? p.q_norm : p.k_norm;
	float4 g[UNITS];
#pragma unroll
	for (int i = 0; i < UNITS; ++i) {
		const int c = (i * LANES + lane) * 4;
		g[i] = gain && c < n ? __ldg(reinterpret_cast<const float4 *>(gain + c)) : make_float4(1.f, 1.f, 1.f, 1.f);
	}
	pdl_wait();
	pdl_trigger();
	const int pos = m < p.M ? __ldcg(p.pos + m) : -1, seq = m / p.rows_per_seq;
	const bool live = pos >= 0 && pos < p.max_seq;
	if (m < p.M && !live && lane == 0) atomicExch(p.status, DN_BAD_POSITION);      // a position outside the cache is dropped
	const R *src = reinterpret_cast<const R *>(p.raw) + (size_t)m * p.raw_ld + (value ? (nq + nk) * p.dim + (r - nq - nk) * p.vdim : r * p.dim);
	float4 v[UNITS];
	float s = 0.f;
#pragma unroll
	for (int i = 0; i < UNITS; ++i) {
		const int c = (i * LANES + lane) * 4;
		v[i] = live && c < n ? Elem<R>::ldcg4(src + c) : make_float4(0.f, 0.f, 0.f, 0.f);
		s = fmaf(v[i].x, v[i].x, fmaf(v[i].y, v[i].y, fmaf(v[i].z, v[i].z, fmaf(v[i].w, v[i].w, s))));
	}
#pragma unroll
	for (int d = LANES / 2; d > 0; d >>= 1) s += __shfl_xor_sync(0xffffffffu, s, d);
	if (!live) return;
	float f = gain ? 1.f / sqrtf(s / (float)p.dim_true + p.eps) : 1.f;
	if (query) f *= gqa_query_factor(p);
	const size_t cache_row = (size_t)seq * p.max_seq + pos;
	T *dst = query ? nullptr : value ? reinterpret_cast<T *>(p.v_cache) + (cache_row * p.kv_heads + (r - nq - nk)) * p.vdim
									 : reinterpret_cast<T *>(p.k_cache) + (cache_row * nk + (r - nq)) * p.dim;
	const size_t qo = ((size_t)m * nq + r) * p.dim;
#pragma unroll
	for (int i = 0; i < UNITS; ++i) {
		const int c = (i * LANES + lane) * 4;
		if (c < n) {
			const float4 o = make_float4(v[i].x * f * g[i].x, v[i].y * f * g[i].y, v[i].z * f * g[i].z, v[i].w * f * g[i].w);
			if (!query) {
				Elem<T>::store4(dst + c, o);
			} else if (sizeof(T) == 4) {
				*reinterpret_cast<float4 *>(p.q_f32 + qo + c) = o;
			} else {
				Elem<bf16>::store4(reinterpret_cast<bf16 *>(p.q_hi) + qo + c, o);
				if (p.q_lo) {
					auto rest = [](float a) { return a - __bfloat162float(__float2bfloat16_rn(a)); };
					Elem<bf16>::store4(reinterpret_cast<bf16 *>(p.q_lo) + qo + c, make_float4(rest(o.x), rest(o.y), rest(o.z), rest(o.w)));
				}
			}
		}
	}
}

// ---- attention over a range of keys, bf16 -----------------------------------------------------------------------------
constexpr int GA_KEYS = 32;              // keys per tile
constexpr int GA_ROWS = 16;              // (map, query head) rows per CTA
constexpr size_t GA_STATIC = 8 * 1024;   // more than its static shared memory and what the system keeps

struct GaPlan {
	int kd, krow, vrow, stages;          // key entries; bytes of a staged key / value row (padded against bank conflicts)
	size_t smem;
};
__host__ __device__ inline GaPlan ga_plan(int maps, int dim, int vdim) {
	GaPlan g;
	g.kd = maps * dim;
	g.krow = g.kd * 2 + 16;
	g.vrow = vdim * 2 + 16;
	const size_t q = 2 * GA_ROWS * (size_t)g.krow, tile = GA_KEYS * (size_t)(g.krow + g.vrow);
	g.stages = q + 3 * tile <= 100 * 1024 ? 3 : q + 2 * tile <= 100 * 1024 ? 2 : q + 3 * tile <= 200 * 1024 ? 3 : q + 2 * tile <= 200 * 1024 ? 2 : 1;
	g.smem = q + g.stages * tile;
	return g;
}

template <int NTW>                       // 8-column tiles of the values per warp: vdim <= 64 * NTW
__global__ void __launch_bounds__(DN_THREADS) gqa_attend_kernel(const GqaArgs p) {
	extern __shared__ __align__(16) unsigned char ga_smem[];
	__shared__ float s_s[2][GA_ROWS][GA_KEYS + 1];
	__shared__ __align__(16) bf16 s_p[2][GA_ROWS][GA_KEYS + 8];
	__shared__ float s_corr[GA_ROWS];
	const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gid = lane >> 2, tig = lane & 3;
	const GaPlan g = ga_plan(p.maps, p.dim, p.vdim);
	const int stages = g.stages, ratio = p.heads / p.kv_heads, rows = p.maps * ratio, rtiles = (rows + GA_ROWS - 1) / GA_ROWS;
	const int kvh = blockIdx.y / rtiles, r0 = (blockIdx.y - kvh * rtiles) * GA_ROWS, nr = min(GA_ROWS, rows - r0);
	const int m = blockIdx.z, split = blockIdx.x, seq = m / p.rows_per_seq;
	const int kc = g.kd >> 3, vc = p.vdim >> 3;                             // 16-byte chunks of a key / value row
	// entries of the key rows that this CTA's rows look at (those of their maps)
	const int d_lo = (r0 / ratio) * p.dim, d_hi = ((r0 + nr - 1) / ratio + 1) * p.dim;
	const uint32_t krow = g.krow, vrow = g.vrow, tile_bytes = GA_KEYS * (krow + vrow);
	const uint32_t sq = smem_u32(ga_smem), st = sq + 2 * GA_ROWS * krow;
	// positions are older than the previous launch (see the note on dependent launch), and so are the cache rows before the
	// first position of this call
	const int len = max(1, min(__ldcg(p.pos + m) + 1, p.max_seq)), fresh = __ldcg(p.pos + seq * p.rows_per_seq);
	const int tiles = (len + GA_KEYS - 1) / GA_KEYS;
	const int t_lo = (int)((long long)split * tiles / p.splits), ntiles = (int)((long long)(split + 1) * tiles / p.splits) - t_lo;
	const int k_lo = t_lo * GA_KEYS, k_hi = min(k_lo + ntiles * GA_KEYS, len);
	const size_t kld = (size_t)p.kv_heads * g.kd, vld = (size_t)p.kv_heads * p.vdim;
	const bf16 *kc_g = reinterpret_cast<const bf16 *>(p.k_cache) + (size_t)seq * p.max_seq * kld + (size_t)kvh * g.kd;
	const bf16 *vc_g = reinterpret_cast<const bf16 *>(p.v_cache) + (size_t)seq * p.max_seq * vld + (size_t)kvh * p.vdim;
	auto fetch = [&](int t) {            // keys beyond the range repeat the last one (their scores are masked)
		const uint32_t dk = st + (uint32_t)(t % stages) * tile_bytes, dv = dk + GA_KEYS * krow;
		for (int i = tid; i < GA_KEYS * kc; i += DN_THREADS) {
			const int k = i / kc, c = i - k * kc;
			const int key = min(k_lo + t * GA_KEYS + k, k_hi - 1);
			asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dk + k * krow + c * 16), "l"(kc_g + (size_t)key * kld + c * 8) : "memory");
		}
		for (int i = tid; i < GA_KEYS * vc; i += DN_THREADS) {
			const int k = i / vc, c = i - k * vc;
			const int key = min(k_lo + t * GA_KEYS + k, k_hi - 1);
			asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dv + k * vrow + c * 16), "l"(vc_g + (size_t)key * vld + c * 8) : "memory");
		}
	};
	int old = 0;                          // leading tiles that may be fetched ahead of the wait
	while (old < min(ntiles, stages - 1) && k_lo + (old + 1) * GA_KEYS <= fresh) fetch(old++);
	pdl_wait();
	pdl_trigger();
	for (int i = tid; i < 2 * GA_ROWS * kc; i += DN_THREADS) {              // query rows, zero outside their map
		const int part = i / (GA_ROWS * kc), j = i - part * GA_ROWS * kc, rr = j / kc, c = (j - rr * kc) * 8;
		const int r = r0 + min(rr, nr - 1), map = r / ratio, head = kvh * ratio + r - map * ratio, d = c - map * p.dim;
		uint4 v = make_uint4(0u, 0u, 0u, 0u);
		if (rr < nr && d >= 0 && d < p.dim)
			v = __ldcg(reinterpret_cast<const uint4 *>(reinterpret_cast<const bf16 *>(part ? p.q_lo : p.q_hi) + (((size_t)m * p.heads + head) * p.maps + map) * p.dim + d));
		*reinterpret_cast<uint4 *>(ga_smem + (size_t)(part * GA_ROWS + rr) * krow + c * 2) = v;
	}
	for (int t = 0; t < stages - 1; ++t) {
		if (t >= old && t < ntiles) fetch(t);
		cp_async_commit();
	}

	float acc[NTW][4];
#pragma unroll
	for (int n = 0; n < NTW; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
	float mx[2] = {-INFINITY, -INFINITY}, sum[2] = {0.f, 0.f};          // of rows 2 * warp, 2 * warp + 1
	const float cap2 = p.cap * GQ_LOG2E;
	const int kg = warp & 3, kh = warp >> 2;
	// ldmatrix row addresses: A 16 x 16 (lanes 0-15 rows, upper lanes the second 8 columns), B 8 keys x 16
	const uint32_t a_off = (uint32_t)(lane & 15) * krow + (uint32_t)(lane >> 4) * 16;
	const uint32_t b_off = (uint32_t)(kg * 8 + (lane & 7)) * krow + (uint32_t)((lane >> 3) & 1) * 16;
#pragma unroll 1
	for (int t = 0; t < ntiles; ++t) {
		if (t + stages - 1 < ntiles) fetch(t + stages - 1);
		cp_async_commit();
		if (stages == 3) cp_async_wait<2>();
		else if (stages == 2) cp_async_wait<1>();
		else cp_async_wait<0>();
		__syncthreads();
		const uint32_t kt = st + (uint32_t)(t % stages) * tile_bytes, vt = kt + GA_KEYS * krow;
		// scores of 16 rows x 8 keys; the two warps of a key group share the entries
		float s[4] = {0.f, 0.f, 0.f, 0.f}, sl[4] = {0.f, 0.f, 0.f, 0.f};      // high and remainder parts: two independent chains
#pragma unroll 4
		for (int k = (d_lo >> 4) + kh; k < d_hi >> 4; k += 2) {
			uint32_t a[4], al[4], b[2];
			ldmatrix_x2(b, kt + b_off + k * 32);
			ldmatrix_x4(a, sq + a_off + k * 32);
			ldmatrix_x4(al, sq + GA_ROWS * krow + a_off + k * 32);
			mma16816_bf16(s, a[0], a[1], a[2], a[3], b[0], b[1]);
			mma16816_bf16(sl, al[0], al[1], al[2], al[3], b[0], b[1]);
		}
#pragma unroll
		for (int i = 0; i < 4; ++i) s[i] += sl[i];
		const int c = kg * 8 + 2 * tig;
		s_s[kh][gid][c] = s[0];
		s_s[kh][gid][c + 1] = s[1];
		s_s[kh][gid + 8][c] = s[2];
		s_s[kh][gid + 8][c + 1] = s[3];
		__syncthreads();
		const bool valid = k_lo + t * GA_KEYS + lane < k_hi;
#pragma unroll
		for (int j = 0; j < 2; ++j) {
			const int h = warp * 2 + j;
			const float v = valid ? gqa_score(s_s[0][h][lane] + s_s[1][h][lane], cap2) : -INFINITY;
			const float mn = fmaxf(mx[j], warp_max(v));                     // finite: a tile holds at least one key
			const float pr = exp2f(v - mn), corr = exp2f(mx[j] - mn);
			sum[j] = sum[j] * corr + warp_sum(pr);
			mx[j] = mn;
			const bf16 hi = __float2bfloat16_rn(pr);
			s_p[0][h][lane] = hi;
			s_p[1][h][lane] = __float2bfloat16_rn(pr - __bfloat162float(hi));
			if (lane == 0) s_corr[h] = corr;
		}
		__syncthreads();
		const float c0 = s_corr[gid], c1 = s_corr[gid + 8];
		uint32_t pa[2][2][4];                                              // [hi / lo][16 keys]
#pragma unroll
		for (int q = 0; q < 2; ++q)
#pragma unroll
			for (int k = 0; k < 2; ++k) ldmatrix_x4(pa[q][k], smem_u32(&s_p[q][lane & 15][k * 16 + (lane >> 4) * 8]));
#pragma unroll
		for (int n = 0; n < NTW; ++n) {
			const int col = (n * DN_WARPS + warp) * 8;
			if (col < p.vdim) {
				acc[n][0] *= c0;
				acc[n][1] *= c0;
				acc[n][2] *= c1;
				acc[n][3] *= c1;
#pragma unroll
				for (int k = 0; k < 2; ++k) {
					uint32_t b[2];
					ldmatrix_x2_trans(b, vt + (uint32_t)(k * 16 + (lane & 15)) * vrow + col * 2);
					mma16816_bf16(acc[n], pa[0][k][0], pa[0][k][1], pa[0][k][2], pa[0][k][3], b[0], b[1]);
					mma16816_bf16(acc[n], pa[1][k][0], pa[1][k][1], pa[1][k][2], pa[1][k][3], b[0], b[1]);
				}
			}
		}
		__syncthreads();                                                   // the stage, the scores and the weights are free again
	}
	cp_async_wait<0>();
	// ---- this range's (max, sum) and weighted values per row -------------------------------------------------------------
	auto slot = [&](int rr) {            // of row r0 + rr: (head, map) and range
		const int r = r0 + rr, map = r / ratio, head = kvh * ratio + r - map * ratio;
		return (((size_t)m * p.heads + head) * p.maps + map) * p.splits + split;
	};
#pragma unroll
	for (int j = 0; j < 2; ++j) {
		const int rr = warp * 2 + j;
		if (lane == 0 && rr < nr) reinterpret_cast<float2 *>(p.part_ml)[slot(rr)] = make_float2(mx[j], sum[j]);
	}
#pragma unroll
	for (int j = 0; j < 2; ++j) {
		const int rr = gid + 8 * j;
		if (rr < nr) {
			float *dst = p.part_acc + slot(rr) * p.vdim;
#pragma unroll
			for (int n = 0; n < NTW; ++n) {
				const int col = (n * DN_WARPS + warp) * 8 + 2 * tig;
				if (col < p.vdim) *reinterpret_cast<float2 *>(dst + col) = make_float2(acc[n][2 * j], acc[n][2 * j + 1]);
			}
		}
	}
}

// ---- the same in fp32: one (head, map) and query row per CTA, a warp per key ---------------------------------------------
__global__ void __launch_bounds__(DN_THREADS) gqa_attend_f32_kernel(const GqaArgs p) {
	__shared__ float s_m[DN_WARPS], s_l[DN_WARPS];
	__shared__ __align__(16) float s_acc[DN_WARPS][GQ_V * 128];
	const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
	const int split = blockIdx.x, hm = blockIdx.y, head = hm / p.maps, map = hm - head * p.maps, m = blockIdx.z, seq = m / p.rows_per_seq;
	const int kvh = head / (p.heads / p.kv_heads);
	pdl_wait();
	pdl_trigger();
	const int len = max(1, min(__ldcg(p.pos + m) + 1, p.max_seq)), per = (len + p.splits - 1) / p.splits;
	const int k_lo = min(split * per, len), k_hi = min(k_lo + per, len);
	const size_t kld = (size_t)p.kv_heads * p.maps * p.dim, vld = (size_t)p.kv_heads * p.vdim;
	const float *q = p.q_f32 + ((size_t)m * p.heads * p.maps + hm) * p.dim;
	const float *kg = reinterpret_cast<const float *>(p.k_cache) + (size_t)seq * p.max_seq * kld + (size_t)(kvh * p.maps + map) * p.dim;
	const float *vg = reinterpret_cast<const float *>(p.v_cache) + (size_t)seq * p.max_seq * vld + (size_t)kvh * p.vdim;
	const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
	const float cap2 = p.cap * GQ_LOG2E;
	float4 qv[GQ_V], acc[GQ_V];
#pragma unroll
	for (int i = 0; i < GQ_V; ++i) {
		const int c = (i * 32 + lane) * 4;
		qv[i] = c < p.dim ? __ldcg(reinterpret_cast<const float4 *>(q + c)) : zero;
		acc[i] = zero;
	}
	float mx = -INFINITY, sum = 0.f;
	for (int key = k_lo + warp; key < k_hi; key += DN_WARPS) {
		float4 v[GQ_V];
		float s = 0.f;
#pragma unroll
		for (int i = 0; i < GQ_V; ++i) {
			const int c = (i * 32 + lane) * 4;
			if (i * 128 < p.vdim) v[i] = c < p.vdim ? __ldcg(reinterpret_cast<const float4 *>(vg + (size_t)key * vld + c)) : zero;
			if (c < p.dim) {
				const float4 k = __ldcg(reinterpret_cast<const float4 *>(kg + (size_t)key * kld + c));
				s = fmaf(qv[i].x, k.x, fmaf(qv[i].y, k.y, fmaf(qv[i].z, k.z, fmaf(qv[i].w, k.w, s))));
			}
		}
		s = gqa_score(warp_sum(s), cap2);
		const float mn = fmaxf(mx, s), corr = exp2f(mx - mn), pr = exp2f(s - mn);
		mx = mn;
		sum = sum * corr + pr;
#pragma unroll
		for (int i = 0; i < GQ_V; ++i) {
			if (i * 128 < p.vdim) {
				acc[i].x = fmaf(pr, v[i].x, acc[i].x * corr);
				acc[i].y = fmaf(pr, v[i].y, acc[i].y * corr);
				acc[i].z = fmaf(pr, v[i].z, acc[i].z * corr);
				acc[i].w = fmaf(pr, v[i].w, acc[i].w * corr);
			}
		}
	}
	if (lane == 0) {
		s_m[warp] = mx;
		s_l[warp] = sum;
	}
#pragma unroll
	for (int i = 0; i < GQ_V; ++i)
		if (i * 128 < p.vdim) *reinterpret_cast<float4 *>(&s_acc[warp][(i * 32 + lane) * 4]) = acc[i];
	__syncthreads();
	float M = -INFINITY, L = 0.f;
#pragma unroll
	for (int w = 0; w < DN_WARPS; ++w) M = fmaxf(M, s_m[w]);
	float wt[DN_WARPS];
#pragma unroll
	for (int w = 0; w < DN_WARPS; ++w) {
		wt[w] = s_m[w] == -INFINITY ? 0.f : exp2f(s_m[w] - M);
		L = fmaf(s_l[w], wt[w], L);
	}
	const size_t o = ((size_t)m * p.heads * p.maps + hm) * p.splits + split;
	if (tid == 0) reinterpret_cast<float2 *>(p.part_ml)[o] = make_float2(M, L);
	for (int c = tid; c < p.vdim; c += DN_THREADS) {
		float v = 0.f;
#pragma unroll
		for (int w = 0; w < DN_WARPS; ++w) v = fmaf(s_acc[w][c], wt[w], v);
		p.part_acc[o * p.vdim + c] = v;
	}
}

// ---- merge of the key ranges, combination of the maps, norm over the head's values -----------------------------------------
template <typename T>
__global__ void __launch_bounds__(DN_THREADS) gqa_merge_kernel(const GqaArgs p) {
	__shared__ float s_w[2][GQ_SPLITS];
	__shared__ __align__(16) float s_o[2][GQ_V * 128];
	__shared__ float s_red[DN_WARPS];
	constexpr int SB = 16;
	const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, head = blockIdx.x, m = blockIdx.y;
	pdl_wait();
	pdl_trigger();
	// half of the threads per map, a float4 of the values each; the partials are requested before their weights are known
	const int map = tid >> 7, c = tid & 127, nc = p.vdim >> 2;
	const bool live = map < p.maps && c < nc;
	const size_t base = (((size_t)m * p.heads + head) * p.maps + min(map, p.maps - 1)) * p.splits;
	const float4 *acc = reinterpret_cast<const float4 *>(p.part_acc + base * p.vdim);
	float4 pre[SB];
	auto load = [&](int s0) {
#pragma unroll
		for (int j = 0; j < SB; ++j) pre[j] = live && s0 + j < p.splits ? __ldcg(acc + (size_t)(s0 + j) * nc + c) : make_float4(0.f, 0.f, 0.f, 0.f);
	};
	load(0);
	if ((warp & 3) == 0 && map < p.maps) {
		float2 ml[GQ_SPLITS / 32];
		float M = -INFINITY;
#pragma unroll
		for (int i = 0; i < GQ_SPLITS / 32; ++i) {
			const int s = i * 32 + lane;
			ml[i] = s < p.splits ? __ldcg(reinterpret_cast<const float2 *>(p.part_ml) + base + s) : make_float2(-INFINITY, 0.f);
			M = fmaxf(M, ml[i].x);
		}
		M = warp_max(M);
		float L = 0.f;
#pragma unroll
		for (int i = 0; i < GQ_SPLITS / 32; ++i) {
			ml[i].x = ml[i].x == -INFINITY ? 0.f : exp2f(ml[i].x - M);
			L = fmaf(ml[i].x, ml[i].y, L);
		}
		L = warp_sum(L);
#pragma unroll
		for (int i = 0; i < GQ_SPLITS / 32; ++i) s_w[map][i * 32 + lane] = ml[i].x / L;
	}
	__syncthreads();
	if (live) {
		float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
		for (int s0 = 0; s0 < p.splits; s0 += SB) {
			if (s0) load(s0);
#pragma unroll
			for (int j = 0; j < SB; ++j) {
				const float w = s_w[map][min(s0 + j, GQ_SPLITS - 1)];
				v.x = fmaf(pre[j].x, w, v.x);
				v.y = fmaf(pre[j].y, w, v.y);
				v.z = fmaf(pre[j].z, w, v.z);
				v.w = fmaf(pre[j].w, w, v.w);
			}
		}
		*reinterpret_cast<float4 *>(&s_o[map][4 * c]) = v;
	}
	__syncthreads();
	float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
	if (tid < nc) {
		o = *reinterpret_cast<const float4 *>(&s_o[0][4 * tid]);
		if (p.maps == 2) {
			const float4 b = *reinterpret_cast<const float4 *>(&s_o[1][4 * tid]);
			o = make_float4(fmaf(-p.lambda, b.x, o.x), fmaf(-p.lambda, b.y, o.y), fmaf(-p.lambda, b.z, o.z), fmaf(-p.lambda, b.w, o.w));
		}
	}
	float f = p.out_mul;
	if (p.out_norm) f /= sqrtf(block_sum(fmaf(o.x, o.x, fmaf(o.y, o.y, fmaf(o.z, o.z, o.w * o.w))), s_red) / (float)p.vdim_true + p.eps);
	if (tid < nc) Elem<T>::store4(reinterpret_cast<T *>(p.out) + (size_t)m * p.out_ld + head * p.vdim + 4 * tid, make_float4(o.x * f, o.y * f, o.z * f, o.w * f));
}

}   // namespace

template <typename R, typename T>
static int append_launch(const GqaArgs &p, cudaStream_t stream) {
	const long long rows = (long long)p.M * (p.heads * p.maps + p.kv_heads * (p.maps + 1));
	const int widest = std::max(p.dim, p.vdim);
	auto go = [&](auto kernel, int lanes) { return dn_launch(kernel, dim3((unsigned)((rows * lanes + DN_THREADS - 1) / DN_THREADS)), dim3(DN_THREADS), 0, stream, p); };
	if (widest <= 64) return go(gqa_append_kernel<R, T, 16, 1>, 16);
	if (widest <= 128) return go(gqa_append_kernel<R, T, 16, 2>, 16);
	if (widest <= 256) return go(gqa_append_kernel<R, T, 32, 2>, 32);
	return go(gqa_append_kernel<R, T, 32, GQ_V>, 32);
}

int gqa_append_launch(const GqaArgs &p, int dtype, cudaStream_t stream) {
	if (dtype) return append_launch<float, float>(p, stream);
	return p.raw_t ? append_launch<bf16, bf16>(p, stream) : append_launch<float, bf16>(p, stream);
}

bool gqa_attend_ok(int maps, int dim, int vdim) { return dim <= GQ_V * 128 && vdim <= GQ_V * 128 && ga_plan(maps, dim, vdim).smem <= 220 * 1024; }

int gqa_splits(int M, int heads, int kv_heads, int maps, int max_seq, int dtype) {
	const int per_row = dtype ? heads * maps : kv_heads * ((heads / kv_heads * maps + GA_ROWS - 1) / GA_ROWS);
	const int want = dn_sm_count() / std::max(1, M * per_row);
	return std::max(1, std::min(std::min(GQ_SPLITS, want), (max_seq + GA_KEYS - 1) / GA_KEYS));
}

int gqa_attend_launch(const GqaArgs &p, int dtype, cudaStream_t stream) {
	if (dtype) return dn_launch(gqa_attend_f32_kernel, dim3(p.splits, p.heads * p.maps, p.M), dim3(DN_THREADS), 0, stream, p);
	const GaPlan g = ga_plan(p.maps, p.dim, p.vdim);
	const int rtiles = (p.heads / p.kv_heads * p.maps + GA_ROWS - 1) / GA_ROWS;
	const dim3 grid(p.splits, p.kv_heads * rtiles, p.M), block(DN_THREADS);
	auto go = [&](auto kernel) { return dn_launch_as(1, (int)((g.smem + GA_STATIC) * 100 / (228 * 1024)) + 1, kernel, grid, block, g.smem, stream, p); };
	if (p.vdim <= 64) return go(gqa_attend_kernel<1>);
	if (p.vdim <= 128) return go(gqa_attend_kernel<2>);
	if (p.vdim <= 256) return go(gqa_attend_kernel<4>);
	return go(gqa_attend_kernel<8>);
}

int gqa_merge_launch(const GqaArgs &p, int dtype, cudaStream_t stream) {
	const dim3 grid(p.heads, p.M), block(DN_THREADS);
	return dtype ? dn_launch(gqa_merge_kernel<float>, grid, block, 0, stream, p) : dn_launch(gqa_merge_kernel<bf16>, grid, block, 0, stream, p);
}

}   // namespace gptq
