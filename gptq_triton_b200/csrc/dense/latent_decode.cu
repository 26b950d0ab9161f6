// Latent attention over a cache of latent rows, absorbed form, for few query rows (decode steps, short portions) and, in
// fp32, for any number of them.
//
// The cache row of a position is [latent (kv_rank) | rotated shared key (rot_dim)].  With q = (q_n, q_r) of a head,
//   score = q_n . (W_uk c) + q_r . k_r = (W_uk^T q_n) . c + q_r . k_r,   output = W_uv (sum_j p_j c_j),
// so a step needs no expanded keys or values:
//   latent_absorb   (W_uk^T q_n | q_r) * scale * log2(e) per head; other CTAs of the same launch norm the new latent, rotate the
//                   new key part and write the cache row
//   latent_attend   scores, online softmax in base 2, sum of p_j c_j over one range of the keys
//   latent_value    merges the ranges, applies W_uv and the head's gate
// bf16: the products run on mma.m16n8k16 with 16 heads as rows.  The absorbed query and the softmax weights are split into two
// bf16 values each (high part and remainder), so both keep about 16 bits of mantissa; scores, weights and sums are fp32.
#include <algorithm>

#include "latent.cuh"

namespace gptq {

namespace {

constexpr float LOG2E = 1.4426950408889634f;
constexpr int AB_R = 64;                 // latent columns per CTA of the absorb kernel
constexpr int AB_M = 8;                  // query rows per pass
constexpr int AB_V = 8;                  // float4 units of a latent per lane: kv_rank <= 1024
constexpr int AB_G = DN_THREADS / 16;    // groups of 16 threads: each takes every 16th row of W_uk

template <typename T>
__global__ void __launch_bounds__(DN_THREADS) latent_absorb_kernel(const LatentArgs p) {
	extern __shared__ __align__(16) float ab_q[];                        // [AB_M][dim]
	__shared__ __align__(16) float s_red[DN_WARPS][AB_M][AB_R];
	const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
	const int chunks = (p.kv_rank + AB_R - 1) / AB_R, R = p.kv_rank + p.rot_dim, hd = p.dim + p.rot_dim;
	const int work = p.heads * chunks;
	if ((int)blockIdx.x >= work) {
		// ---- cache rows: RMS norm of the latent, rotation of the shared key part, both fp32; a warp per row ----------
		const int m = (((int)blockIdx.x - work) + blockIdx.y * ((int)gridDim.x - work)) * DN_WARPS + warp;
		pdl_wait();
		pdl_trigger();
		if (m >= p.M) return;
		const int pos = __ldcg(p.pos + m), seq = m / p.rows_per_seq;
		if (pos < 0 || pos >= p.max_seq) {            // a position outside the cache is dropped
			if (lane == 0) atomicExch(p.status, DN_BAD_POSITION);
			return;
		}
		const float *src = p.kv_raw + (size_t)m * R;
		T *dst = reinterpret_cast<T *>(p.cache) + ((size_t)seq * p.max_seq + pos) * R;
		float4 v[AB_V];
		float s = 0.f;
#pragma unroll
		for (int i = 0; i < AB_V; ++i) {
			const int c = (i * 32 + lane) * 4;
			if (i * 128 < p.kv_rank) {
				v[i] = c < p.kv_rank ? __ldcg(reinterpret_cast<const float4 *>(src + c)) : make_float4(0.f, 0.f, 0.f, 0.f);
				s = fmaf(v[i].x, v[i].x, fmaf(v[i].y, v[i].y, fmaf(v[i].z, v[i].z, fmaf(v[i].w, v[i].w, s))));
			}
		}
		const float inv = 1.f / sqrtf(warp_sum(s) / (float)p.kv_width + p.eps);
#pragma unroll
		for (int i = 0; i < AB_V; ++i) {
			const int c = (i * 32 + lane) * 4;
			if (c < p.kv_rank) {
				const float4 w = __ldg(reinterpret_cast<const float4 *>(p.kv_norm + c));
				Elem<T>::store4(dst + c, make_float4(v[i].x * inv * w.x, v[i].y * inv * w.y, v[i].z * inv * w.z, v[i].w * inv * w.w));
			}
		}
		for (int i = lane; i < p.rot_dim / 2; i += 32) {
			const float2 x = __ldcg(reinterpret_cast<const float2 *>(src + p.kv_rank) + i);
			float u = x.x, w = x.y;
			if (2 * i < p.rot_dims) {
				const size_t t = (size_t)pos * (p.rot_dims / 2) + i;
				const float c = __ldg(p.cos_t + t), sn = __ldg(p.sin_t + t), a = u * c - w * sn;
				w = w * c + u * sn;
				u = a;
			}
			Elem<T>::store(dst + p.kv_rank + 2 * i, u);
			Elem<T>::store(dst + p.kv_rank + 2 * i + 1, w);
		}
		return;
	}
	// ---- absorbed queries ---------------------------------------------------------------------------------------------
	const int head = blockIdx.x / chunks, r0 = (blockIdx.x - head * chunks) * AB_R;
	const int r = r0 + (tid & 15) * 4, g = tid >> 4;
	const T *uk = reinterpret_cast<const T *>(p.w_uk) + (size_t)head * p.dim * p.kv_rank + r;
	constexpr int PF = 8;
	float4 w[PF];
	const bool in = r < p.kv_rank;
#pragma unroll
	for (int i = 0; i < PF; ++i) {
		const int d = g + AB_G * i;
		w[i] = (in && d < p.dim) ? Elem<T>::load4(uk + (size_t)d * p.kv_rank) : make_float4(0.f, 0.f, 0.f, 0.f);
	}
	pdl_wait();
	pdl_trigger();
	const float sc = p.scale * LOG2E;
	for (int mb = blockIdx.y * AB_M; mb < p.M; mb += gridDim.y * AB_M) {
		const int nm = min(AB_M, p.M - mb);
		__syncthreads();
		for (int i = tid; i < nm * p.dim; i += DN_THREADS) {
			const int m = i / p.dim, d = i - m * p.dim;
			ab_q[m * p.dim + d] = __ldcg(p.q + (size_t)(mb + m) * p.heads * hd + (size_t)head * hd + d);
		}
		__syncthreads();
		float acc[AB_M][4] = {};
		for (int d0 = 0; d0 < p.dim; d0 += AB_G * PF) {
#pragma unroll
			for (int i = 0; i < PF; ++i) {
				const int d = d0 + g + AB_G * i;
				if (d >= p.dim) break;
				const float4 v = d0 == 0 ? w[i] : (in ? Elem<T>::load4(uk + (size_t)d * p.kv_rank) : make_float4(0.f, 0.f, 0.f, 0.f));
#pragma unroll
				for (int m = 0; m < AB_M; ++m) {
					if (m < nm) {
						const float q = ab_q[m * p.dim + d];
						acc[m][0] = fmaf(q, v.x, acc[m][0]);
						acc[m][1] = fmaf(q, v.y, acc[m][1]);
						acc[m][2] = fmaf(q, v.z, acc[m][2]);
						acc[m][3] = fmaf(q, v.w, acc[m][3]);
					}
				}
			}
		}
#pragma unroll
		for (int m = 0; m < AB_M; ++m) {
			if (m < nm) {
#pragma unroll
				for (int e = 0; e < 4; ++e) acc[m][e] += __shfl_xor_sync(0xffffffffu, acc[m][e], 16);
				if (lane < 16) *reinterpret_cast<float4 *>(&s_red[warp][m][lane * 4]) = make_float4(acc[m][0], acc[m][1], acc[m][2], acc[m][3]);
			}
		}
		__syncthreads();
		auto put = [&](int m, int col, float v) {
			const size_t o = ((size_t)(mb + m) * p.heads + head) * R + col;
			if (sizeof(T) == 4) {
				p.qa_f32[o] = v;
			} else {
				const bf16 hi = __float2bfloat16_rn(v);
				reinterpret_cast<bf16 *>(p.qa_hi)[o] = hi;
				reinterpret_cast<bf16 *>(p.qa_lo)[o] = __float2bfloat16_rn(v - __bfloat162float(hi));
			}
		};
		for (int i = tid; i < nm * AB_R; i += DN_THREADS) {
			const int m = i / AB_R, c = i - m * AB_R;
			if (r0 + c < p.kv_rank) {
				float v = 0.f;
#pragma unroll
				for (int k = 0; k < DN_WARPS; ++k) v += s_red[k][m][c];
				put(m, r0 + c, v * sc);
			}
		}
		if (r0 == 0)
			for (int i = tid; i < nm * p.rot_dim; i += DN_THREADS) {
				const int m = i / p.rot_dim, c = i - m * p.rot_dim;
				put(m, p.kv_rank + c, __ldcg(p.q + (size_t)(mb + m) * p.heads * hd + (size_t)head * hd + p.dim + c) * sc);
			}
	}
}

// ---- attention over a range of keys, bf16 -----------------------------------------------------------------------------
constexpr int AT_KEYS = 32;              // keys per tile
constexpr int AT_HEADS = 16;             // heads per CTA

__host__ __device__ inline int at_stages(int R) {
	const size_t row = (size_t)R * 2 + 16, tile = AT_KEYS * row, q = 2 * AT_HEADS * row;
	const size_t room = 200 * 1024;
	return q + 3 * tile <= room ? 3 : q + 2 * tile <= room ? 2 : 1;
}

template <int NTW>                       // 8-column tiles of the latent per warp: kv_rank <= 64 * NTW
__global__ void __launch_bounds__(DN_THREADS) latent_attend_kernel(const LatentArgs p) {
	extern __shared__ __align__(16) unsigned char at_smem[];
	__shared__ float s_s[2][AT_HEADS][AT_KEYS + 1];
	__shared__ __align__(16) bf16 s_p[2][AT_HEADS][AT_KEYS + 8];
	__shared__ float s_corr[AT_HEADS];
	const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gid = lane >> 2, tig = lane & 3;
	const int R = p.kv_rank + p.rot_dim, ks = R >> 4, chunks = R >> 3;      // R is a multiple of 16
	const uint32_t row = (uint32_t)R * 2 + 16;
	const int stages = at_stages(R);
	const int m = blockIdx.z, h0 = blockIdx.y * AT_HEADS, split = blockIdx.x, seq = m / p.rows_per_seq;
	const uint32_t sq = smem_u32(at_smem), sk = sq + 2 * AT_HEADS * row;
	// positions are older than the previous launch (see the note on dependent launch), and so are the cache rows before the
	// first position of this call
	const int len = max(1, min(__ldcg(p.pos + m) + 1, p.max_seq)), fresh = __ldcg(p.pos + seq * p.rows_per_seq);
	const int tiles = (len + AT_KEYS - 1) / AT_KEYS;
	const int t_lo = (int)((long long)split * tiles / p.splits), ntiles = (int)((long long)(split + 1) * tiles / p.splits) - t_lo;
	const int k_lo = t_lo * AT_KEYS, k_hi = min(k_lo + ntiles * AT_KEYS, len);
	const bf16 *cache = reinterpret_cast<const bf16 *>(p.cache) + (size_t)seq * p.max_seq * R;
	auto fetch = [&](int t) {            // keys beyond the range repeat the last one (their scores are masked)
		const uint32_t dst = sk + (uint32_t)(t % stages) * AT_KEYS * row;
		for (int i = tid; i < AT_KEYS * chunks; i += DN_THREADS) {
			const int k = i / chunks, c = i - k * chunks;
			const int key = min(k_lo + t * AT_KEYS + k, k_hi - 1);
			asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst + k * row + c * 16), "l"(cache + (size_t)key * R + c * 8) : "memory");
		}
	};
	int old = 0;                          // leading tiles that may be fetched ahead of the wait
	while (old < min(ntiles, stages - 1) && k_lo + (old + 1) * AT_KEYS <= fresh) fetch(old++);
	pdl_wait();
	pdl_trigger();
	for (int i = tid; i < 2 * AT_HEADS * chunks; i += DN_THREADS) {
		const int part = i / (AT_HEADS * chunks), j = i - part * AT_HEADS * chunks, hh = j / chunks, c = j - hh * chunks;
		const bf16 *src = reinterpret_cast<const bf16 *>(part ? p.qa_lo : p.qa_hi) + ((size_t)m * p.heads + min(h0 + hh, p.heads - 1)) * R + c * 8;
		asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(sq + (part * AT_HEADS + hh) * row + c * 16), "l"(src) : "memory");
	}
	for (int t = 0; t < stages - 1; ++t) {
		if (t >= old && t < ntiles) fetch(t);
		cp_async_commit();
	}

	float acc[NTW][4];
#pragma unroll
	for (int n = 0; n < NTW; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
	float mx[2] = {-INFINITY, -INFINITY}, sum[2] = {0.f, 0.f};          // of head rows 2 * warp, 2 * warp + 1
	const int kg = warp & 3, kh = warp >> 2;
	// ldmatrix row addresses: A 16 x 16 (lanes 0-15 rows, upper lanes the second 8 columns), B 8 keys x 16
	const uint32_t a_off = (uint32_t)(lane & 15) * row + (uint32_t)(lane >> 4) * 16;
	const uint32_t b_off = (uint32_t)(kg * 8 + (lane & 7)) * row + (uint32_t)((lane >> 3) & 1) * 16;
#pragma unroll 1
	for (int t = 0; t < ntiles; ++t) {
		if (t + stages - 1 < ntiles) fetch(t + stages - 1);
		cp_async_commit();
		if (stages == 3) cp_async_wait<2>();
		else if (stages == 2) cp_async_wait<1>();
		else cp_async_wait<0>();
		__syncthreads();
		const uint32_t kt = sk + (uint32_t)(t % stages) * AT_KEYS * row;
		// scores of 16 heads x 8 keys; the two warps of a key group share the k range
		float s[4] = {0.f, 0.f, 0.f, 0.f}, sl[4] = {0.f, 0.f, 0.f, 0.f};      // high and remainder parts: two independent chains
#pragma unroll 4
		for (int k = kh; k < ks; k += 2) {
			uint32_t a[4], al[4], b[2];
			ldmatrix_x2(b, kt + b_off + k * 32);
			ldmatrix_x4(a, sq + a_off + k * 32);
			ldmatrix_x4(al, sq + AT_HEADS * row + a_off + k * 32);
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
		const bool valid = k_lo + t * AT_KEYS + lane < k_hi;
#pragma unroll
		for (int j = 0; j < 2; ++j) {
			const int h = warp * 2 + j;
			const float v = valid ? s_s[0][h][lane] + s_s[1][h][lane] : -INFINITY;
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
			if (col < p.kv_rank) {
				acc[n][0] *= c0;
				acc[n][1] *= c0;
				acc[n][2] *= c1;
				acc[n][3] *= c1;
#pragma unroll
				for (int k = 0; k < 2; ++k) {
					uint32_t b[2];
					ldmatrix_x2_trans(b, kt + (uint32_t)(k * 16 + (lane & 15)) * row + col * 2);
					mma16816_bf16(acc[n], pa[0][k][0], pa[0][k][1], pa[0][k][2], pa[0][k][3], b[0], b[1]);
					mma16816_bf16(acc[n], pa[1][k][0], pa[1][k][1], pa[1][k][2], pa[1][k][3], b[0], b[1]);
				}
			}
		}
		__syncthreads();                                                   // the stage, the scores and the weights are free again
	}
	cp_async_wait<0>();
	// ---- this range's (max, sum) and weighted latent per head -------------------------------------------------------------
#pragma unroll
	for (int j = 0; j < 2; ++j) {
		const int h = h0 + warp * 2 + j;
		if (lane == 0 && h < p.heads) reinterpret_cast<float2 *>(p.part_ml)[((size_t)m * p.heads + h) * p.splits + split] = make_float2(mx[j], sum[j]);
	}
#pragma unroll
	for (int n = 0; n < NTW; ++n) {
		const int col = (n * DN_WARPS + warp) * 8 + 2 * tig;
		if (col < p.kv_rank) {
#pragma unroll
			for (int j = 0; j < 2; ++j) {
				const int h = h0 + gid + 8 * j;
				if (h < p.heads)
					*reinterpret_cast<float2 *>(p.part_acc + (((size_t)m * p.heads + h) * p.splits + split) * p.kv_rank + col) = make_float2(acc[n][2 * j], acc[n][2 * j + 1]);
			}
		}
	}
}

// ---- the same in fp32: one head and query row per CTA, a warp per key ---------------------------------------------------
constexpr int AF_V = 8;                  // float4 units of the latent per lane: kv_rank <= 1024
constexpr int AF_RV = 2;                 // ... and of the rotated part: rot_dim <= 256

__global__ void __launch_bounds__(DN_THREADS) latent_attend_f32_kernel(const LatentArgs p) {
	__shared__ float s_m[DN_WARPS], s_l[DN_WARPS];
	__shared__ __align__(16) float s_acc[DN_WARPS][AF_V * 128];
	const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
	const int R = p.kv_rank + p.rot_dim, split = blockIdx.x, head = blockIdx.y, m = blockIdx.z, seq = m / p.rows_per_seq;
	pdl_wait();
	pdl_trigger();
	const int len = max(1, min(__ldcg(p.pos + m) + 1, p.max_seq)), per = (len + p.splits - 1) / p.splits;
	const int k_lo = min(split * per, len), k_hi = min(k_lo + per, len);
	const float *q = p.qa_f32 + ((size_t)m * p.heads + head) * R, *cache = reinterpret_cast<const float *>(p.cache) + (size_t)seq * p.max_seq * R;
	const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
	float4 qn[AF_V], qr[AF_RV], acc[AF_V];
#pragma unroll
	for (int i = 0; i < AF_V; ++i) {
		const int c = (i * 32 + lane) * 4;
		qn[i] = c < p.kv_rank ? __ldcg(reinterpret_cast<const float4 *>(q + c)) : zero;
		acc[i] = zero;
	}
#pragma unroll
	for (int i = 0; i < AF_RV; ++i) {
		const int c = (i * 32 + lane) * 4;
		qr[i] = c < p.rot_dim ? __ldcg(reinterpret_cast<const float4 *>(q + p.kv_rank + c)) : zero;
	}
	float mx = -INFINITY, sum = 0.f;
	for (int key = k_lo + warp; key < k_hi; key += DN_WARPS) {
		const float *kr = cache + (size_t)key * R;
		float4 kv[AF_V];
		float s = 0.f;
#pragma unroll
		for (int i = 0; i < AF_V; ++i) {
			const int c = (i * 32 + lane) * 4;
			if (i * 128 < p.kv_rank) {
				kv[i] = c < p.kv_rank ? __ldcg(reinterpret_cast<const float4 *>(kr + c)) : zero;
				s = fmaf(qn[i].x, kv[i].x, fmaf(qn[i].y, kv[i].y, fmaf(qn[i].z, kv[i].z, fmaf(qn[i].w, kv[i].w, s))));
			}
		}
#pragma unroll
		for (int i = 0; i < AF_RV; ++i) {
			const int c = (i * 32 + lane) * 4;
			if (c < p.rot_dim) {
				const float4 v = __ldcg(reinterpret_cast<const float4 *>(kr + p.kv_rank + c));
				s = fmaf(qr[i].x, v.x, fmaf(qr[i].y, v.y, fmaf(qr[i].z, v.z, fmaf(qr[i].w, v.w, s))));
			}
		}
		s = warp_sum(s);
		const float mn = fmaxf(mx, s), corr = exp2f(mx - mn), pr = exp2f(s - mn);
		mx = mn;
		sum = sum * corr + pr;
#pragma unroll
		for (int i = 0; i < AF_V; ++i) {
			if (i * 128 < p.kv_rank) {
				acc[i].x = fmaf(pr, kv[i].x, acc[i].x * corr);
				acc[i].y = fmaf(pr, kv[i].y, acc[i].y * corr);
				acc[i].z = fmaf(pr, kv[i].z, acc[i].z * corr);
				acc[i].w = fmaf(pr, kv[i].w, acc[i].w * corr);
			}
		}
	}
	if (lane == 0) {
		s_m[warp] = mx;
		s_l[warp] = sum;
	}
#pragma unroll
	for (int i = 0; i < AF_V; ++i)
		if (i * 128 < p.kv_rank) *reinterpret_cast<float4 *>(&s_acc[warp][(i * 32 + lane) * 4]) = acc[i];
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
	const size_t o = ((size_t)m * p.heads + head) * p.splits + split;
	if (tid == 0) reinterpret_cast<float2 *>(p.part_ml)[o] = make_float2(M, L);
	for (int c = tid; c < p.kv_rank; c += DN_THREADS) {
		float v = 0.f;
#pragma unroll
		for (int w = 0; w < DN_WARPS; ++w) v = fmaf(s_acc[w][c], wt[w], v);
		p.part_acc[o * p.kv_rank + c] = v;
	}
}

// ---- merge of the key ranges, W_uv, gate -----------------------------------------------------------------------------
constexpr int VA_ROWS = 32;              // value rows per CTA: four per warp
constexpr int VA_SPLITS = 64;

template <typename T>
__global__ void __launch_bounds__(DN_THREADS, 1) latent_value_kernel(const LatentArgs p) {
	extern __shared__ __align__(16) float va_lat[];      // [2][kv_rank]
	__shared__ float s_w[VA_SPLITS];
	constexpr int E = 16 / sizeof(T), PF = 2 * sizeof(T) / 2, RW = VA_ROWS / DN_WARPS, SB = 16;
	const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, head = blockIdx.y, m = blockIdx.z, v0 = blockIdx.x * VA_ROWS + warp * RW;
	const T *uv = reinterpret_cast<const T *>(p.w_uv) + (size_t)head * p.vdim * p.kv_rank;
	const uint4 zero4 = make_uint4(0u, 0u, 0u, 0u);
	uint4 w[RW][PF];                     // this warp's rows of W_uv, up to 512 columns
	auto load_w = [&](int r, int i) {
		const int c = (i * 32 + lane) * E;
		return v0 + r < p.vdim && c < p.kv_rank ? ld_nc_v4(uv + (size_t)(v0 + r) * p.kv_rank + c) : zero4;
	};
#pragma unroll
	for (int r = 0; r < RW; ++r)
#pragma unroll
		for (int i = 0; i < PF; ++i) w[r][i] = load_w(r, i);
	pdl_wait();
	pdl_trigger();
	const size_t base = ((size_t)m * p.heads + head) * p.splits;
	const float gate = p.gate ? __ldcg(p.gate + (size_t)m * p.gate_ld + head) : 1.f;
	// weighted sum over the ranges: half the threads take the even ranges, half the odd ones; the partials are requested before
	// their weights are known
	const int half = tid >> 7, nc = p.kv_rank >> 2;
	const float4 *acc = reinterpret_cast<const float4 *>(p.part_acc + base * p.kv_rank);
	float4 pre[SB];
	auto load_acc = [&](int s0, int c) {
#pragma unroll
		for (int j = 0; j < SB; ++j) {
			const int s = s0 + 2 * j + half;
			pre[j] = s < p.splits && c < nc ? __ldcg(acc + (size_t)s * nc + c) : make_float4(0.f, 0.f, 0.f, 0.f);
		}
	};
	load_acc(0, tid & 127);
	if (warp == 0) {
		float2 ml[VA_SPLITS / 32];
		float M = -INFINITY;
#pragma unroll
		for (int i = 0; i < VA_SPLITS / 32; ++i) {
			const int s = i * 32 + lane;
			ml[i] = s < p.splits ? __ldcg(reinterpret_cast<const float2 *>(p.part_ml) + base + s) : make_float2(-INFINITY, 0.f);
			M = fmaxf(M, ml[i].x);
		}
		M = warp_max(M);
		float L = 0.f;
#pragma unroll
		for (int i = 0; i < VA_SPLITS / 32; ++i) {
			ml[i].x = ml[i].x == -INFINITY ? 0.f : exp2f(ml[i].x - M);
			L = fmaf(ml[i].x, ml[i].y, L);
		}
		L = warp_sum(L);
#pragma unroll
		for (int i = 0; i < VA_SPLITS / 32; ++i) s_w[i * 32 + lane] = ml[i].x / L;
	}
	__syncthreads();
	for (int c = tid & 127; c < nc; c += 128) {
		float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
		for (int s0 = 0; s0 < p.splits; s0 += 2 * SB) {
			if (s0 || c >= 128) load_acc(s0, c);
#pragma unroll
			for (int j = 0; j < SB; ++j) {
				const float ws = s_w[min(s0 + 2 * j + half, VA_SPLITS - 1)];
				v.x = fmaf(pre[j].x, ws, v.x);
				v.y = fmaf(pre[j].y, ws, v.y);
				v.z = fmaf(pre[j].z, ws, v.z);
				v.w = fmaf(pre[j].w, ws, v.w);
			}
		}
		*reinterpret_cast<float4 *>(va_lat + half * p.kv_rank + 4 * c) = v;
	}
	__syncthreads();
	float sum[RW] = {};
	auto dot = [&](int r, int c, uint4 a) {
		const float4 l0 = *reinterpret_cast<const float4 *>(va_lat + c), l1 = *reinterpret_cast<const float4 *>(va_lat + p.kv_rank + c);
		if (sizeof(T) == 4) {
			sum[r] = fmaf(__uint_as_float(a.x), l0.x + l1.x, fmaf(__uint_as_float(a.y), l0.y + l1.y, fmaf(__uint_as_float(a.z), l0.z + l1.z, fmaf(__uint_as_float(a.w), l0.w + l1.w, sum[r]))));
		} else {
			const float4 k0 = *reinterpret_cast<const float4 *>(va_lat + c + 4), k1 = *reinterpret_cast<const float4 *>(va_lat + p.kv_rank + c + 4);
			const float4 f = Elem<bf16>::unpack(make_uint2(a.x, a.y)), g = Elem<bf16>::unpack(make_uint2(a.z, a.w));
			sum[r] = fmaf(f.x, l0.x + l1.x, fmaf(f.y, l0.y + l1.y, fmaf(f.z, l0.z + l1.z, fmaf(f.w, l0.w + l1.w, sum[r]))));
			sum[r] = fmaf(g.x, k0.x + k1.x, fmaf(g.y, k0.y + k1.y, fmaf(g.z, k0.z + k1.z, fmaf(g.w, k0.w + k1.w, sum[r]))));
		}
	};
#pragma unroll
	for (int i = 0; i < PF; ++i) {
		const int c = (i * 32 + lane) * E;
		if (c < p.kv_rank) {
#pragma unroll
			for (int r = 0; r < RW; ++r) dot(r, c, w[r][i]);
		}
	}
	for (int i = PF; i * 32 * E < p.kv_rank; ++i) {
		const int c = (i * 32 + lane) * E;
		if (c < p.kv_rank) {
#pragma unroll
			for (int r = 0; r < RW; ++r) dot(r, c, load_w(r, i));
		}
	}
#pragma unroll
	for (int r = 0; r < RW; ++r) {
		const float v = warp_sum(sum[r]);
		if (lane == 0 && v0 + r < p.vdim) Elem<T>::store(reinterpret_cast<T *>(p.out) + (size_t)m * p.out_ld + head * p.vdim + v0 + r, v * gate);
	}
}

}   // namespace

int latent_absorb_launch(const LatentArgs &p, bool queries, int dtype, cudaStream_t stream) {
	LatentArgs a = p;
	if (!queries) a.heads = 0;                         // cache rows only
	const int work = a.heads * ((a.kv_rank + AB_R - 1) / AB_R), gy = queries ? std::max(1, std::min(1024, (a.M + AB_M - 1) / AB_M)) : 1;
	const int append = a.kv_raw ? (a.M + gy * DN_WARPS - 1) / (gy * DN_WARPS) : 0;
	if (work + append == 0) return GPTQ_OK;
	const size_t smem = (size_t)AB_M * a.dim * sizeof(float);
	return dtype ? dn_launch(latent_absorb_kernel<float>, dim3(work + append, gy), dim3(DN_THREADS), smem, stream, a)
				 : dn_launch(latent_absorb_kernel<bf16>, dim3(work + append, gy), dim3(DN_THREADS), smem, stream, a);
}

bool latent_attend_ok(int kv_rank, int rot_dim) { return kv_rank <= 1024 && rot_dim <= 256; }

int latent_splits(int M, int heads, int max_seq, int dtype) {
	const int per_row = dtype ? heads : (heads + AT_HEADS - 1) / AT_HEADS;
	const int want = dn_sm_count() / std::max(1, M * per_row);
	return std::max(1, std::min(std::min(VA_SPLITS, want), (max_seq + AT_KEYS - 1) / AT_KEYS));
}

int latent_attend_launch(const LatentArgs &p, int dtype, cudaStream_t stream) {
	if (dtype) return dn_launch(latent_attend_f32_kernel, dim3(p.splits, p.heads, p.M), dim3(DN_THREADS), 0, stream, p);
	const int R = p.kv_rank + p.rot_dim;
	const size_t row = (size_t)R * 2 + 16, smem = 2 * AT_HEADS * row + (size_t)at_stages(R) * AT_KEYS * row;
	const dim3 grid(p.splits, (p.heads + AT_HEADS - 1) / AT_HEADS, p.M), block(DN_THREADS);
	if (p.kv_rank <= 64) return dn_launch(latent_attend_kernel<1>, grid, block, smem, stream, p);
	if (p.kv_rank <= 128) return dn_launch(latent_attend_kernel<2>, grid, block, smem, stream, p);
	if (p.kv_rank <= 256) return dn_launch(latent_attend_kernel<4>, grid, block, smem, stream, p);
	if (p.kv_rank <= 512) return dn_launch(latent_attend_kernel<8>, grid, block, smem, stream, p);
	return dn_launch(latent_attend_kernel<16>, grid, block, smem, stream, p);
}

int latent_value_launch(const LatentArgs &p, int dtype, cudaStream_t stream) {
	const dim3 grid((p.vdim + VA_ROWS - 1) / VA_ROWS, p.heads, p.M), block(DN_THREADS);
	const size_t smem = 2 * (size_t)p.kv_rank * sizeof(float);
	return dtype ? dn_launch(latent_value_kernel<float>, grid, block, smem, stream, p) : dn_launch(latent_value_kernel<bf16>, grid, block, smem, stream, p);
}

}   // namespace gptq
