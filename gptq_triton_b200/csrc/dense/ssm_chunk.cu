// The recurrence of ssm_scan.cu for bf16 prompts of any sizes (ssm_tc.cu takes those that fit its tiles), in chunks of 128 tokens: what a chunk adds is a few small matrix products, only
// the state goes from chunk to chunk.  With s_i the sum of a * dt over the chunk's tokens up to i (base 2),
//   ssm_chunk_state   S_c = sum_j 2^(s_last - s_j) dt_j x_j B_j^T                          per chunk and head, all at once
//   ssm_chunk_pass    state in front of every chunk: S <- 2^s_last S + S_c                 over the chunks, all entries at once
//   ssm_chunk_out     y_i = 2^s_i S C_i + sum_{j <= i} (C_i . B_j) 2^(s_i - s_j) dt_j x_j + d x_i, times silu(z_i)
// Products run on mma.m16n8k16.  x, B and C are the convolution's bf16 results; every factor that carries a decay, a step size
// or the state is fp32 and enters a product as a bf16 high part and a bf16 remainder.
#include <algorithm>

#include "ssm.cuh"

namespace gptq {

namespace {

// 2^x; underflow to zero is what a decay wants
__device__ __forceinline__ float ex2f_fast(float x) {
	float r;
	asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
	return r;
}

constexpr int SC_L = SS_CHUNK;                    // tokens per chunk
constexpr int SC_P = 64;                          // value entries per CTA
constexpr int SC_PAD = 8;                         // bf16 entries behind a staged row, against bank conflicts

struct Chunk {
	int head, p0, np, c, seq, t0, nt, g, inner;
};
__device__ __forceinline__ Chunk chunk_of(const SsmArgs &p, int chunks) {
	Chunk k;
	const int slices = (p.vdim + SC_P - 1) / SC_P;
	k.head = blockIdx.x / slices;
	k.p0 = (blockIdx.x - k.head * slices) * SC_P;
	k.np = min(SC_P, p.vdim - k.p0);
	k.c = blockIdx.y % chunks;
	k.seq = blockIdx.y / chunks;
	k.t0 = k.c * SC_L;
	k.nt = min(SC_L, p.rows_per_seq - k.t0);
	k.g = k.head / (p.heads / p.groups);
	k.inner = p.heads * p.vdim;
	return k;
}

// Step sizes of the chunk and prefix sums of a * dt * log2(e), formed in fp64 and kept in two parts (differences must stay exact behind
// tokens that decay by orders of magnitude); tokens behind the end have step size 0.  One warp.
struct Decays {
	float dt[SC_L], hi[SC_L], lo[SC_L];
	__device__ float between(int i, int j) const { return (hi[i] - hi[j]) + (lo[i] - lo[j]); }
};
__device__ __forceinline__ void chunk_decays(const SsmArgs &p, const Chunk &k, int lane, Decays &out) {
	const float bias = __ldg(p.dt_bias + k.head), a = __ldg(p.a + k.head) * 1.4426950408889634f;
	constexpr int PER = SC_L / 32;
	float dt[PER];
	double run = 0.0;
#pragma unroll
	for (int i = 0; i < PER; ++i) {
		const int t = lane * PER + i;
		dt[i] = t < k.nt ? ssm_softplus(__ldcg(p.dt + ((size_t)k.seq * p.rows_per_seq + k.t0 + t) * p.dt_ld + k.head) + bias) : 0.f;
		run += (double)(a * dt[i]);
	}
	double before = run;
#pragma unroll
	for (int d = 1; d < 32; d <<= 1) {
		const double v = __shfl_up_sync(0xffffffffu, before, d);
		if (lane >= d) before += v;
	}
	before -= run;
#pragma unroll
	for (int i = 0; i < PER; ++i) {
		before += (double)(a * dt[i]);
		const int t = lane * PER + i;
		const float hi = (float)before;
		out.dt[t] = dt[i];
		out.hi[t] = hi;
		out.lo[t] = (float)(before - (double)hi);
	}
}

// rows of `cols` bf16 entries (zero beyond `n` rows and `cols` columns, up to `width`) into shared memory; aligned rows arrive
// asynchronously (cp_async_wait)
__device__ __forceinline__ void stage_rows(bf16 *dst, int ld, const bf16 *src, size_t src_ld, int rows, int n, int cols, int width, bool vec) {
	const int units = width >> 3, step_r = DN_THREADS / units, step_c = DN_THREADS - step_r * units;
	int r = threadIdx.x / units, c = threadIdx.x - r * units;
#pragma unroll 1
	for (; r < rows; r += step_r) {
		bf16 *d = dst + (size_t)r * ld + 8 * c;
		const bf16 *s = src + (size_t)r * src_ld + 8 * c;
		if (vec && r < n && 8 * c + 8 <= cols) {
			cp_async16(d, s);
		} else {
			uint4 v = make_uint4(0u, 0u, 0u, 0u);
			if (r < n) {
				unsigned short e[8];
#pragma unroll
				for (int j = 0; j < 8; ++j) e[j] = 8 * c + j < cols ? __ldcg(reinterpret_cast<const unsigned short *>(s) + j) : (unsigned short)0;
				v = make_uint4(e[0] | (uint32_t)e[1] << 16, e[2] | (uint32_t)e[3] << 16, e[4] | (uint32_t)e[5] << 16, e[6] | (uint32_t)e[7] << 16);
			}
			*reinterpret_cast<uint4 *>(d) = v;
		}
		c += step_c;
		if (c >= units) {
			c -= units;
			++r;
		}
	}
}
__device__ __forceinline__ void split2(float a, float b, uint32_t &hi, uint32_t &lo) {
	hi = pack_bf16(a, b);
	lo = pack_bf16(a - __uint_as_float(hi << 16), b - __uint_as_float(hi & 0xFFFF0000u));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], uint32_t addr) {
	asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}

// every 16-byte unit of the x, B and C rows of a head starts on a 16-byte boundary
__host__ __device__ __forceinline__ bool sc_vec(const SsmArgs &p) { return p.vdim % 8 == 0 && p.state % 8 == 0 && p.conv_ld % 8 == 0; }

__host__ __device__ __forceinline__ int sc_round(int n, int to) { return (n + to - 1) / to * to; }

// ---- state that a chunk adds: [value entries x tokens] times [tokens x state entries] ---------------------------------------------
__global__ void __launch_bounds__(DN_THREADS, 2) ssm_chunk_state_kernel(const SsmArgs p, int chunks) {
	extern __shared__ __align__(16) unsigned char cs_smem[];
	__shared__ Decays s_d;
	const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gid = lane >> 2, tig = lane & 3;
	const Chunk k = chunk_of(p, chunks);
	const int nw = sc_round(p.state, 16), ldb = nw + SC_PAD;
	constexpr int LDX = SC_P + SC_PAD;
	bf16 *sxh = reinterpret_cast<bf16 *>(cs_smem), *sxl = sxh + SC_L * LDX, *sb = sxl + SC_L * LDX;
	const bool vec = sc_vec(p);
	pdl_wait();
	pdl_trigger();
	const bf16 *u = reinterpret_cast<const bf16 *>(p.u) + ((size_t)k.seq * p.rows_per_seq + k.t0) * p.conv_ld;
	stage_rows(sxh, LDX, u + k.head * p.vdim + k.p0, p.conv_ld, SC_L, k.nt, k.np, SC_P, vec);
	stage_rows(sb, ldb, u + k.inner + k.g * p.state, p.conv_ld, SC_L, k.nt, p.state, nw, vec);
	cp_async_commit();
	if (warp == 0) chunk_decays(p, k, lane, s_d);
	cp_async_wait<0>();
	__syncthreads();
	for (int i = tid; i < SC_L * SC_P / 2; i += DN_THREADS) {          // inputs times decay to the chunk's end and step size
		const int t = i / (SC_P / 2), c = (i - t * (SC_P / 2)) * 2;
		uint32_t *h = reinterpret_cast<uint32_t *>(sxh + t * LDX + c);
		const uint32_t v = *h;
		const float f = ex2f_fast(s_d.between(SC_L - 1, t)) * s_d.dt[t];
		uint32_t hi, lo;
		split2(__uint_as_float(v << 16) * f, __uint_as_float(v & 0xFFFF0000u) * f, hi, lo);
		*h = hi;
		*reinterpret_cast<uint32_t *>(sxl + t * LDX + c) = lo;
	}
	__syncthreads();
	if (tid == 0 && k.p0 == 0) p.chunk_decay[((size_t)k.seq * chunks + k.c) * p.heads + k.head] = ex2f_fast(s_d.hi[SC_L - 1] + s_d.lo[SC_L - 1]);
	// warp: 16 value entries, half of the state entries in passes of 32
	const int pr = (warp & 3) * 16, hw = sc_round(nw / 2, 16), n_lo = (warp >> 2) * hw, n_hi = min(n_lo + hw, nw);
	if (pr >= k.np) return;
	float *dst = p.chunk_s + (((size_t)k.seq * chunks + k.c) * p.heads + k.head) * p.vdim * p.state + (size_t)k.p0 * p.state;
	// A 16 x 16 from rows of tokens (transposed): matrices (rows 0-7, k 0-7), (rows 8-15, k 0-7), (rows 0-7, k 8-15), (rows 8-15, k 8-15)
	const uint32_t a_off = (uint32_t)(((lane >> 4) * 8 + (lane & 7)) * LDX + pr + ((lane >> 3) & 1) * 8) * 2;
	// B 16 x 16 from rows of tokens (transposed): (k 0-7, n 0-7), (k 8-15, n 0-7), (k 0-7, n 8-15), (k 8-15, n 8-15)
	const uint32_t b_off = (uint32_t)((lane & 15) * ldb + (lane >> 4) * 8) * 2;
	const int ksteps = (k.nt + 15) >> 4;
	for (int n0 = n_lo; n0 < n_hi; n0 += 32) {
		float acc[4][4] = {};
		const bool two = n0 + 16 < n_hi;
#pragma unroll 2
		for (int s = 0; s < ksteps; ++s) {
			uint32_t ah[4], al[4], b[4];
			ldmatrix_x4_trans(ah, smem_u32(sxh) + a_off + s * 16 * LDX * 2);
			ldmatrix_x4_trans(al, smem_u32(sxl) + a_off + s * 16 * LDX * 2);
#pragma unroll
			for (int h = 0; h < 2; ++h) {
				if (h && !two) break;
				ldmatrix_x4_trans(b, smem_u32(sb) + b_off + (s * 16 * ldb + n0 + 16 * h) * 2);
#pragma unroll
				for (int q = 0; q < 2; ++q) {
					mma16816_bf16(acc[2 * h + q], ah[0], ah[1], ah[2], ah[3], b[2 * q], b[2 * q + 1]);
					mma16816_bf16(acc[2 * h + q], al[0], al[1], al[2], al[3], b[2 * q], b[2 * q + 1]);
				}
			}
		}
#pragma unroll
		for (int q = 0; q < 4; ++q) {
#pragma unroll
			for (int e = 0; e < 4; ++e) {
				const int r = pr + gid + 8 * (e >> 1), n = n0 + 8 * q + 2 * tig + (e & 1);
				if (r < k.np && n < n_hi && n < p.state) dst[(size_t)r * p.state + n] = acc[q][e];
			}
		}
	}
}

// ---- the state from chunk to chunk; chunk_s becomes the state in front of every chunk ---------------------------------------------
__global__ void __launch_bounds__(DN_THREADS) ssm_chunk_pass_kernel(const SsmArgs p, int chunks) {
	const int per = p.vdim * p.state, i = blockIdx.x * DN_THREADS + threadIdx.x, head = blockIdx.y, seq = blockIdx.z;
	pdl_wait();
	pdl_trigger();
	if (i >= per) return;
	const int start = __ldcg(p.pos + (size_t)seq * p.rows_per_seq);
	float *s = p.s + ((size_t)seq * p.heads + head) * per + i;
	float *cs = p.chunk_s + ((size_t)seq * chunks * p.heads + head) * per + i;
	const float *cd = p.chunk_decay + (size_t)seq * chunks * p.heads + head;
	float run = start > 0 ? __ldcg(s) : 0.f;
	constexpr int U = 8;
	for (int c0 = 0; c0 < chunks; c0 += U) {
		float v[U], d[U];
#pragma unroll
		for (int j = 0; j < U; ++j) {
			v[j] = c0 + j < chunks ? __ldcg(cs + (size_t)(c0 + j) * p.heads * per) : 0.f;
			d[j] = c0 + j < chunks ? __ldcg(cd + (size_t)(c0 + j) * p.heads) : 0.f;
		}
#pragma unroll
		for (int j = 0; j < U; ++j)
			if (c0 + j < chunks) {
				cs[(size_t)(c0 + j) * p.heads * per] = run;
				run = fmaf(d[j], run, v[j]);
			}
	}
	*s = run;
}

// ---- outputs: a warp per 16 tokens -----------------------------------------------------------------------------------------------
template <int NK>                        // 16-entry steps of the state: state <= 16 * NK
__global__ void __launch_bounds__(DN_THREADS, NK > 8 ? 1 : 2) ssm_chunk_out_kernel(const SsmArgs p, int chunks) {
	extern __shared__ __align__(16) unsigned char co_smem[];
	__shared__ Decays s_d;
	const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gid = lane >> 2, tig = lane & 3;
	const Chunk k = chunk_of(p, chunks);
	const int nw = sc_round(p.state, 16), nk = nw >> 4, ldb = nw + SC_PAD, pw = sc_round(k.np, 16);
	constexpr int LDX = SC_P + SC_PAD;
	bf16 *sb = reinterpret_cast<bf16 *>(co_smem), *sx = sb + SC_L * ldb, *ssh = sx + SC_L * LDX, *ssl = ssh + SC_P * ldb;
	const bool vec = sc_vec(p);
	pdl_wait();
	pdl_trigger();
	const size_t row0 = (size_t)k.seq * p.rows_per_seq + k.t0;
	const bf16 *u = reinterpret_cast<const bf16 *>(p.u) + row0 * p.conv_ld, *raw = reinterpret_cast<const bf16 *>(p.raw) + row0 * p.raw_ld;
	stage_rows(sb, ldb, u + k.inner + k.g * p.state, p.conv_ld, SC_L, k.nt, p.state, nw, vec);
	stage_rows(sx, LDX, u + k.head * p.vdim + k.p0, p.conv_ld, SC_L, k.nt, k.np, SC_P, vec);
	cp_async_commit();
	// C of this warp's 16 tokens, as A fragments
	const int r0 = warp * 16;
	uint32_t cf[NK][4];
	const bf16 *cg = u + k.inner + (p.groups + k.g) * p.state;
#pragma unroll
	for (int s = 0; s < NK; ++s)
#pragma unroll
		for (int e = 0; e < 4; ++e) {
			const int t = r0 + gid + 8 * (e & 1), n = 16 * s + 2 * tig + 8 * (e >> 1);
			cf[s][e] = 0u;
			if (t < k.nt) {
				const unsigned short *src = reinterpret_cast<const unsigned short *>(cg + (size_t)t * p.conv_ld + n);
				if (vec && n + 1 < p.state) cf[s][e] = __ldcg(reinterpret_cast<const uint32_t *>(src));
				else cf[s][e] = (n < p.state ? (uint32_t)__ldcg(src) : 0u) | (n + 1 < p.state ? (uint32_t)__ldcg(src + 1) << 16 : 0u);
			}
		}
	if (warp == 0) chunk_decays(p, k, lane, s_d);
	// state in front of the chunk, in two parts; eight requests of a thread at a time
	const float *prev = p.chunk_s + (((size_t)k.seq * chunks + k.c) * p.heads + k.head) * p.vdim * p.state + (size_t)k.p0 * p.state;
	auto put = [&](int r, int n, float a, float b) {
		uint32_t hi, lo;
		split2(a, b, hi, lo);
		*reinterpret_cast<uint32_t *>(ssh + r * ldb + n) = hi;
		*reinterpret_cast<uint32_t *>(ssl + r * ldb + n) = lo;
	};
	if (p.state % 16 == 0) {                          // rows without padding, consecutive in memory
		const int quads = p.state >> 2, all = k.np * quads;
		for (int i0 = tid; i0 < all; i0 += 8 * DN_THREADS) {
			float4 v[8];
#pragma unroll
			for (int j = 0; j < 8; ++j)
				if (i0 + j * DN_THREADS < all) v[j] = __ldcg(reinterpret_cast<const float4 *>(prev) + i0 + j * DN_THREADS);
#pragma unroll
			for (int j = 0; j < 8; ++j) {
				const int i = i0 + j * DN_THREADS, r = i / quads, n = (i - r * quads) * 4;
				if (i < all) {
					put(r, n, v[j].x, v[j].y);
					put(r, n + 2, v[j].z, v[j].w);
				}
			}
		}
		for (int i = tid; i < (pw - k.np) * (nw / 2); i += DN_THREADS) put(k.np + i / (nw / 2), i % (nw / 2) * 2, 0.f, 0.f);
	} else {
		for (int i = tid; i < pw * (nw / 2); i += DN_THREADS) {
			const int r = i / (nw / 2), n = (i - r * (nw / 2)) * 2;
			put(r, n, r < k.np && n < p.state ? __ldcg(prev + (size_t)r * p.state + n) : 0.f, r < k.np && n + 1 < p.state ? __ldcg(prev + (size_t)r * p.state + n + 1) : 0.f);
		}
	}
	cp_async_wait<0>();
	__syncthreads();
	float acc[SC_P / 8][4];
#pragma unroll
	for (int q = 0; q < SC_P / 8; ++q) acc[q][0] = acc[q][1] = acc[q][2] = acc[q][3] = 0.f;
	const int i0 = r0 + gid, i1 = i0 + 8;
	if (r0 < k.nt) {
		// ---- from the state: rows of S are value entries, columns state entries ----
		const uint32_t s_off = (uint32_t)(((lane >> 4) * 8 + (lane & 7)) * ldb + ((lane >> 3) & 1) * 8) * 2;      // two 8-row groups x two 8-column halves
#pragma unroll
		for (int s = 0; s < NK; ++s) {
			if (s >= nk) break;
#pragma unroll
			for (int q = 0; q < SC_P / 16; ++q) {
				if (16 * q >= k.np) break;
				uint32_t h[4], l[4];
				ldmatrix_x4(h, smem_u32(ssh) + s_off + (q * 16 * ldb + s * 16) * 2);
				ldmatrix_x4(l, smem_u32(ssl) + s_off + (q * 16 * ldb + s * 16) * 2);
#pragma unroll
				for (int e = 0; e < 2; ++e) {
					mma16816_bf16(acc[2 * q + e], cf[s][0], cf[s][1], cf[s][2], cf[s][3], h[2 * e], h[2 * e + 1]);
					mma16816_bf16(acc[2 * q + e], cf[s][0], cf[s][1], cf[s][2], cf[s][3], l[2 * e], l[2 * e + 1]);
				}
			}
		}
		const float e0 = ex2f_fast(s_d.hi[i0] + s_d.lo[i0]), e1 = ex2f_fast(s_d.hi[i1] + s_d.lo[i1]);
#pragma unroll
		for (int q = 0; q < SC_P / 8; ++q) {
			acc[q][0] *= e0;
			acc[q][1] *= e0;
			acc[q][2] *= e1;
			acc[q][3] *= e1;
		}
		// ---- from the chunk's own tokens, 16 at a time up to the diagonal ----
		const uint32_t b_off = (uint32_t)(((lane >> 4) * 8 + (lane & 7)) * ldb + ((lane >> 3) & 1) * 8) * 2;
		const uint32_t x_off = (uint32_t)((lane & 15) * LDX + (lane >> 4) * 8) * 2;
#pragma unroll 1
		for (int j0 = 0; j0 <= r0; j0 += 16) {
			float gm[2][4] = {};
#pragma unroll
			for (int s = 0; s < NK; ++s) {
				if (s >= nk) break;
				uint32_t b[4];
				ldmatrix_x4(b, smem_u32(sb) + b_off + (j0 * ldb + s * 16) * 2);
				mma16816_bf16(gm[0], cf[s][0], cf[s][1], cf[s][2], cf[s][3], b[0], b[1]);
				mma16816_bf16(gm[1], cf[s][0], cf[s][1], cf[s][2], cf[s][3], b[2], b[3]);
			}
#pragma unroll
			for (int h = 0; h < 2; ++h)
#pragma unroll
				for (int e = 0; e < 4; ++e) {
					const int j = j0 + 8 * h + 2 * tig + (e & 1), i = r0 + gid + 8 * (e >> 1);
					gm[h][e] = j <= i ? gm[h][e] * ex2f_fast(s_d.between(i, j)) * s_d.dt[j] : 0.f;
				}
			uint32_t ah[4], al[4];               // accumulator layout = A fragment layout, two 8-column tiles side by side
			split2(gm[0][0], gm[0][1], ah[0], al[0]);
			split2(gm[0][2], gm[0][3], ah[1], al[1]);
			split2(gm[1][0], gm[1][1], ah[2], al[2]);
			split2(gm[1][2], gm[1][3], ah[3], al[3]);
#pragma unroll
			for (int q = 0; q < SC_P / 16; ++q) {
				if (16 * q >= k.np) break;
				uint32_t x[4];
				ldmatrix_x4_trans(x, smem_u32(sx) + x_off + (j0 * LDX + q * 16) * 2);
#pragma unroll
				for (int e = 0; e < 2; ++e) {
					mma16816_bf16(acc[2 * q + e], ah[0], ah[1], ah[2], ah[3], x[2 * e], x[2 * e + 1]);
					mma16816_bf16(acc[2 * q + e], al[0], al[1], al[2], al[3], x[2 * e], x[2 * e + 1]);
				}
			}
		}
		// ---- skip, gate, store ----
		const float d = __ldg(p.d + k.head);
#pragma unroll
		for (int q = 0; q < SC_P / 8; ++q) {
#pragma unroll
			for (int h = 0; h < 2; ++h) {
				const int t = r0 + gid + 8 * h, c = 8 * q + 2 * tig;
				if (t < k.nt && c < k.np) {
					const int col = k.head * p.vdim + k.p0 + c;
					const bf16 *x = sx + t * LDX + c, *z = raw + (size_t)t * p.raw_ld + p.z_at + col;
					bf16 *o = reinterpret_cast<bf16 *>(p.out) + (row0 + t) * p.out_ld + col;
					if (vec) {                       // even columns: both entries are there
						const uint32_t xv = *reinterpret_cast<const uint32_t *>(x), zv = __ldcg(reinterpret_cast<const uint32_t *>(z));
						*reinterpret_cast<uint32_t *>(o) = pack_bf16(fmaf(d, __uint_as_float(xv << 16), acc[q][2 * h]) * silu_fast(__uint_as_float(zv << 16)),
																 fmaf(d, __uint_as_float(xv & 0xFFFF0000u), acc[q][2 * h + 1]) * silu_fast(__uint_as_float(zv & 0xFFFF0000u)));
					} else {
						Elem<bf16>::store(o, fmaf(d, __bfloat162float(x[0]), acc[q][2 * h]) * silu_fast(Elem<bf16>::ldcg(z)));
						if (c + 1 < k.np) Elem<bf16>::store(o + 1, fmaf(d, __bfloat162float(x[1]), acc[q][2 * h + 1]) * silu_fast(Elem<bf16>::ldcg(z + 1)));
					}
				}
			}
		}
	}
	// ---- the convolution's last inputs, by the CTAs of the last chunk ----
	if (k.c == chunks - 1) {
		const int T = p.rows_per_seq, last = min(T, p.taps), start = __ldcg(p.pos + (size_t)k.seq * T);
		const bool shared = k.p0 == 0 && k.head % (p.heads / p.groups) == 0;
		const int count = k.np + (shared ? 2 * p.state : 0);
		const bf16 *in = reinterpret_cast<const bf16 *>(p.raw) + (size_t)k.seq * T * p.raw_ld + p.conv_at;
		float *ring = p.ring + (size_t)k.seq * p.taps * p.conv_ld;
		for (int i = tid; i < last * count; i += DN_THREADS) {
			const int t = T - last + i / count, e = i % count;
			const int c = e < k.np ? k.head * p.vdim + k.p0 + e : e < k.np + p.state ? k.inner + k.g * p.state + e - k.np : k.inner + (p.groups + k.g) * p.state + e - k.np - p.state;
			ring[(size_t)((start + t) % p.taps) * p.conv_ld + c] = Elem<bf16>::ldcg(in + (size_t)t * p.raw_ld + c);
		}
	}
}

}   // namespace

int ssm_chunk_launch(const SsmArgs &p, cudaStream_t stream) {
	const int T = p.rows_per_seq, seqs = p.M / T, chunks = (T + SC_L - 1) / SC_L, slices = (p.vdim + SC_P - 1) / SC_P;
	const int ldb = sc_round(p.state, 16) + SC_PAD, ldx = SC_P + SC_PAD;
	const dim3 grid(p.heads * slices, chunks * seqs), block(DN_THREADS);
	const size_t smem_s = (size_t)SC_L * (2 * ldx + ldb) * 2, smem_o = ((size_t)SC_L * (ldb + ldx) + 2 * (size_t)SC_P * ldb) * 2;
	if (int rc = dn_launch(ssm_chunk_state_kernel, grid, block, smem_s, stream, p, chunks)) return rc;
	const int per = p.vdim * p.state;
	if (int rc = dn_launch(ssm_chunk_pass_kernel, dim3((per + DN_THREADS - 1) / DN_THREADS, p.heads, seqs), block, 0, stream, p, chunks)) return rc;
	if (p.state <= 32) return dn_launch(ssm_chunk_out_kernel<2>, grid, block, smem_o, stream, p, chunks);
	if (p.state <= 64) return dn_launch(ssm_chunk_out_kernel<4>, grid, block, smem_o, stream, p, chunks);
	if (p.state <= 128) return dn_launch(ssm_chunk_out_kernel<8>, grid, block, smem_o, stream, p, chunks);
	return dn_launch(ssm_chunk_out_kernel<16>, grid, block, smem_o, stream, p, chunks);
}

}   // namespace gptq
