// Shared pieces of the dense-weight library (bf16 or fp32 weights [N, K], K contiguous): element access, the row
// preparation that precedes a projection, and the epilogues that follow one.
//
// Programmatic dependent launch: every kernel here calls pdl_trigger() AFTER its own pdl_wait().  A kernel can therefore
// only start once everything two launches back has completed, and may read such data (positions, older cache rows,
// weights) ahead of its own pdl_wait(); what its direct predecessor wrote is read after it, through L2 (__ldcg), because a
// line may have been cached in L1 before the predecessor wrote it.
#pragma once

#include <utility>

#include <cuda_bf16.h>

#include "../common.cuh"
#include "../../../include/dense_b200.h"

namespace gptq {

typedef __nv_bfloat16 bf16;

constexpr int DN_THREADS = 256;
constexpr int DN_WARPS = DN_THREADS / 32;
constexpr int DN_STATUS_SLOT = DENSE_CONTROL_BYTES / 4 - 1;      // same place as in the other library's workspaces
constexpr int DN_BAD_POSITION = 4;                                // status value: position outside the tables / the cache

template <typename T> struct Elem;
template <> struct Elem<bf16> {
	static __device__ __forceinline__ float4 load4(const bf16 *p) {
		const uint2 v = __ldg(reinterpret_cast<const uint2 *>(p));
		return unpack(v);
	}
	static __device__ __forceinline__ float4 unpack(uint2 v) {
		return make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xFFFF0000u), __uint_as_float(v.y << 16), __uint_as_float(v.y & 0xFFFF0000u));
	}
	static __device__ __forceinline__ void store4(bf16 *p, float4 v) {
		__nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
		uint2 o;
		o.x = *reinterpret_cast<uint32_t *>(&a);
		o.y = *reinterpret_cast<uint32_t *>(&b);
		*reinterpret_cast<uint2 *>(p) = o;
	}
	static __device__ __forceinline__ void store8(bf16 *p, const float *v) {
		uint4 o;
		uint32_t *w = reinterpret_cast<uint32_t *>(&o);
#pragma unroll
		for (int i = 0; i < 4; ++i) {
			__nv_bfloat162 a = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
			w[i] = *reinterpret_cast<uint32_t *>(&a);
		}
		*reinterpret_cast<uint4 *>(p) = o;
	}
	static __device__ __forceinline__ float ldcg(const bf16 *p) {
		return __uint_as_float((uint32_t)__ldcg(reinterpret_cast<const unsigned short *>(p)) << 16);
	}
	static __device__ __forceinline__ float4 ldcg4(const bf16 *p) { return unpack(__ldcg(reinterpret_cast<const uint2 *>(p))); }
	static __device__ __forceinline__ float ldg(const bf16 *p) { return __uint_as_float((uint32_t)__ldg(reinterpret_cast<const unsigned short *>(p)) << 16); }
	static __device__ __forceinline__ void store(bf16 *p, float v) { *p = __float2bfloat16_rn(v); }
};
template <> struct Elem<float> {
	static __device__ __forceinline__ float4 load4(const float *p) { return __ldg(reinterpret_cast<const float4 *>(p)); }
	static __device__ __forceinline__ void store4(float *p, float4 v) { *reinterpret_cast<float4 *>(p) = v; }
	static __device__ __forceinline__ void store8(float *p, const float *v) {
		store4(p, make_float4(v[0], v[1], v[2], v[3]));
		store4(p + 4, make_float4(v[4], v[5], v[6], v[7]));
	}
	static __device__ __forceinline__ float ldcg(const float *p) { return __ldcg(p); }
	static __device__ __forceinline__ float4 ldcg4(const float *p) { return __ldcg(reinterpret_cast<const float4 *>(p)); }
	static __device__ __forceinline__ float ldg(const float *p) { return __ldg(p); }
	static __device__ __forceinline__ void store(float *p, float v) { *p = v; }
};

__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
	__nv_bfloat162 a = __floats2bfloat162_rn(lo, hi);
	return *reinterpret_cast<uint32_t *>(&a);
}

// D(16x8) += A(16x16, row) * B(16x8, col), bf16 operands; fragment ownership as in mma16816
__device__ __forceinline__ void mma16816_bf16(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
	asm volatile(
		"mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
		: "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
		: "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], uint32_t addr) {
	asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldmatrix_x2(uint32_t (&r)[2], uint32_t addr) {
	asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldmatrix_x2_trans(uint32_t (&r)[2], uint32_t addr) {
	asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(addr) : "memory");
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
	for (int d = 16; d > 0; d >>= 1) v += __shfl_xor_sync(0xffffffffu, v, d);
	return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
	for (int d = 16; d > 0; d >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, d));
	return v;
}

// Sum over the 256 threads of the CTA; `slot` (DN_WARPS floats of shared memory) must not be in use by an earlier call.
__device__ __forceinline__ float block_sum(float v, float *slot) {
	v = warp_sum(v);
	if ((threadIdx.x & 31) == 0) slot[threadIdx.x >> 5] = v;
	__syncthreads();
	float t = 0.f;
#pragma unroll
	for (int i = 0; i < DN_WARPS; ++i) t += slot[i];
	return t;
}

__device__ __forceinline__ float sigmoid_f32(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float silu_exact(float z) { return z / (1.f + expf(-z)); }
// for results that become bf16
__device__ __forceinline__ float silu_fast(float z) { return __fdividef(z, 1.f + __expf(-z)); }
// 0.5 z (1 + tanh u) with 1 + tanh u = 2 / (1 + exp(-2 u)), u = sqrt(2 / pi) (z + 0.044715 z^3)
__device__ __forceinline__ float gelu_tanh(float z) { return z / (1.f + expf(-1.5957691216057308f * fmaf(0.044715f * z, z * z, z))); }
__device__ __forceinline__ float activation(int act, float z) { return act == DENSE_ACT_GELU ? gelu_tanh(z) : silu_exact(z); }

// ---- row preparation ------------------------------------------------------------------------------------------------
// Forms row m of the residual stream and the row that the next projection reads, all in fp32:
//   x = table[token] (+ pos_table[pos])                   (start of a step), or
//   x = x_in + norm(y) * gain + shift                     (residual; norm: none, LayerNorm or RMS norm; gain and shift carry
//                                                          the norm's affine part, layer scales and residual multipliers)
//   out = x, or norm(x) * fin_w + fin_b                   (LayerNorm, RMS norm, RMS norm of equal parts)
// Rows are padded with zeros from `width` to `ld` columns.
using RowPrep = dense_rows_t;

constexpr int RP_REGS = 4;              // float4 units of a row that a thread keeps in registers
constexpr int RP_SMEM = 4 * DN_WARPS + DENSE_MAX_NORM_GROUPS;      // floats of shared memory that a preparation uses

__device__ __forceinline__ float4 add4(float4 a, float4 b) { return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w); }
__device__ __forceinline__ float rp_sqdev(float4 v, float mean, int c, int width) {
	float s = 0.f;
	const float a = v.x - mean, b = v.y - mean, d = v.z - mean, e = v.w - mean;
	if (c < width) s = fmaf(a, a, s);
	if (c + 1 < width) s = fmaf(b, b, s);
	if (c + 2 < width) s = fmaf(d, d, s);
	if (c + 3 < width) s = fmaf(e, e, s);
	return s;
}
// (v - mean) * inv * gain + shift, gain and shift optional
__device__ __forceinline__ float4 rp_affine(float4 v, float mean, float inv, const float *gain, const float *shift, int u) {
	const float4 g = gain ? __ldg(reinterpret_cast<const float4 *>(gain) + u) : make_float4(1.f, 1.f, 1.f, 1.f);
	const float4 s = shift ? __ldg(reinterpret_cast<const float4 *>(shift) + u) : make_float4(0.f, 0.f, 0.f, 0.f);
	return make_float4(fmaf((v.x - mean) * inv, g.x, s.x), fmaf((v.y - mean) * inv, g.y, s.y), fmaf((v.z - mean) * inv, g.z, s.z), fmaf((v.w - mean) * inv, g.w, s.w));
}

// The RMS norm of equal parts of row x (global memory, `width` columns): a warp sums a share of a part, the shares of a part
// are added in order.  inv: fin_groups (or DN_WARPS, if that is more) floats of shared memory.
template <typename T, typename S>
__device__ void norm_parts(const RowPrep &p, const S *x, T *dst, float *inv) {
	const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, n = p.width / p.fin_groups;
	const int shares = p.fin_groups >= DN_WARPS ? 1 : DN_WARPS / p.fin_groups;
	const bool quads = n % 4 == 0;                      // parts are whole groups of four entries (of the padded row, which is aligned)
	const int per = quads ? ((n >> 2) + shares - 1) / shares * 4 : (n + shares - 1) / shares;
	constexpr int KEEP = 8;                             // units of a share that a lane keeps in registers
	if (quads && p.fin_groups * shares == DN_WARPS && per <= KEEP * 128) {
		const int g = warp / shares, c0 = g * n + (warp - g * shares) * per, c1 = min(c0 + per, (g + 1) * n);
		float4 v[KEEP];
		float s = 0.f;
#pragma unroll
		for (int i = 0; i < KEEP; ++i) {
			const int c = c0 + 4 * (lane + 32 * i);
			v[i] = c < c1 ? Elem<S>::ldcg4(x + c) : make_float4(0.f, 0.f, 0.f, 0.f);
			s = fmaf(v[i].x, v[i].x, fmaf(v[i].y, v[i].y, fmaf(v[i].z, v[i].z, fmaf(v[i].w, v[i].w, s))));
		}
		s = warp_sum(s);
		if (shares > 1) {
			if (lane == 0) inv[warp] = s;
			__syncthreads();
			s = 0.f;
			for (int i = 0; i < shares; ++i) s += inv[g * shares + i];
		}
		const float f = 1.f / sqrtf(s / (float)n + p.eps);
#pragma unroll
		for (int i = 0; i < KEEP; ++i) {
			const int c = c0 + 4 * (lane + 32 * i);
			if (c < c1) {
				const float4 w = p.fin_w ? __ldg(reinterpret_cast<const float4 *>(p.fin_w + c)) : make_float4(1.f, 1.f, 1.f, 1.f);
				Elem<T>::store4(dst + c, make_float4(v[i].x * f * w.x, v[i].y * f * w.y, v[i].z * f * w.z, v[i].w * f * w.w));
			}
		}
		for (int c = p.width + tid; c < p.ld; c += DN_THREADS) Elem<T>::store(dst + c, 0.f);
		return;
	}
	for (int i = warp; i < p.fin_groups * shares; i += DN_WARPS) {
		const int g = i / shares, c0 = (i - g * shares) * per, c1 = min(c0 + per, n);
		float s = 0.f;
		if (quads) {
#pragma unroll 8
			for (int c = c0 + 4 * lane; c < c1; c += 128) {
				const float4 v = Elem<S>::ldcg4(x + (size_t)g * n + c);
				s = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, s))));
			}
		} else {
			for (int c = c0 + lane; c < c1; c += 32) {
				const float v = Elem<S>::ldcg(x + (size_t)g * n + c);
				s = fmaf(v, v, s);
			}
		}
		s = warp_sum(s);
		if (lane == 0) inv[i] = s;
	}
	__syncthreads();
	float f = 0.f;
	if (tid < p.fin_groups) {
		float s = 0.f;
		for (int i = 0; i < shares; ++i) s += inv[tid * shares + i];
		f = 1.f / sqrtf(s / (float)n + p.eps);
	}
	__syncthreads();
	if (tid < p.fin_groups) inv[tid] = f;
	__syncthreads();
	for (int u = tid; u < p.ld >> 2; u += DN_THREADS) {
		const float4 v = Elem<S>::ldcg4(x + 4 * u);
		const int c = 4 * u, g = min(c / n, p.fin_groups - 1), edge = (g + 1) * n;
		const float f0 = inv[g];
		float4 w = p.fin_w ? __ldg(reinterpret_cast<const float4 *>(p.fin_w) + u) : make_float4(1.f, 1.f, 1.f, 1.f);
		if (edge >= c + 4 || g == p.fin_groups - 1) {
			w.x *= f0; w.y *= f0; w.z *= f0; w.w *= f0;
		} else {                          // parts that end inside the unit (they may be shorter than one)
			auto at = [&](int i) { return inv[min((c + i) / n, p.fin_groups - 1)]; };
			w.x *= f0; w.y *= at(1); w.z *= at(2); w.w *= at(3);
		}
		Elem<T>::store4(dst + c, make_float4(v.x * w.x, v.y * w.y, v.z * w.z, v.w * w.w));
	}
}

// The whole CTA (256 threads) prepares one row.  dst: where the T row goes (global or shared memory); write_x: also store
// the new residual row.  red: RP_SMEM floats of shared memory, reused across rows (callers synchronise between rows).
template <typename T>
__device__ void prepare_row(const RowPrep &p, int m, T *dst, bool write_x, float *red) {
	const int tid = threadIdx.x, nu = p.ld >> 2;
	size_t xb = (size_t)m * p.ld, pb = 0;
	const size_t yb = xb;
	if (p.fin_groups > 1) {
		if (p.x_t) norm_parts<T, T>(p, reinterpret_cast<const T *>(p.x_in) + xb, dst, red + 4 * DN_WARPS);
		else norm_parts<T, float>(p, reinterpret_cast<const float *>(p.x_in) + xb, dst, red + 4 * DN_WARPS);
		return;
	}
	if (p.table) {
		long long t = __ldcg(reinterpret_cast<const long long *>(p.token) + m);
		if (t < 0 || t >= p.vocab) {          // never index the table out of range
			if (tid == 0) atomicExch(p.status, DN_BAD_POSITION);
			t = 0;
		}
		xb = (size_t)t * p.ld;
		if (p.pos_table) {
			int q = __ldcg(p.pos + m);
			if (q < 0 || q >= p.max_pos) {
				if (tid == 0) atomicExch(p.status, DN_BAD_POSITION);
				q = 0;
			}
			pb = (size_t)q * p.ld;
		}
	}
	auto read_x = [&](int u) {
		if (!p.table) return p.x_t ? Elem<T>::ldcg4(reinterpret_cast<const T *>(p.x_in) + xb + 4 * u) : __ldcg(reinterpret_cast<const float4 *>(reinterpret_cast<const float *>(p.x_in) + xb) + u);
		const float4 v = Elem<T>::load4(reinterpret_cast<const T *>(p.table) + xb + 4 * u);
		return p.pos_table ? add4(v, Elem<T>::load4(reinterpret_cast<const T *>(p.pos_table) + pb + 4 * u)) : v;
	};
	float4 x[RP_REGS], y[RP_REGS];
	const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
	for (int i = 0; i < RP_REGS; ++i) {
		const int u = tid + i * DN_THREADS;
		x[i] = u < nu ? read_x(u) : zero;
		y[i] = (p.y && u < nu) ? __ldcg(reinterpret_cast<const float4 *>(p.y + yb) + u) : zero;
	}
	const float inv_n = 1.f / (float)p.width;
	float mean = 0.f, inv = 1.f;
	if (p.y && p.y_norm != DENSE_NORM_NONE) {
		float s = 0.f;
		if (p.y_norm == DENSE_NORM_LAYER) {
#pragma unroll
			for (int i = 0; i < RP_REGS; ++i) s += (y[i].x + y[i].y) + (y[i].z + y[i].w);
			for (int u = tid + RP_REGS * DN_THREADS; u < nu; u += DN_THREADS) {
				const float4 v = __ldcg(reinterpret_cast<const float4 *>(p.y + yb) + u);
				s += (v.x + v.y) + (v.z + v.w);
			}
			mean = block_sum(s, red) * inv_n;
			s = 0.f;
		}
#pragma unroll
		for (int i = 0; i < RP_REGS; ++i) s += rp_sqdev(y[i], mean, 4 * (tid + i * DN_THREADS), p.width);
		for (int u = tid + RP_REGS * DN_THREADS; u < nu; u += DN_THREADS)
			s += rp_sqdev(__ldcg(reinterpret_cast<const float4 *>(p.y + yb) + u), mean, 4 * u, p.width);
		inv = 1.f / sqrtf(block_sum(s, red + DN_WARPS) * inv_n + p.eps);
	}
	auto next_x = [&](float4 xv, float4 yv, int u) { return p.y ? add4(xv, rp_affine(yv, mean, inv, p.gain, p.shift, u)) : xv; };
	const bool norm = p.fin_norm != DENSE_NORM_NONE;
#pragma unroll
	for (int i = 0; i < RP_REGS; ++i) {
		const int u = tid + i * DN_THREADS;
		if (u < nu) {
			x[i] = next_x(x[i], y[i], u);
			if (write_x) reinterpret_cast<float4 *>(p.x_out + yb)[u] = x[i];
			if (!norm) Elem<T>::store4(dst + 4 * u, x[i]);
		}
	}
	auto far_x = [&](int u) {          // units beyond the registers are formed again where they are needed
		return next_x(read_x(u), p.y ? __ldcg(reinterpret_cast<const float4 *>(p.y + yb) + u) : zero, u);
	};
	if (!norm) {
		for (int u = tid + RP_REGS * DN_THREADS; u < nu; u += DN_THREADS) {
			const float4 v = far_x(u);
			if (write_x) reinterpret_cast<float4 *>(p.x_out + yb)[u] = v;
			Elem<T>::store4(dst + 4 * u, v);
		}
		return;
	}
	// norm of the new row (x_out must not be x_in when rows are longer than the registers hold: the row is read again)
	float s = 0.f, fm = 0.f;
	if (p.fin_norm == DENSE_NORM_LAYER) {
#pragma unroll
		for (int i = 0; i < RP_REGS; ++i) s += (x[i].x + x[i].y) + (x[i].z + x[i].w);
		for (int u = tid + RP_REGS * DN_THREADS; u < nu; u += DN_THREADS) {
			const float4 v = far_x(u);
			s += (v.x + v.y) + (v.z + v.w);
		}
		fm = block_sum(s, red + 2 * DN_WARPS) * inv_n;
		s = 0.f;
	}
#pragma unroll
	for (int i = 0; i < RP_REGS; ++i) s += rp_sqdev(x[i], fm, 4 * (tid + i * DN_THREADS), p.width);
	for (int u = tid + RP_REGS * DN_THREADS; u < nu; u += DN_THREADS) s += rp_sqdev(far_x(u), fm, 4 * u, p.width);
	const float fi = 1.f / sqrtf(block_sum(s, red + 3 * DN_WARPS) * inv_n + p.eps);
	for (int i = 0, u = tid; u < nu; ++i, u += DN_THREADS) {
		float4 v;
		if (i < RP_REGS) {
			v = i == 0 ? x[0] : i == 1 ? x[1] : i == 2 ? x[2] : x[3];
		} else {
			v = far_x(u);
			if (write_x) reinterpret_cast<float4 *>(p.x_out + yb)[u] = v;
		}
		v = rp_affine(v, fm, fi, p.fin_w, p.fin_b, u);
		Elem<T>::store4(dst + 4 * u, v);
	}
}

// ---- epilogues ------------------------------------------------------------------------------------------------------
// Every fp32 result of a projection belongs to a pair of columns (n, n + 1), n even (GATED: gate column and up column).
using DenseEpi = dense_epilogue_t;

__device__ __forceinline__ int epi_pos(const DenseEpi &e, int m) {
	int pos = __ldcg(e.pos + m);
	if (pos < 0 || pos >= e.max_pos) {
		atomicExch(e.status, DN_BAD_POSITION);
		pos = 0;
	}
	return pos;
}

// row of the per-token table; a token outside it has been reported when the embedding was looked up
__device__ __forceinline__ long long epi_tab_row(const DenseEpi &e, int m) {
	const long long t = __ldcg(reinterpret_cast<const long long *>(e.tab_token) + m);
	return t < 0 || t >= e.tab_rows ? 0 : t;
}

// One pair of results of row m.  T is the activation type.
template <typename T>
__device__ __forceinline__ void epi_pair(const DenseEpi &e, int m, int n, float a, float b) {
	switch (e.mode) {
		case DENSE_EPI_F32:
		case DENSE_EPI_LOGITS:
			*reinterpret_cast<float2 *>(reinterpret_cast<float *>(e.out) + (size_t)m * e.ldo + n) = make_float2(a * e.scale, b * e.scale);
			break;
		case DENSE_EPI_T: {
			T *o = reinterpret_cast<T *>(e.out) + (size_t)m * e.ldo + n;
			Elem<T>::store(o, a);
			Elem<T>::store(o + 1, b);
			break;
		}
		case DENSE_EPI_MIXED:
			if (n < e.n_q) {
				T *o = reinterpret_cast<T *>(e.out) + (size_t)m * e.ldo + n;
				Elem<T>::store(o, a);
				Elem<T>::store(o + 1, b);
			} else {
				*reinterpret_cast<float2 *>(e.kv_out + (size_t)m * e.n_kv + (n - e.n_q)) = make_float2(a, b);
			}
			break;
		case DENSE_EPI_TABLE: {
			T *o = reinterpret_cast<T *>(e.out) + (size_t)m * e.ldo + n;
			const T *t = reinterpret_cast<const T *>(e.tab) + epi_tab_row(e, m) * e.tab_ld + e.tab_col + n;
			Elem<T>::store(o, activation(e.act, a) * Elem<T>::ldg(t));
			Elem<T>::store(o + 1, activation(e.act, b) * Elem<T>::ldg(t + 1));
			break;
		}
		case DENSE_EPI_QKV: {
			if (n < e.n_q) {
				const int off = n % e.head_dim - e.rot_at;
				if (off >= 0 && off < e.rot_dims) {
					const size_t t = (size_t)epi_pos(e, m) * (e.rot_dims >> 1) + (off >> 1);
					const float c = __ldg(e.cos_t + t), s = __ldg(e.sin_t + t);
					const float u = a * c - b * s;
					b = b * c + a * s;
					a = u;
				}
				const size_t i = (size_t)m * e.n_q + n;
				if (e.q_f32) {
					*reinterpret_cast<float2 *>(reinterpret_cast<float *>(e.q_out) + i) = make_float2(a, b);
				} else {
					*reinterpret_cast<uint32_t *>(reinterpret_cast<bf16 *>(e.q_out) + i) = pack_bf16(a, b);
				}
			} else if (n < e.n_q + e.n_kv) {
				*reinterpret_cast<float2 *>(e.kv_out + (size_t)m * e.n_kv + (n - e.n_q)) = make_float2(a, b);
			} else if (n < e.n_q + e.n_kv + e.n_gate) {
				float *g = e.gate_out + (size_t)m * e.n_gate + (n - e.n_q - e.n_kv);
				g[0] = sigmoid_f32(a);
				g[1] = sigmoid_f32(b);
			}
			break;
		}
	}
}

// Sixteen consecutive columns of row m (n a multiple of 16), as a tensor-core epilogue holds them.
template <typename T>
__device__ __forceinline__ void epi_16(const DenseEpi &e, int m, int n, const float (&v)[16]) {
	if (e.mode == DENSE_EPI_F32 || e.mode == DENSE_EPI_LOGITS) {
		float4 *o = reinterpret_cast<float4 *>(reinterpret_cast<float *>(e.out) + (size_t)m * e.ldo + n);
#pragma unroll
		for (int i = 0; i < 4; ++i) o[i] = make_float4(v[4 * i] * e.scale, v[4 * i + 1] * e.scale, v[4 * i + 2] * e.scale, v[4 * i + 3] * e.scale);
	} else if (e.mode == DENSE_EPI_MIXED && n >= e.n_q) {
		float4 *o = reinterpret_cast<float4 *>(e.kv_out + (size_t)m * e.n_kv + (n - e.n_q));
#pragma unroll
		for (int i = 0; i < 4; ++i) o[i] = make_float4(v[4 * i], v[4 * i + 1], v[4 * i + 2], v[4 * i + 3]);
	} else if (e.mode == DENSE_EPI_T || e.mode == DENSE_EPI_MIXED) {
		T *o = reinterpret_cast<T *>(e.out) + (size_t)m * e.ldo + n;
#pragma unroll
		for (int i = 0; i < 2; ++i) Elem<T>::store8(o + 8 * i, v + 8 * i);
	} else if (e.mode == DENSE_EPI_TABLE) {
		T *o = reinterpret_cast<T *>(e.out) + (size_t)m * e.ldo + n;
		const T *t = reinterpret_cast<const T *>(e.tab) + epi_tab_row(e, m) * e.tab_ld + e.tab_col + n;
		float r[16];
#pragma unroll
		for (int i = 0; i < 4; ++i) {
			const float4 f = Elem<T>::load4(t + 4 * i);
			r[4 * i] = activation(e.act, v[4 * i]) * f.x;
			r[4 * i + 1] = activation(e.act, v[4 * i + 1]) * f.y;
			r[4 * i + 2] = activation(e.act, v[4 * i + 2]) * f.z;
			r[4 * i + 3] = activation(e.act, v[4 * i + 3]) * f.w;
		}
#pragma unroll
		for (int i = 0; i < 2; ++i) Elem<T>::store8(o + 8 * i, r + 8 * i);
	} else if (e.mode == DENSE_EPI_GATED) {         // eight gate columns, then the eight up columns of the same outputs
		T *o = reinterpret_cast<T *>(e.out) + (size_t)m * e.ldo + (n >> 1);
		float r[8];
#pragma unroll
		for (int i = 0; i < 8; ++i) r[i] = activation(e.act, v[i]) * v[8 + i];
		Elem<T>::store8(o, r);
	} else {          // QKV: a group of 16 columns lies in one head, on one side of rot_at, in one section
		if (n < e.n_q) {
			const int off = n % e.head_dim - e.rot_at;
			float r[16];
			if (off >= 0 && off < e.rot_dims) {
				const size_t t = (size_t)epi_pos(e, m) * (e.rot_dims >> 1) + (off >> 1);
#pragma unroll
				for (int i = 0; i < 8; ++i) {
					const bool in = off + 2 * i < e.rot_dims;
					const float c = in ? __ldg(e.cos_t + t + i) : 1.f, s = in ? __ldg(e.sin_t + t + i) : 0.f;
					r[2 * i] = v[2 * i] * c - v[2 * i + 1] * s;
					r[2 * i + 1] = v[2 * i + 1] * c + v[2 * i] * s;
				}
			} else {
#pragma unroll
				for (int i = 0; i < 16; ++i) r[i] = v[i];
			}
			const size_t o = (size_t)m * e.n_q + n;
			if (e.q_f32) {
#pragma unroll
				for (int i = 0; i < 4; ++i)
					reinterpret_cast<float4 *>(reinterpret_cast<float *>(e.q_out) + o)[i] = make_float4(r[4 * i], r[4 * i + 1], r[4 * i + 2], r[4 * i + 3]);
			} else {
#pragma unroll
				for (int i = 0; i < 2; ++i)
					reinterpret_cast<uint4 *>(reinterpret_cast<bf16 *>(e.q_out) + o)[i] = make_uint4(pack_bf16(r[8 * i], r[8 * i + 1]), pack_bf16(r[8 * i + 2], r[8 * i + 3]),
																									pack_bf16(r[8 * i + 4], r[8 * i + 5]), pack_bf16(r[8 * i + 6], r[8 * i + 7]));
			}
		} else if (n < e.n_q + e.n_kv) {
			float4 *o = reinterpret_cast<float4 *>(e.kv_out + (size_t)m * e.n_kv + (n - e.n_q));
#pragma unroll
			for (int i = 0; i < 4; ++i) o[i] = make_float4(v[4 * i], v[4 * i + 1], v[4 * i + 2], v[4 * i + 3]);
		} else {
#pragma unroll
			for (int i = 0; i < 16; ++i) {
				const int g = n - e.n_q - e.n_kv + i;
				if (g < e.n_gate) e.gate_out[(size_t)m * e.n_gate + g] = sigmoid_f32(v[i]);
			}
		}
	}
}

// order-preserving map of a float to an unsigned key; ties go to the lower index
__device__ __forceinline__ unsigned long long argmax_key(float f, int idx) {
	const uint32_t u = __float_as_uint(f);
	const uint32_t k = (u & 0x80000000u) ? ~u : (u | 0x80000000u);
	return ((unsigned long long)k << 32) | (uint32_t)~idx;
}

struct DenseArgs {
	const void *x;                   // [M, ldx] T, when there is no row preparation
	long long ldx;
	const void *w;                   // [N, ldw] T, K columns used
	long long ldw;
	int M, K, N;
	int prep;                        // 0: x, 1: rows are prepared by the kernel
	RowPrep rp;
	DenseEpi e;
	int *status;
	float *ws;                       // scratch of a split K: [parts, M, N to 16], or NULL
	int parts;
};

// launchers (dense_skinny.cu, dense_tc.cu, dense_simt.cu)
int dense_skinny_launch(const DenseArgs &a, int dtype, cudaStream_t stream);
bool dense_skinny_ok(int M, int K, int dtype);
int dense_tc_parts(int M, int K, int N);
int dense_tc_launch(const DenseArgs &a, cudaStream_t stream);
int dense_simt_launch(const DenseArgs &a, cudaStream_t stream);

int dense_rows_launch(const RowPrep &p, int M, void *h, long long ldh, int dtype, cudaStream_t stream);

int dn_sm_count();
int dn_smem_opt_in(const void *kernel, size_t bytes);

// ---- clusters: barriers, and stores into another CTA's shared memory -------------------------------------------------------------
__device__ __forceinline__ uint32_t cluster_rank() {
	uint32_t r;
	asm volatile("mov.u32 %0, %%cluster_ctarank;" : "=r"(r));
	return r;
}
__device__ __forceinline__ void cluster_arrive() { asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory"); }
__device__ __forceinline__ void cluster_wait() { asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory"); }
__device__ __forceinline__ uint32_t cluster_map(uint32_t addr, uint32_t rank) {
	uint32_t r;
	asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(addr), "r"(rank));
	return r;
}
__device__ __forceinline__ void cluster_store2(uint32_t addr, float a, float b) {
	asm volatile("st.shared::cluster.v2.f32 [%0], {%1, %2};" ::"r"(addr), "f"(a), "f"(b) : "memory");
}

// cluster: CTAs per cluster; carveout: percentage of an SM's memory that is asked for as shared memory, or -1 (the driver's choice).
// In a chain of dependent launches an SM never falls idle, so it keeps the largest split that a kernel of the chain asked for, and the
// projections behind it lose the L1 that their loads in flight need: kernels of a decode step ask for no more than they use.
template <typename... KArgs, typename... Args>
static int dn_launch_as(int cluster, int carveout, void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream, Args &&...args) {
	if (smem > 16 * 1024)          // static shared memory comes on top (at most 32 KB)
		if (int rc = dn_smem_opt_in(reinterpret_cast<const void *>(kernel), smem)) return rc;
	cudaLaunchConfig_t cfg = {};
	cfg.gridDim = grid;
	cfg.blockDim = block;
	cfg.dynamicSmemBytes = smem;
	cfg.stream = stream;
	cudaLaunchAttribute attr[3];
	attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
	attr[0].val.programmaticStreamSerializationAllowed = 1;
	cfg.attrs = attr;
	cfg.numAttrs = 1;
	if (cluster > 1) {
		cudaLaunchAttribute &a = attr[cfg.numAttrs++];
		a.id = cudaLaunchAttributeClusterDimension;
		a.val.clusterDim.x = cluster;
		a.val.clusterDim.y = a.val.clusterDim.z = 1;
	}
	if (carveout >= 0) {
		cudaLaunchAttribute &a = attr[cfg.numAttrs++];
		a.id = cudaLaunchAttributePreferredSharedMemoryCarveout;
		a.val.sharedMemCarveout = carveout;
	}
	return cuda_status(cudaLaunchKernelEx(&cfg, kernel, std::forward<Args>(args)...));
}

template <typename... KArgs, typename... Args>
static int dn_launch(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream, Args &&...args) {
	return dn_launch_as(1, -1, kernel, grid, block, smem, stream, std::forward<Args>(args)...);
}
}   // namespace gptq
