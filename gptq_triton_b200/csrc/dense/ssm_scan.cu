// Selective state-space recurrence (Mamba-2) token by token, fp32 throughout: decode steps and portions of any length.  (Longer
// bf16 portions run in chunks, ssm_chunk.cu, behind the same convolution.)
//
//   ssm_step   one token per sequence: convolution, state update, output and gate in one kernel
//   ssm_conv   portions: convolution and silu of all channels
//   ssm_scan   portions: the recurrence over the tokens, in blocks that are staged in shared memory
// A CTA owns 32 value entries of one head: a warp holds four rows of the state (a row: one value entry, all N state entries
// across the lanes) in registers from the first token to the last.  The convolution's last inputs live in a ring with the slot
// position mod taps, so that a step writes a slot that no CTA of the same launch reads; a portion's ring entries are written by the
// scan, behind the convolution that reads the old ones.  What lies before position 0 counts as zero, whatever the buffers hold.
#include <algorithm>

#include "ssm.cuh"

namespace gptq {

namespace {

constexpr int SS_RW = 4;                          // state rows per warp
constexpr int SS_PV = SS_RW * DN_WARPS;           // value entries per CTA
constexpr int SS_TB = 16;                         // tokens per staged block

struct Slice {                                    // channels that a CTA works on, in the order [x slice | B | C]
	int x0, nx, b0, c0, N;
	__device__ int count() const { return nx + 2 * N; }
	__device__ int channel(int i) const { return i < nx ? x0 + i : i < nx + N ? b0 + i - nx : c0 + i - nx - N; }
};
__device__ __forceinline__ Slice slice_of(const SsmArgs &p, int head, int p0) {
	const int inner = p.heads * p.vdim, g = head / (p.heads / p.groups);
	return {head * p.vdim + p0, min(SS_PV, p.vdim - p0), inner + g * p.state, inner + (p.groups + g) * p.state, p.state};
}
// every channel's ring entry has one writer: the x channels their CTA, B and C the first slice of the first head of their group
__device__ __forceinline__ bool writes_ring(const SsmArgs &p, const Slice &s, int i, int head, int p0) {
	return i < s.nx || (p0 == 0 && head % (p.heads / p.groups) == 0);
}

template <int NI>
struct State {                                    // rows p0 + warp * SS_RW + r, entries lane + 32 i
	float v[SS_RW][NI];
	__device__ void load(const float *s, int row0, int rows, int N, int lane, bool zero) {
#pragma unroll
		for (int r = 0; r < SS_RW; ++r)
#pragma unroll
			for (int i = 0; i < NI; ++i) {
				const int n = lane + 32 * i;
				v[r][i] = !zero && row0 + r < rows && n < N ? __ldcg(s + (size_t)(row0 + r) * N + n) : 0.f;
			}
	}
	__device__ void store(float *s, int row0, int rows, int N, int lane) const {
#pragma unroll
		for (int r = 0; r < SS_RW; ++r)
#pragma unroll
			for (int i = 0; i < NI; ++i) {
				const int n = lane + 32 * i;
				if (row0 + r < rows && n < N) s[(size_t)(row0 + r) * N + n] = v[r][i];
			}
	}
	// one token; returns the outputs of the warp's rows (all lanes)
	__device__ void step(const float *x, const float *b, const float *c, float dt, float decay, int N, int lane, float (&y)[SS_RW]) {
		float bn[NI], cn[NI];
#pragma unroll
		for (int i = 0; i < NI; ++i) {
			const int n = lane + 32 * i;
			bn[i] = n < N ? b[n] : 0.f;
			cn[i] = n < N ? c[n] : 0.f;
		}
#pragma unroll
		for (int r = 0; r < SS_RW; ++r) {
			const float dx = dt * x[r];
			y[r] = 0.f;
#pragma unroll
			for (int i = 0; i < NI; ++i) {
				v[r][i] = fmaf(decay, v[r][i], dx * bn[i]);
				y[r] = fmaf(v[r][i], cn[i], y[r]);
			}
		}
#pragma unroll
		for (int r = 0; r < SS_RW; ++r) y[r] = warp_sum(y[r]);
	}
};

__device__ __forceinline__ bool bad_position(const SsmArgs &p, int pos) {
	if (pos >= 0) return false;
	if (threadIdx.x == 0) atomicExch(p.status, DN_BAD_POSITION);
	return true;
}

template <int NI>
__global__ void __launch_bounds__(DN_THREADS) ssm_step_kernel(const SsmArgs p) {
	constexpr int CH = (SS_PV + 2 * 32 * NI + DN_THREADS - 1) / DN_THREADS;
	__shared__ float s_u[SS_PV + 2 * 32 * NI];
	const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
	const int head = blockIdx.y, p0 = blockIdx.x * SS_PV, m = blockIdx.z;
	const Slice sl = slice_of(p, head, p0);
	const int pos = __ldcg(p.pos + m);            // older than the previous launch, like the state and the ring
	float *ring = p.ring + (size_t)m * p.taps * p.conv_ld;
	float *s = p.s + ((size_t)m * p.heads + head) * p.vdim * p.state;
	State<NI> st;
	st.load(s, p0 + warp * SS_RW, p.vdim, p.state, lane, pos <= 0);
	float u[CH], w_now[CH];
#pragma unroll
	for (int j = 0; j < CH; ++j) {
		const int i = tid + j * DN_THREADS;
		u[j] = w_now[j] = 0.f;
		if (i < sl.count()) {
			const int c = sl.channel(i);
			u[j] = __ldg(p.conv_b + c);
			w_now[j] = __ldg(p.conv_w + (size_t)(p.taps - 1) * p.conv_ld + c);
			for (int k = p.taps - 1; k > 0; --k)
				if (pos - k >= 0) u[j] = fmaf(__ldg(p.conv_w + (size_t)(p.taps - 1 - k) * p.conv_ld + c), __ldcg(ring + (size_t)((pos - k) % p.taps) * p.conv_ld + c), u[j]);
		}
	}
	const float bias = __ldg(p.dt_bias + head), a = __ldg(p.a + head), d = __ldg(p.d + head);
	pdl_wait();
	pdl_trigger();
	if (bad_position(p, pos)) return;
	const float *raw = reinterpret_cast<const float *>(p.raw) + (size_t)m * p.raw_ld;
	const float dt_raw = __ldcg(p.dt + (size_t)m * p.dt_ld + head);
	const int row = p0 + warp * SS_RW + lane;     // lanes below SS_RW finish a row
	const float z = lane < SS_RW && row < p.vdim ? __ldcg(raw + p.z_at + head * p.vdim + row) : 0.f;
#pragma unroll
	for (int j = 0; j < CH; ++j) {
		const int i = tid + j * DN_THREADS;
		if (i < sl.count()) {
			const int c = sl.channel(i);
			const float in = __ldcg(raw + p.conv_at + c);
			s_u[i] = silu_exact(fmaf(w_now[j], in, u[j]));
			if (writes_ring(p, sl, i, head, p0)) ring[(size_t)(pos % p.taps) * p.conv_ld + c] = in;
		}
	}
	__syncthreads();
	const float dt = ssm_softplus(dt_raw + bias), decay = expf(a * dt);
	float x[SS_RW], y[SS_RW];
#pragma unroll
	for (int r = 0; r < SS_RW; ++r) x[r] = warp * SS_RW + r < sl.nx ? s_u[warp * SS_RW + r] : 0.f;
	st.step(x, s_u + sl.nx, s_u + sl.nx + sl.N, dt, decay, p.state, lane, y);
	st.store(s, p0 + warp * SS_RW, p.vdim, p.state, lane);
#pragma unroll
	for (int r = 0; r < SS_RW; ++r)
		if (lane == r && row < p.vdim) reinterpret_cast<float *>(p.out)[(size_t)m * p.out_ld + head * p.vdim + row] = fmaf(d, x[r], y[r]) * silu_exact(z);
}

template <typename T> __device__ __forceinline__ float2 load2(const T *p);
template <> __device__ __forceinline__ float2 load2<float>(const float *p) { return __ldcg(reinterpret_cast<const float2 *>(p)); }
template <> __device__ __forceinline__ float2 load2<bf16>(const bf16 *p) {
	const uint32_t v = __ldcg(reinterpret_cast<const uint32_t *>(p));
	return make_float2(__uint_as_float(v << 16), __uint_as_float(v & 0xFFFF0000u));
}
__device__ __forceinline__ void store2(float *p, float2 v) { *reinterpret_cast<float2 *>(p) = v; }
__device__ __forceinline__ void store2(bf16 *p, float2 v) { *reinterpret_cast<uint32_t *>(p) = pack_bf16(v.x, v.y); }

// thread per pair of channels, a window of W >= taps inputs in registers over a block of tokens
template <typename T, int W>
__global__ void __launch_bounds__(DN_THREADS) ssm_conv_kernel(const SsmArgs p, int block) {
	constexpr int U = 8;                          // tokens whose inputs are requested together
	const int c = (blockIdx.x * DN_THREADS + threadIdx.x) * 2, t0 = blockIdx.y * block, seq = blockIdx.z, n = p.rows_per_seq;
	if (c >= p.heads * p.vdim + 2 * p.groups * p.state) return;          // (rows are padded to an even number)
	const float2 zero = make_float2(0.f, 0.f);
	float2 w[W], in[W];                           // in[W - 1]: the current token
#pragma unroll
	for (int k = 0; k < W; ++k) w[k] = W - 1 - k < p.taps ? __ldg(reinterpret_cast<const float2 *>(p.conv_w + (size_t)(p.taps - W + k) * p.conv_ld + c)) : zero;
	const float2 b = __ldg(reinterpret_cast<const float2 *>(p.conv_b + c));
	pdl_wait();
	pdl_trigger();
	const int start = __ldcg(p.pos + (size_t)seq * n);
	if (start < 0) {
		atomicExch(p.status, DN_BAD_POSITION);
		return;
	}
	const T *raw = reinterpret_cast<const T *>(p.raw) + (size_t)seq * n * p.raw_ld + p.conv_at + c;
	T *u = reinterpret_cast<T *>(p.u) + (size_t)seq * n * p.conv_ld + c;
	auto input = [&](int t) {                     // of this portion, of the ring, or zero before the sequence
		if (t >= 0) return load2<T>(raw + (size_t)t * p.raw_ld);
		return start + t >= 0 ? load2<float>(p.ring + ((size_t)seq * p.taps + (start + t) % p.taps) * p.conv_ld + c) : zero;
	};
#pragma unroll
	for (int k = 0; k < W - 1; ++k) in[k + 1] = W - 1 - k < p.taps ? input(t0 + k - (W - 1)) : zero;
	const int t1 = min(t0 + block, n);
	for (int t = t0; t < t1; t += U) {
		float2 next[U];
#pragma unroll
		for (int j = 0; j < U; ++j) next[j] = t + j < t1 ? load2<T>(raw + (size_t)(t + j) * p.raw_ld) : zero;
#pragma unroll
		for (int j = 0; j < U; ++j) {
#pragma unroll
			for (int k = 0; k < W - 1; ++k) in[k] = in[k + 1];
			in[W - 1] = next[j];
			float2 v = b;
#pragma unroll
			for (int k = 0; k < W; ++k) {
				v.x = fmaf(w[k].x, in[k].x, v.x);
				v.y = fmaf(w[k].y, in[k].y, v.y);
			}
			if (t + j < t1) store2(u + (size_t)(t + j) * p.conv_ld, sizeof(T) == 2 ? make_float2(silu_fast(v.x), silu_fast(v.y)) : make_float2(silu_exact(v.x), silu_exact(v.y)));
		}
	}
}

template <int NI>
__global__ void __launch_bounds__(DN_THREADS) ssm_scan_kernel(const SsmArgs p) {
	__shared__ float s_u[SS_TB][SS_PV + 2 * 32 * NI], s_z[SS_TB][SS_PV], s_dt[SS_TB], s_decay[SS_TB];
	const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
	const int head = blockIdx.y, p0 = blockIdx.x * SS_PV, seq = blockIdx.z, T = p.rows_per_seq;
	const Slice sl = slice_of(p, head, p0);
	const float bias = __ldg(p.dt_bias + head), a = __ldg(p.a + head), d = __ldg(p.d + head);
	float *s = p.s + ((size_t)seq * p.heads + head) * p.vdim * p.state;
	pdl_wait();
	pdl_trigger();
	const int start = __ldcg(p.pos + (size_t)seq * T);
	if (bad_position(p, start)) return;
	State<NI> st;
	st.load(s, p0 + warp * SS_RW, p.vdim, p.state, lane, start == 0);
	const float *raw = reinterpret_cast<const float *>(p.raw) + (size_t)seq * T * p.raw_ld, *u = reinterpret_cast<const float *>(p.u) + (size_t)seq * T * p.conv_ld;
	const int row = p0 + warp * SS_RW + lane;
	for (int t0 = 0; t0 < T; t0 += SS_TB) {
		const int nt = min(SS_TB, T - t0), n = sl.count();
		__syncthreads();
		for (int i = tid; i < nt * n; i += DN_THREADS) {
			const int t = i / n, k = i - t * n;
			s_u[t][k] = __ldcg(u + (size_t)(t0 + t) * p.conv_ld + sl.channel(k));
		}
		for (int i = tid; i < nt * sl.nx; i += DN_THREADS) {
			const int t = i / sl.nx, k = i - t * sl.nx;
			s_z[t][k] = silu_exact(__ldcg(raw + (size_t)(t0 + t) * p.raw_ld + p.z_at + sl.x0 + k));
		}
		if (tid < nt) {
			const float dt = ssm_softplus(__ldcg(p.dt + ((size_t)seq * T + t0 + tid) * p.dt_ld + head) + bias);
			s_dt[tid] = dt;
			s_decay[tid] = expf(a * dt);
		}
		__syncthreads();
		for (int t = 0; t < nt; ++t) {
			float x[SS_RW], y[SS_RW];
#pragma unroll
			for (int r = 0; r < SS_RW; ++r) x[r] = warp * SS_RW + r < sl.nx ? s_u[t][warp * SS_RW + r] : 0.f;
			st.step(x, &s_u[t][sl.nx], &s_u[t][sl.nx + sl.N], s_dt[t], s_decay[t], p.state, lane, y);
#pragma unroll
			for (int r = 0; r < SS_RW; ++r)
				if (lane == r && row < p.vdim) reinterpret_cast<float *>(p.out)[((size_t)seq * T + t0 + t) * p.out_ld + head * p.vdim + row] = fmaf(d, x[r], y[r]) * s_z[t][warp * SS_RW + r];
		}
	}
	st.store(s, p0 + warp * SS_RW, p.vdim, p.state, lane);
	float *ring = p.ring + (size_t)seq * p.taps * p.conv_ld;
	const int last = min(T, p.taps);
	for (int i = tid; i < last * sl.count(); i += DN_THREADS) {
		const int t = T - last + i / sl.count(), k = i % sl.count(), c = sl.channel(k);
		if (writes_ring(p, sl, k, head, p0)) ring[(size_t)((start + t) % p.taps) * p.conv_ld + c] = __ldcg(raw + (size_t)t * p.raw_ld + p.conv_at + c);
	}
}

}   // namespace

int ssm_step_launch(const SsmArgs &p, cudaStream_t stream) {
	const dim3 grid((p.vdim + SS_PV - 1) / SS_PV, p.heads, p.M), block(DN_THREADS);
	if (p.state <= 32) return dn_launch(ssm_step_kernel<1>, grid, block, 0, stream, p);
	if (p.state <= 64) return dn_launch(ssm_step_kernel<2>, grid, block, 0, stream, p);
	if (p.state <= 128) return dn_launch(ssm_step_kernel<4>, grid, block, 0, stream, p);
	return dn_launch(ssm_step_kernel<8>, grid, block, 0, stream, p);
}

template <typename T>
static int conv_launch(const SsmArgs &p, cudaStream_t stream) {
	const int pairs = (p.heads * p.vdim + 2 * p.groups * p.state + 1) / 2, cb = (pairs + DN_THREADS - 1) / DN_THREADS, seqs = p.M / p.rows_per_seq;
	int block = 64;                               // tokens per CTA: fewer when that leaves SMs idle
	while (block > 8 && (long long)cb * seqs * ((p.rows_per_seq + block - 1) / block) < 4 * dn_sm_count()) block /= 2;
	const dim3 grid(cb, (p.rows_per_seq + block - 1) / block, seqs), threads(DN_THREADS);
	if (p.taps <= 4) return dn_launch(ssm_conv_kernel<T, 4>, grid, threads, 0, stream, p, block);
	if (p.taps <= 8) return dn_launch(ssm_conv_kernel<T, 8>, grid, threads, 0, stream, p, block);
	return dn_launch(ssm_conv_kernel<T, 16>, grid, threads, 0, stream, p, block);
}

int ssm_conv_launch(const SsmArgs &p, int dtype, cudaStream_t stream) { return dtype ? conv_launch<float>(p, stream) : conv_launch<bf16>(p, stream); }

int ssm_scan_launch(const SsmArgs &p, cudaStream_t stream) {
	const dim3 grid((p.vdim + SS_PV - 1) / SS_PV, p.heads, p.M / p.rows_per_seq), block(DN_THREADS);
	if (p.state <= 32) return dn_launch(ssm_scan_kernel<1>, grid, block, 0, stream, p);
	if (p.state <= 64) return dn_launch(ssm_scan_kernel<2>, grid, block, 0, stream, p);
	if (p.state <= 128) return dn_launch(ssm_scan_kernel<4>, grid, block, 0, stream, p);
	return dn_launch(ssm_scan_kernel<8>, grid, block, 0, stream, p);
}

}   // namespace gptq
