// fp32 projection for many rows: 64 x 64 output tiles on the FMA units, true fp32 products and sums.
#include "dense.cuh"

namespace gptq {

namespace {

constexpr int SI_T = 64, SI_K = 16, SI_LD = SI_T + 4;

__global__ void __launch_bounds__(DN_THREADS) dense_simt_kernel(const DenseArgs p) {
	__shared__ __align__(16) float s_buf[SI_T * SI_LD];       // operand tiles, later the output tile
	float(*sx)[SI_LD] = reinterpret_cast<float(*)[SI_LD]>(s_buf);
	float(*sw)[SI_LD] = reinterpret_cast<float(*)[SI_LD]>(s_buf + SI_K * SI_LD);
	const int tid = threadIdx.x, m0 = blockIdx.y * SI_T, n0 = blockIdx.x * SI_T;
	const int tm = (tid >> 4) * 4, tn = (tid & 15) * 4;
	const float *x = reinterpret_cast<const float *>(p.x), *w = reinterpret_cast<const float *>(p.w);
	float acc[4][4] = {};
	const int lr = tid >> 2, lk = (tid & 3) * 4;              // one float4 of each operand per thread and K step
	pdl_wait();
	pdl_trigger();
	for (int k0 = 0; k0 < p.K; k0 += SI_K) {                  // K % 16 == 0
		float4 xv = make_float4(0.f, 0.f, 0.f, 0.f), wv = xv;
		if (m0 + lr < p.M) xv = __ldcg(reinterpret_cast<const float4 *>(x + (size_t)(m0 + lr) * p.ldx + k0 + lk));
		if (n0 + lr < p.N) wv = __ldg(reinterpret_cast<const float4 *>(w + (size_t)(n0 + lr) * p.ldw + k0 + lk));
		__syncthreads();
		sx[lk][lr] = xv.x; sx[lk + 1][lr] = xv.y; sx[lk + 2][lr] = xv.z; sx[lk + 3][lr] = xv.w;
		sw[lk][lr] = wv.x; sw[lk + 1][lr] = wv.y; sw[lk + 2][lr] = wv.z; sw[lk + 3][lr] = wv.w;
		__syncthreads();
#pragma unroll
		for (int k = 0; k < SI_K; ++k) {
			const float4 a = *reinterpret_cast<const float4 *>(&sx[k][tm]), b = *reinterpret_cast<const float4 *>(&sw[k][tn]);
			const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
			for (int i = 0; i < 4; ++i)
#pragma unroll
				for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
		}
	}
	__syncthreads();
	float(*so)[SI_LD] = reinterpret_cast<float(*)[SI_LD]>(s_buf);
#pragma unroll
	for (int i = 0; i < 4; ++i) *reinterpret_cast<float4 *>(&so[tm + i][tn]) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
	__syncthreads();
	const int row = tid >> 2, n = n0 + (tid & 3) * 16;
	if (m0 + row < p.M && n < p.N) {
		float v[16];
#pragma unroll
		for (int i = 0; i < 16; ++i) v[i] = so[row][(tid & 3) * 16 + i];
		epi_16<float>(p.e, m0 + row, n, v);
	}
}

}   // namespace

int dense_simt_launch(const DenseArgs &a, cudaStream_t stream) {
	return dn_launch(dense_simt_kernel, dim3((a.N + SI_T - 1) / SI_T, (a.M + SI_T - 1) / SI_T), dim3(DN_THREADS), 0, stream, a);
}

}   // namespace gptq
