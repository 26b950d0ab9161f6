// extern "C" entry points of libdense_b200.so: argument checks and kernel selection.
#include <mutex>
#include <set>
#include <utility>

#include "gqa.cuh"
#include "latent.cuh"
#include "ssm.cuh"

namespace gptq {

thread_local int g_last_cuda_error = 0;

int dn_sm_count() {
	static int cached[64] = {0};
	int dev = 0;
	if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return 148;
	if (cached[dev] == 0) {
		int n = 0;
		if (cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || n <= 0) n = 148;
		cached[dev] = n;
	}
	return cached[dev];
}

// raises a kernel's dynamic shared memory limit to the most a CTA may have, once per kernel and device
int dn_smem_opt_in(const void *kernel, size_t bytes) {
	static std::mutex mutex;
	static std::set<std::pair<int, const void *>> done;
	int dev = 0;
	if (cudaError_t e = cudaGetDevice(&dev)) return cuda_status(e);
	std::lock_guard<std::mutex> lock(mutex);
	if (done.count({dev, kernel})) return GPTQ_OK;
	cudaFuncAttributes attr;
	if (cudaError_t e = cudaFuncGetAttributes(&attr, kernel)) return cuda_status(e);
	const size_t room = 227 * 1024 - attr.sharedSizeBytes;
	if (bytes > room) return GPTQ_ERR_UNSUPPORTED;
	if (cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)room)) return cuda_status(e);
	done.insert({dev, kernel});
	return GPTQ_OK;
}

static bool rows_bad(const RowPrep &r, int dtype) {
	if (r.width < 1 || r.ld < r.width || r.ld % 16 != 0 || !(r.eps >= 0.f) || !r.status) return true;
	if (r.table ? !r.token || r.vocab < 1 : !r.x_in) return true;
	if (r.pos_table && (!r.table || !r.pos || r.max_pos < 1)) return true;
	if (r.y_norm < DENSE_NORM_NONE || r.y_norm > DENSE_NORM_RMS || r.fin_norm < DENSE_NORM_NONE || r.fin_norm > DENSE_NORM_RMS) return true;
	if ((r.fin_w || r.fin_b) && r.fin_norm == DENSE_NORM_NONE) return true;
	if (r.fin_groups < 1 || r.fin_groups > DENSE_MAX_NORM_GROUPS) return true;
	if (r.fin_groups > 1 && (r.fin_norm != DENSE_NORM_RMS || r.width % r.fin_groups || r.table || r.y || r.x_out || r.fin_b)) return true;
	if (r.x_out && (const void *)r.x_out == r.x_in) return true;
	return !aligned16(r.pos_table) || !aligned16(r.x_in) || !aligned16(r.x_out) || !aligned16(r.y) || !aligned16(r.gain) || !aligned16(r.shift) || !aligned16(r.fin_w) || !aligned16(r.fin_b) || !aligned16(r.table);
}

static bool latent_bad(const LatentArgs &a, int dtype, bool attend) {
	if (a.M < 1 || a.rows_per_seq < 1 || a.M % a.rows_per_seq || a.heads < 1 || a.dim < 16 || a.rot_dim < 16 || a.vdim < 16 || a.kv_rank < 16) return true;
	if (a.dim % 16 || a.rot_dim % 16 || a.vdim % 16 || a.kv_rank % 16 || a.rot_dims % 2 || a.rot_dims < 0 || a.rot_dims > a.rot_dim) return true;
	if (a.kv_width < 1 || a.kv_width > a.kv_rank || a.max_seq < 1 || a.splits < 1 || a.splits > 64 || (dtype != 0 && dtype != 1)) return true;
	if (!a.pos || !a.cache || !a.status) return true;
	if (a.kv_raw && (!a.kv_norm || !a.cos_t || !a.sin_t)) return true;
	if (attend && (dtype ? !a.qa_f32 : !a.qa_hi || !a.qa_lo)) return true;
	return false;
}

static bool gqa_bad(const GqaArgs &a, int dtype) {
	if (a.M < 1 || a.rows_per_seq < 1 || a.M % a.rows_per_seq || a.heads < 1 || a.kv_heads < 1 || a.heads % a.kv_heads || a.maps < 1 || a.maps > 2) return true;
	if (a.dim < 16 || a.vdim < 16 || a.dim % 16 || a.vdim % 16 || a.dim_true < 1 || a.dim_true > a.dim || a.vdim_true < 1 || a.vdim_true > a.vdim) return true;
	if (a.max_seq < 1 || a.splits < 1 || a.splits > 64 || !(a.cap >= 0.f) || !(a.eps >= 0.f) || (dtype != 0 && dtype != 1)) return true;
	return !a.pos || !a.k_cache || !a.v_cache || !a.status || (dtype ? !a.q_f32 : !a.q_hi);
}

static bool ssm_bad(const SsmArgs &a) {
	if (a.M < 1 || a.rows_per_seq < 1 || a.M % a.rows_per_seq || a.heads < 1 || a.vdim < 1 || a.state < 1 || a.state > SS_MAX_STATE) return true;
	if (a.groups < 1 || a.heads % a.groups || a.taps < 1 || a.taps > SS_MAX_TAPS) return true;
	const int inner = a.heads * a.vdim, channels = inner + 2 * a.groups * a.state;
	if (a.z_at < 0 || a.conv_at < 0 || a.conv_ld < channels || a.z_at + inner > a.raw_ld || a.conv_at + a.conv_ld > a.raw_ld || a.dt_ld < a.heads) return true;
	if (a.conv_ld % 16 || a.conv_at % 16 || a.z_at % 16 || a.raw_ld % 16) return true;
	return !a.raw || !a.dt || !a.pos || !a.conv_w || !a.conv_b || !a.dt_bias || !a.a || !a.d || !a.ring || !a.s || !a.status;
}

}   // namespace gptq

using namespace gptq;

extern "C" {

int dense_version(void) { return 100; }
int dense_last_cuda_error(void) { return g_last_cuda_error; }
int dense_decode_rows_ok(int M, int K, int dtype) { return dense_skinny_ok(M, K, dtype) ? 1 : 0; }

int dense_matmul(const void *x, int64_t ldx, const void *w, int64_t ldw, int M, int K, int N, int dtype, const dense_rows_t *rows, const dense_epilogue_t *epi, float *scratch,
				 int *status, void *stream) {
	if (!w || !epi || !status || M < 0 || K < 16 || N < 1 || (dtype != 0 && dtype != 1) || (!rows && !x)) return GPTQ_ERR_INVALID;
	if (M == 0) return GPTQ_OK;
	if (K % 16) return GPTQ_ERR_SHAPE;
	if (!aligned16(w) || ldw % 8 || ldw < K || (!rows && (!aligned16(x) || ldx % 8 || ldx < K))) return GPTQ_ERR_ALIGN;
	const int n16 = (N + 15) / 16 * 16;
	switch (epi->mode) {
		case DENSE_EPI_F32:
		case DENSE_EPI_T:
		case DENSE_EPI_LOGITS:
			if (!epi->out || epi->ldo < n16 || epi->ldo % 8) return GPTQ_ERR_INVALID;
			break;
		case DENSE_EPI_TABLE:
			if (!epi->out || epi->ldo < n16 || epi->ldo % 8 || !epi->tab || !epi->tab_token || epi->tab_rows < 1) return GPTQ_ERR_INVALID;
			if (epi->tab_col < 0 || epi->tab_col % 8 || epi->tab_ld % 8 || epi->tab_ld < epi->tab_col + n16 || !aligned16(epi->tab)) return GPTQ_ERR_ALIGN;
			break;
		case DENSE_EPI_MIXED:
			if (!epi->out || epi->n_q < 16 || epi->n_q % 16 || epi->n_kv % 16 || epi->n_q + epi->n_kv != N || epi->ldo < epi->n_q || epi->ldo % 8) return GPTQ_ERR_INVALID;
			if (epi->n_kv && !epi->kv_out) return GPTQ_ERR_INVALID;
			break;
		case DENSE_EPI_GATED:
			if (!epi->out || N % 16 || epi->ldo < N / 2 || epi->ldo % 8) return GPTQ_ERR_INVALID;
			break;
		case DENSE_EPI_QKV:
			if (!epi->q_out || !epi->pos || !epi->cos_t || !epi->sin_t || !epi->status || epi->max_pos < 1 || epi->head_dim < 16) return GPTQ_ERR_INVALID;
			if (epi->n_q % epi->head_dim || epi->head_dim % 16 || epi->rot_at % 16 || epi->rot_dims % 2 || epi->n_kv % 16) return GPTQ_ERR_SHAPE;
			if (epi->n_kv && !epi->kv_out) return GPTQ_ERR_INVALID;
			if (epi->n_gate && (!epi->gate_out || epi->n_gate % 16)) return GPTQ_ERR_INVALID;
			if (dtype == 1 && !epi->q_f32) return GPTQ_ERR_INVALID;
			break;
		default:
			return GPTQ_ERR_INVALID;
	}
	if (epi->act != DENSE_ACT_SILU && epi->act != DENSE_ACT_GELU) return GPTQ_ERR_INVALID;
	if (epi->mode == DENSE_EPI_LOGITS && epi->best && (!epi->ticket || !epi->tok || !epi->pos_inout)) return GPTQ_ERR_INVALID;
	DenseArgs a = {};
	a.x = x;
	a.ldx = ldx;
	a.w = w;
	a.ldw = ldw;
	a.M = M;
	a.K = K;
	a.N = N;
	a.e = *epi;
	a.status = status;
	a.ws = scratch;
	if (!aligned16(scratch)) return GPTQ_ERR_ALIGN;
	if (rows) {
		if (rows_bad(*rows, dtype) || rows->ld != K) return GPTQ_ERR_INVALID;
		a.prep = 1;
		a.rp = *rows;
	}
	const cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
	if (dense_skinny_ok(M, K, dtype)) return dense_skinny_launch(a, dtype, st);
	if (rows || epi->best) return GPTQ_ERR_UNSUPPORTED;
	return dtype ? dense_simt_launch(a, st) : dense_tc_launch(a, st);
}

int64_t dense_matmul_scratch(int M, int K, int N, int dtype) {
	if (dtype || M < 1 || K < 16 || N < 1 || dense_skinny_ok(M, K, dtype)) return 0;
	const int parts = dense_tc_parts(M, K, N);
	return parts > 1 ? (int64_t)parts * M * ((N + 15) / 16 * 16) : 0;
}

int dense_prepare_rows(const dense_rows_t *rows, int M, void *h, int64_t ldh, int dtype, void *stream) {
	if (!rows || !h || M < 0 || (dtype != 0 && dtype != 1) || rows_bad(*rows, dtype) || ldh < rows->ld || ldh % 8 || !aligned16(h)) return GPTQ_ERR_INVALID;
	if (M == 0) return GPTQ_OK;
	return dense_rows_launch(*rows, M, h, ldh, dtype, reinterpret_cast<cudaStream_t>(stream));
}

int dense_latent_splits(int M, int heads, int max_seq, int dtype) { return M < 1 || heads < 1 || max_seq < 1 ? 1 : latent_splits(M, heads, max_seq, dtype); }

int dense_latent_append(const dense_latent_t *a, int dtype, void *stream) {
	if (!a || latent_bad(*a, dtype, false) || !a->kv_raw) return GPTQ_ERR_INVALID;
	return latent_absorb_launch(*a, false, dtype, reinterpret_cast<cudaStream_t>(stream));
}
int dense_latent_absorb(const dense_latent_t *a, int dtype, void *stream) {
	if (!a || latent_bad(*a, dtype, true) || !a->q || !a->w_uk) return GPTQ_ERR_INVALID;
	return latent_absorb_launch(*a, true, dtype, reinterpret_cast<cudaStream_t>(stream));
}
int dense_latent_attend(const dense_latent_t *a, int dtype, void *stream) {
	if (!a || latent_bad(*a, dtype, true) || !a->part_ml || !a->part_acc) return GPTQ_ERR_INVALID;
	if (!latent_attend_ok(a->kv_rank, a->rot_dim)) return GPTQ_ERR_UNSUPPORTED;
	return latent_attend_launch(*a, dtype, reinterpret_cast<cudaStream_t>(stream));
}
int dense_latent_value(const dense_latent_t *a, int dtype, void *stream) {
	if (!a || latent_bad(*a, dtype, false) || !a->part_ml || !a->part_acc || !a->w_uv || !a->out || a->out_ld < (int64_t)a->heads * a->vdim) return GPTQ_ERR_INVALID;
	return latent_value_launch(*a, dtype, reinterpret_cast<cudaStream_t>(stream));
}

int dense_latent_prefill_ok(int dim, int rot_dim, int vdim) { return latent_prefill_ok(dim, rot_dim, vdim) ? 1 : 0; }

int dense_latent_prefill(const dense_latent_prefill_t *a, void *stream) {
	if (!a || a->t < 1 || a->start < 0 || a->S != a->start + a->t || a->heads < 1 || !(a->scale > 0.f)) return GPTQ_ERR_INVALID;
	if (a->dim < 16 || a->rot_dim < 16 || a->vdim < 16 || a->kv_rank < 16 || a->dim % 16 || a->rot_dim % 16 || a->vdim % 16 || a->kv_rank % 16) return GPTQ_ERR_SHAPE;
	if (!a->q || !a->k || !a->vt || !a->cache || !a->out || !a->status) return GPTQ_ERR_INVALID;
	if (a->ldv % 8 || a->ldv < a->S || a->out_ld % 8 || a->out_ld < (int64_t)a->heads * a->vdim) return GPTQ_ERR_ALIGN;
	if (!latent_prefill_ok(a->dim, a->rot_dim, a->vdim)) return GPTQ_ERR_UNSUPPORTED;
	return latent_prefill_launch(*a, reinterpret_cast<cudaStream_t>(stream));
}


int dense_gqa_splits(int M, int heads, int kv_heads, int maps, int max_seq, int dtype) {
	return M < 1 || heads < 1 || kv_heads < 1 || maps < 1 || max_seq < 1 ? 1 : gqa_splits(M, heads, kv_heads, maps, max_seq, dtype);
}

int dense_gqa_append(const dense_gqa_t *a, int dtype, void *stream) {
	if (!a || gqa_bad(*a, dtype) || !a->raw) return GPTQ_ERR_INVALID;
	if (a->dim > 512 || a->vdim > 512) return GPTQ_ERR_UNSUPPORTED;
	if (!aligned16(a->raw) || a->raw_ld % 4 || a->raw_ld < (int64_t)(a->heads + a->kv_heads) * a->maps * a->dim + (int64_t)a->kv_heads * a->vdim) return GPTQ_ERR_ALIGN;
	return gqa_append_launch(*a, dtype, reinterpret_cast<cudaStream_t>(stream));
}
int dense_gqa_attend(const dense_gqa_t *a, int dtype, void *stream) {
	if (!a || gqa_bad(*a, dtype) || !a->part_ml || !a->part_acc || (!dtype && !a->q_lo)) return GPTQ_ERR_INVALID;
	if (!gqa_attend_ok(a->maps, a->dim, a->vdim) || a->M > 65535) return GPTQ_ERR_UNSUPPORTED;
	return gqa_attend_launch(*a, dtype, reinterpret_cast<cudaStream_t>(stream));
}
int dense_gqa_merge(const dense_gqa_t *a, int dtype, void *stream) {
	if (!a || gqa_bad(*a, dtype) || !a->part_ml || !a->part_acc || !a->out || a->out_ld % 8 || a->out_ld < (int64_t)a->heads * a->vdim) return GPTQ_ERR_INVALID;
	if (a->vdim > 512 || a->M > 65535) return GPTQ_ERR_UNSUPPORTED;
	return gqa_merge_launch(*a, dtype, reinterpret_cast<cudaStream_t>(stream));
}

int dense_gqa_prefill_maps(int maps, int dim, int vdim) { return gqa_prefill_maps(maps, dim, vdim); }
int dense_gqa_prefill(const dense_gqa_t *a, int start, void *stream) {
	if (!a || gqa_bad(*a, 0) || start < 0 || start + a->M > a->max_seq || a->rows_per_seq != a->M) return GPTQ_ERR_INVALID;
	const int maps = gqa_prefill_maps(a->maps, a->dim, a->vdim);
	if (!maps) return GPTQ_ERR_UNSUPPORTED;
	if (maps == 2 ? !a->out || a->out_ld % 8 || a->out_ld < (int64_t)a->heads * a->vdim || !aligned16(a->out) : !a->part_ml || !a->part_acc || a->splits != 1) return GPTQ_ERR_INVALID;
	if (!aligned16(a->q_hi) || !aligned16(a->k_cache) || !aligned16(a->v_cache)) return GPTQ_ERR_ALIGN;
	return gqa_prefill_launch(*a, start, reinterpret_cast<cudaStream_t>(stream));
}

int dense_ssm_step(const dense_ssm_t *a, void *stream) {
	if (!a || ssm_bad(*a) || a->rows_per_seq != 1 || !a->out || a->out_ld < (int64_t)a->heads * a->vdim || a->M > 65535) return GPTQ_ERR_INVALID;
	return ssm_step_launch(*a, reinterpret_cast<cudaStream_t>(stream));
}
int dense_ssm_conv(const dense_ssm_t *a, int dtype, void *stream) {
	if (!a || ssm_bad(*a) || !a->u || !aligned16(a->u) || !aligned16(a->raw) || (dtype != 0 && dtype != 1)) return GPTQ_ERR_INVALID;
	return ssm_conv_launch(*a, dtype, reinterpret_cast<cudaStream_t>(stream));
}
int dense_ssm_scan(const dense_ssm_t *a, void *stream) {
	if (!a || ssm_bad(*a) || !a->u || !a->out || a->out_ld < (int64_t)a->heads * a->vdim) return GPTQ_ERR_INVALID;
	return ssm_scan_launch(*a, reinterpret_cast<cudaStream_t>(stream));
}
int dense_ssm_chunked_scratch(const dense_ssm_t *a) { return a && !ssm_bad(*a) && ssm_tc_ok(*a) ? 0 : 1; }
int dense_ssm_chunked(const dense_ssm_t *a, void *stream) {
	if (!a || ssm_bad(*a) || !a->u || !a->out || a->out_ld % 2 || a->out_ld < (int64_t)a->heads * a->vdim || (!ssm_tc_ok(*a) && (!a->chunk_s || !a->chunk_decay))) return GPTQ_ERR_INVALID;
	if (!aligned16(a->u) || !aligned16(a->raw) || !aligned16(a->out)) return GPTQ_ERR_ALIGN;
	if ((long long)(a->M / a->rows_per_seq) * ((a->rows_per_seq + SS_CHUNK - 1) / SS_CHUNK) > 65535) return GPTQ_ERR_UNSUPPORTED;
	return ssm_tc_ok(*a) ? ssm_tc_launch(*a, reinterpret_cast<cudaStream_t>(stream)) : ssm_chunk_launch(*a, reinterpret_cast<cudaStream_t>(stream));
}

}   // extern "C"
