"""ctypes binding of libdense_b200.so (declared in include/dense_b200.h).  Like the other binding it has no fallback: a
missing library or a failing kernel raises."""
from __future__ import annotations

import ctypes
from ctypes import c_float, c_int, c_int64, c_void_p
from pathlib import Path
from typing import Optional

import torch

from ._lib import GptqB200Error, ptr, register_status_buffer, require_cuda, stream_ptr      # noqa: F401

LIB_PATH = Path(__file__).resolve().parent / 'libdense_b200.so'
CONTROL_BYTES = 16384

EPI_F32, EPI_T, EPI_GATED, EPI_QKV, EPI_LOGITS, EPI_TABLE, EPI_MIXED = range(7)
ACT_CODE = {'silu': 0, 'gelu_tanh': 1}
NORM_NONE, NORM_LAYER, NORM_RMS = range(3)
MAX_NORM_GROUPS = 256
SSM_CHUNK = 128
DTYPE_CODE = {torch.bfloat16: 0, torch.float32: 1}

_P, _I = c_void_p, c_int


class Rows(ctypes.Structure):
	_fields_ = [('x_in', _P), ('x_t', _I), ('x_out', _P), ('y', _P), ('gain', _P), ('shift', _P), ('fin_w', _P), ('fin_b', _P), ('table', _P), ('token', _P),
				('vocab', c_int64), ('pos_table', _P), ('pos', _P), ('max_pos', _I), ('y_norm', _I), ('fin_norm', _I), ('fin_groups', _I), ('width', _I), ('ld', _I), ('eps', c_float), ('status', _P)]


class Epilogue(ctypes.Structure):
	_fields_ = [('mode', _I), ('out', _P), ('ldo', c_int64), ('scale', c_float),
				('n_q', _I), ('head_dim', _I), ('rot_at', _I), ('rot_dims', _I), ('n_kv', _I), ('n_gate', _I),
				('cos_t', _P), ('sin_t', _P), ('pos', _P), ('max_pos', _I), ('q_out', _P), ('q_f32', _I), ('kv_out', _P), ('gate_out', _P), ('status', _P),
				('best', _P), ('ticket', _P), ('tok', _P), ('pos_inout', _P), ('act', _I), ('tab', _P), ('tab_ld', c_int64), ('tab_rows', c_int64), ('tab_col', _I),
				('tab_token', _P)]


class Latent(ctypes.Structure):
	_fields_ = [(n, _I) for n in ('M', 'rows_per_seq', 'heads', 'dim', 'rot_dim', 'vdim', 'kv_rank', 'kv_width', 'rot_dims', 'max_seq', 'splits')] + [
		('scale', c_float), ('eps', c_float), ('pos', _P), ('q', _P), ('w_uk', _P), ('w_uv', _P), ('kv_raw', _P), ('kv_norm', _P), ('cos_t', _P), ('sin_t', _P),
		('cache', _P), ('qa_hi', _P), ('qa_lo', _P), ('qa_f32', _P), ('part_ml', _P), ('part_acc', _P), ('gate', _P), ('gate_ld', _I), ('out', _P), ('out_ld', c_int64),
		('status', _P)]


class LatentPrefill(ctypes.Structure):
	_fields_ = [(n, _I) for n in ('t', 'start', 'S', 'heads', 'dim', 'rot_dim', 'vdim', 'kv_rank')] + [
		('scale', c_float), ('q', _P), ('k', _P), ('vt', _P), ('ldv', c_int64), ('cache', _P), ('gate', _P), ('gate_ld', _I), ('out', _P), ('out_ld', c_int64), ('status', _P)]


class Gqa(ctypes.Structure):
	_fields_ = [(n, _I) for n in ('M', 'rows_per_seq', 'heads', 'kv_heads', 'maps', 'dim', 'vdim', 'dim_true', 'vdim_true', 'max_seq', 'splits')] + [
		(n, c_float) for n in ('scale', 'cap', 'eps', 'lambda_', 'out_mul', 'bound')] + [
		('out_norm', _I), ('pos', _P), ('raw', _P), ('raw_t', _I), ('raw_ld', c_int64), ('q_norm', _P), ('k_norm', _P), ('k_cache', _P), ('v_cache', _P), ('q_hi', _P), ('q_lo', _P),
		('q_f32', _P), ('part_ml', _P), ('part_acc', _P), ('out', _P), ('out_ld', c_int64), ('status', _P)]


class Ssm(ctypes.Structure):
	_fields_ = [(n, _I) for n in ('M', 'rows_per_seq', 'heads', 'vdim', 'state', 'groups', 'taps', 'z_at', 'conv_at', 'conv_ld')] + [
		('raw_ld', c_int64), ('dt_ld', c_int64)] + [(n, _P) for n in ('raw', 'dt', 'pos', 'conv_w', 'conv_b', 'dt_bias', 'a', 'd', 'ring', 's', 'u', 'chunk_s', 'chunk_decay', 'out')] + [
		('out_ld', c_int64), ('status', _P)]


_SIGNATURES = {
	'dense_version': (c_int, []),
	'dense_last_cuda_error': (c_int, []),
	'dense_matmul': (c_int, [_P, c_int64, _P, c_int64, _I, _I, _I, _I, _P, _P, _P, _P, _P]),
	'dense_matmul_scratch': (c_int64, [_I, _I, _I, _I]),
	'dense_decode_rows_ok': (c_int, [_I, _I, _I]),
	'dense_prepare_rows': (c_int, [_P, _I, _P, c_int64, _I, _P]),
	'dense_latent_splits': (c_int, [_I, _I, _I, _I]),
	'dense_latent_append': (c_int, [_P, _I, _P]),
	'dense_latent_absorb': (c_int, [_P, _I, _P]),
	'dense_latent_attend': (c_int, [_P, _I, _P]),
	'dense_latent_value': (c_int, [_P, _I, _P]),
	'dense_latent_prefill_ok': (c_int, [_I, _I, _I]),
	'dense_latent_prefill': (c_int, [_P, _P]),
	'dense_gqa_splits': (c_int, [_I, _I, _I, _I, _I, _I]),
	'dense_gqa_append': (c_int, [_P, _I, _P]),
	'dense_gqa_attend': (c_int, [_P, _I, _P]),
	'dense_gqa_merge': (c_int, [_P, _I, _P]),
	'dense_gqa_prefill_maps': (c_int, [_I, _I, _I]),
	'dense_gqa_prefill': (c_int, [_P, _I, _P]),
	'dense_ssm_step': (c_int, [_P, _P]),
	'dense_ssm_conv': (c_int, [_P, _I, _P]),
	'dense_ssm_scan': (c_int, [_P, _P]),
	'dense_ssm_chunked': (c_int, [_P, _P]),
	'dense_ssm_chunked_scratch': (c_int, [_P]),
}

_lib: Optional[ctypes.CDLL] = None
launches = 0          # kernels launched through this binding (an entry point that returns a status is one launch unless its caller says more)


def exported_symbols():
	"""Names that include/dense_b200.h declares."""
	return list(_SIGNATURES)


def lib() -> ctypes.CDLL:
	global _lib
	if _lib is None:
		if not LIB_PATH.exists():
			raise ImportError(f'{LIB_PATH} is missing: build it with `python -m gptq_triton_b200.build` (needs nvcc with sm_100a support). '
							  'There is no CPU or Triton fallback.')
		l = ctypes.CDLL(str(LIB_PATH))
		for name, (res, args) in _SIGNATURES.items():
			fn = getattr(l, name)
			fn.restype, fn.argtypes = res, args
		_lib = l
	return _lib


_MESSAGES = {-1: 'invalid argument', -2: 'shape violates a divisibility rule', -4: 'pointer or leading dimension misaligned', -5: 'CUDA error', -6: 'not supported'}


def check(code: int, what: str, kernels: int = 1):
	global launches
	launches += kernels
	if code != 0:
		extra = f' (cudaError {lib().dense_last_cuda_error()})' if code == -5 else ''
		raise (ValueError if code in (-1, -2, -4) else GptqB200Error)(f'{what}: {_MESSAGES.get(code, "unknown error code")}{extra}')


def control_buffer(device) -> torch.Tensor:
	"""Zeroed control words of an engine (arrival counters, candidates of the greedy choice, status word), registered with
	_lib.kernel_status()."""
	buf = torch.zeros(CONTROL_BYTES, dtype=torch.uint8, device=device)
	register_status_buffer(buf)
	return buf


def status_ptr(control: torch.Tensor) -> c_void_p:
	return c_void_p(control.data_ptr() + CONTROL_BYTES - 4)
