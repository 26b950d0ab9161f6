"""Grouped-query attention with cached keys and values, one or two softmax maps per head over the same values.

With two maps (differential attention) a head's output is the difference a_1 - lambda * a_2 of two attentions, normed over the
head's values.  Queries and keys may be RMS-normed per head and map, scores soft-capped; there is no rotation.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn as nn

from . import _dense
from ._lib import ptr, stream_ptr
from .dense import Norm, Stream, epilogue, linear, pad_to, padded, project_stream


# portions of more rows than this per sequence run on the tensor-core prompt kernel (bf16)
DECODE_MAX_ROWS = 8


@dataclass(frozen=True)
class GroupedAttentionSpec:
	heads: int
	kv_heads: int
	dim: int                    # query / key entries per head and map
	vdim: int
	scale: float
	softcap: Optional[float] = None
	maps: int = 1
	diff: float = 0.0           # two maps: the constant part of lambda; the normed difference is multiplied by 1 - diff

	def __post_init__(self):
		if min(self.heads, self.kv_heads, self.dim, self.vdim) < 1 or self.heads % self.kv_heads or self.maps not in (1, 2) or (self.softcap is not None and not self.softcap > 0):
			raise ValueError(f'grouped-query attention sizes: {self}')
		if padded(self.dim) > 512 or padded(self.vdim) > 512:
			raise ValueError(f'the grouped-query attention kernels hold head vectors of up to 512 entries: {self}')

	def cache_layout(self, max_seq: int):
		return {'k': (max_seq, self.kv_heads * self.maps * padded(self.dim)), 'v': (max_seq, self.kv_heads * padded(self.vdim))}


class GroupedAttention(nn.Module):
	"""Query, key and value rows form one matrix; head vectors are padded with zeros to multiples of 16.  lam: the factor of the
	second map (a number of the layer)."""

	def __init__(self, spec: GroupedAttentionSpec, q, k, v, o, q_norm=None, k_norm=None, lam: float = 0.0):
		super().__init__()
		self.spec, self.lam = spec, float(lam)
		H, G, n, D, V = spec.heads, spec.kv_heads, spec.maps, spec.dim, spec.vdim
		self.D, self.V = padded(D), padded(V)
		width, w = q.shape[1], padded(q.shape[1])
		rows = [pad_to(t.reshape(h, d, width), h, p, w).reshape(h * p, w) for t, h, d, p in ((q, H * n, D, self.D), (k, G * n, D, self.D), (v, G, V, self.V))]
		self.register_buffer('w_in', torch.cat(rows).contiguous())
		self.register_buffer('w_o', pad_to(o.reshape(width, H, V), w, H, self.V).reshape(w, H * self.V).contiguous())
		self.register_buffer('q_norm', None if q_norm is None else pad_to(q_norm.float(), self.D))
		self.register_buffer('k_norm', None if k_norm is None else pad_to(k_norm.float(), self.D))
		# vectors of unit root mean square have length sqrt(dim): what the norm weights say about the argument of the cap's tanh
		self.bound = 0.0
		if spec.softcap and q_norm is not None and k_norm is not None:
			self.bound = D * float(q_norm.abs().max()) * float(k_norm.abs().max()) * abs(spec.scale) / spec.softcap

	def forward(self, stream: Stream, cache, pos: torch.Tensor, rows_per_seq: int, start: Optional[int], control: torch.Tensor, norm: Optional[Norm] = None):
		"""stream: M = sequences * rows_per_seq rows at positions pos (int32 [M]); cache: k and v [sequences, max_seq, ...], written
		here.  start: the portion's first position, None for a decode step (positions are known to the device only).  Returns
		(residual stream x, sublayer output y), both fp32."""
		s, dev, dt = self.spec, control.device, self.w_in.dtype
		M, max_seq = stream.rows, cache['k'].shape[1]
		maps = 0 if start is None or dt == torch.float32 or rows_per_seq <= DECODE_MAX_ROWS else _dense.lib().dense_gqa_prefill_maps(s.maps, self.D, self.V)
		raw = torch.empty((M, self.w_in.shape[0]), dtype=dt if maps else torch.float32, device=dev)
		x = project_stream(stream, self.w_in, epilogue(_dense.EPI_T if maps else _dense.EPI_F32, raw), control, final=norm)
		a = self.arguments(raw, cache, pos, rows_per_seq, stream.eps, control)
		lib, code, st = _dense.lib(), _dense.DTYPE_CODE[dt], stream_ptr(dev)
		out = torch.empty((M, s.heads * self.V), dtype=dt, device=dev)
		if maps:
			self._prompt(a, out, rows_per_seq, start, maps, cache)
		else:
			scratch = self.buffers(a, out, max_seq if start is None else start + rows_per_seq)      # noqa: F841 (alive until the launches)
			_dense.check(lib.dense_gqa_append(ctypes.byref(a), code, st), 'dense_gqa_append')
			_dense.check(lib.dense_gqa_attend(ctypes.byref(a), code, st), 'dense_gqa_attend')
			_dense.check(lib.dense_gqa_merge(ctypes.byref(a), code, st), 'dense_gqa_merge')
		return x, linear(out, self.w_o, control)

	def arguments(self, raw, cache, pos, rows_per_seq: int, eps: float, control) -> '_dense.Gqa':
		s, a = self.spec, _dense.Gqa()
		a.M, a.rows_per_seq, a.heads, a.kv_heads, a.maps = pos.numel(), rows_per_seq, s.heads, s.kv_heads, s.maps
		a.dim, a.vdim, a.dim_true, a.vdim_true, a.max_seq, a.splits = self.D, self.V, s.dim, s.vdim, cache['k'].shape[1], 1
		a.scale, a.cap, a.eps, a.lambda_, a.bound = s.scale, s.softcap or 0.0, eps, self.lam, self.bound
		a.out_norm, a.out_mul = int(s.maps == 2), 1.0 - s.diff if s.maps == 2 else 1.0
		a.pos, a.raw, a.raw_t, a.raw_ld, a.q_norm, a.k_norm = ptr(pos), ptr(raw), int(raw.dtype != torch.float32), raw.stride(0), ptr(self.q_norm), ptr(self.k_norm)
		a.k_cache, a.v_cache, a.status = ptr(cache['k']), ptr(cache['v']), _dense.status_ptr(control)
		return a

	def buffers(self, a: '_dense.Gqa', out, keys: int):
		"""Scratch for up to `keys` visible positions, entered into `a`; returns what must stay alive."""
		s, dev, f32 = self.spec, out.device, out.dtype == torch.float32
		a.splits = _dense.lib().dense_gqa_splits(a.M, s.heads, s.kv_heads, s.maps, keys, _dense.DTYPE_CODE[out.dtype])
		q = torch.empty((1 if f32 else 2, a.M, s.heads * s.maps, self.D), dtype=out.dtype, device=dev)
		ml = torch.empty((a.M, s.heads * s.maps, a.splits, 2), dtype=torch.float32, device=dev)
		acc = torch.empty((a.M, s.heads * s.maps, a.splits, self.V), dtype=torch.float32, device=dev)
		a.part_ml, a.part_acc, a.out, a.out_ld = ptr(ml), ptr(acc), ptr(out), out.stride(0)
		if f32:
			a.q_f32 = ptr(q)
		else:
			a.q_hi, a.q_lo = ptr(q[0]), ptr(q[1])
		return q, ml, acc

	def _prompt(self, a: '_dense.Gqa', out, t: int, start: int, maps: int, cache):
		"""Normed queries and cache rows of all sequences, then the tensor-core attention kernel per sequence."""
		s, dev, lib = self.spec, out.device, _dense.lib()
		st = stream_ptr(dev)
		q = torch.empty((a.M, s.heads * s.maps * self.D), dtype=out.dtype, device=dev)
		a.q_hi, a.out, a.out_ld, a.splits = ptr(q), ptr(out), out.stride(0), 1
		if maps < s.maps or s.maps == 1:
			ml = torch.empty((a.M, s.heads * s.maps, 2), dtype=torch.float32, device=dev)
			acc = torch.empty((a.M, s.heads * s.maps, self.V), dtype=torch.float32, device=dev)
			a.part_ml, a.part_acc = ptr(ml), ptr(acc)
		_dense.check(lib.dense_gqa_append(ctypes.byref(a), 0, st), 'dense_gqa_append')
		for b in range(a.M // t):
			one = _dense.Gqa.from_buffer_copy(a)
			rows = slice(b * t, (b + 1) * t)
			one.M, one.q_hi, one.out, one.k_cache, one.v_cache = t, ptr(q[rows]), ptr(out[rows]), ptr(cache['k'][b]), ptr(cache['v'][b])
			if a.part_ml:
				one.part_ml, one.part_acc = ptr(ml[rows]), ptr(acc[rows])
			_dense.check(lib.dense_gqa_prefill(ctypes.byref(one), start, st), 'dense_gqa_prefill')
		if a.part_ml:
			_dense.check(lib.dense_gqa_merge(ctypes.byref(a), 0, st), 'dense_gqa_merge')


def diff_lambda(lq1: torch.Tensor, lk1: torch.Tensor, lq2: torch.Tensor, lk2: torch.Tensor, diff: float) -> float:
	"""exp(lq1 . lk1) - exp(lq2 . lk2) + diff."""
	dot = lambda a, b: (a.double() * b.double()).sum()
	return float(dot(lq1, lk1).exp() - dot(lq2, lk2).exp()) + diff
