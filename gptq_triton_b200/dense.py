"""Decoder building blocks with dense bf16 or fp32 weights: projections with fused input and output steps, gated MLPs, norms
ahead of a projection (LayerNorm, RMS norm, RMS norm of equal parts), post-norm residual sublayers, a per-token side input.

The residual stream is fp32 throughout.  Feature sizes are padded with zeros to multiples of 16 when weights are loaded, so
the kernels need no edge cases inside a row; sizes that enter a mean stay the true ones.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass, replace
from typing import Optional

import torch
import torch.nn as nn

from . import _dense
from ._lib import ptr, require_cuda, stream_ptr

# at most this many rows are prepared (residual add, norms) inside the projection that reads them: every CTA repeats the
# preparation, which pays for a row or two and not for more
FUSED_ROWS = 2


def padded(n: int) -> int:
	return (n + 15) // 16 * 16


def pad_to(t: torch.Tensor, *shape: int) -> torch.Tensor:
	"""Zero-pads at the end of every dimension."""
	if tuple(t.shape) == shape:
		return t
	out = torch.zeros(shape, dtype=t.dtype, device=t.device)
	out[tuple(slice(0, n) for n in t.shape)] = t
	return out


@dataclass
class Stream:
	"""The residual stream between two sublayers, not yet formed: rows of `table` by token (plus rows of `pos_table` by
	position), or x (+ norm(y) * gain + shift).  The next projection (or the row kernel) forms it.  x is fp32, or (rows that are
	not the residual stream) in the activation dtype."""
	width: int
	ld: int
	eps: float
	table: Optional[torch.Tensor] = None
	token: Optional[torch.Tensor] = None
	pos_table: Optional[torch.Tensor] = None
	pos: Optional[torch.Tensor] = None
	x: Optional[torch.Tensor] = None
	y: Optional[torch.Tensor] = None
	y_norm: int = _dense.NORM_NONE
	gain: Optional[torch.Tensor] = None
	shift: Optional[torch.Tensor] = None

	@property
	def rows(self) -> int:
		return self.token.numel() if self.x is None else self.x.shape[0]

	def take(self, index: torch.Tensor) -> 'Stream':
		"""The stream of some rows only."""
		pick = lambda t: None if t is None else t.index_select(0, index)
		flat = lambda t: None if t is None else t.reshape(-1).index_select(0, index)
		return replace(self, token=flat(self.token), pos=flat(self.pos), x=pick(self.x), y=pick(self.y))

	def then(self, x: torch.Tensor, y: torch.Tensor, y_norm: int = _dense.NORM_NONE, gain: Optional[torch.Tensor] = None, shift: Optional[torch.Tensor] = None) -> 'Stream':
		"""The stream x + norm(y) * gain + shift."""
		return Stream(self.width, self.ld, self.eps, x=x, y=y, y_norm=y_norm, gain=gain, shift=shift)

	def spec(self, control: torch.Tensor, x_out: Optional[torch.Tensor], final: Optional['Norm']) -> '_dense.Rows':
		r = _dense.Rows()
		if self.x is None:
			r.table, r.token, r.vocab = ptr(self.table), ptr(self.token), self.table.shape[0]
			if self.pos_table is not None:
				r.pos_table, r.pos, r.max_pos = ptr(self.pos_table), ptr(self.pos), self.pos_table.shape[0]
		else:
			r.x_in, r.x_t = ptr(self.x), int(self.x.dtype != torch.float32)
		r.x_out, r.y, r.y_norm, r.gain, r.shift = ptr(x_out), ptr(self.y), self.y_norm, ptr(self.gain), ptr(self.shift)
		r.fin_groups = 1
		if final is not None:
			r.fin_norm, r.fin_w, r.fin_b, r.fin_groups = final.kind, ptr(final.weight), ptr(final.bias), final.parts
		r.width, r.ld, r.eps, r.status = self.width, self.ld, self.eps, _dense.status_ptr(control)
		return r


def prepare_rows(stream: Stream, control: torch.Tensor, dtype: torch.dtype, keep: bool, final=None):
	"""Forms the stream in a kernel of its own: returns (rows for the next projection, new residual stream or None)."""
	M, dev = stream.rows, control.device
	h = torch.empty((M, stream.ld), dtype=dtype, device=dev)
	x = torch.empty((M, stream.ld), dtype=torch.float32, device=dev) if keep else None
	spec = stream.spec(control, x, final)
	_dense.check(_dense.lib().dense_prepare_rows(ctypes.byref(spec), M, ptr(h), stream.ld, _dense.DTYPE_CODE[dtype], stream_ptr(dev)), 'dense_prepare_rows')
	return h, x


def matmul(x, w: torch.Tensor, epi: '_dense.Epilogue', control: torch.Tensor, rows: Optional['_dense.Rows'] = None, M: Optional[int] = None):
	"""epilogue(x W^T); x [M, K] with unit column stride, or None with `rows` (the kernel forms its rows itself)."""
	require_cuda(w, control, *([] if x is None else [x]))
	assert w.stride(1) == 1 and (x is None or x.stride(1) == 1 and x.dtype == w.dtype)
	N, K = w.shape
	rows_n = x.shape[0] if x is not None else M
	lib, code = _dense.lib(), _dense.DTYPE_CODE[w.dtype]
	need = lib.dense_matmul_scratch(rows_n, K, N, code)
	scratch = torch.empty(need, dtype=torch.float32, device=w.device) if need else None
	rc = lib.dense_matmul(ptr(x), 0 if x is None else x.stride(0), ptr(w), w.stride(0), rows_n, K, N, code, None if rows is None else ctypes.byref(rows),
						  ctypes.byref(epi), ptr(scratch), _dense.status_ptr(control), stream_ptr(w.device))
	_dense.check(rc, 'dense_matmul', 2 if need else 1)


def project_stream(stream: Stream, w: torch.Tensor, epi: '_dense.Epilogue', control: torch.Tensor, keep: bool = True, final=None) -> Optional[torch.Tensor]:
	"""Projection of the residual stream: forms the rows inside the projection when they are few, else in the row kernel.
	Returns the new residual stream [M, ld] fp32 (None without `keep`)."""
	M = stream.rows
	if M <= FUSED_ROWS and _dense.lib().dense_decode_rows_ok(M, stream.ld, _dense.DTYPE_CODE[w.dtype]):
		x = torch.empty((M, stream.ld), dtype=torch.float32, device=w.device) if keep else None
		matmul(None, w, epi, control, rows=stream.spec(control, x, final), M=M)
		return x
	h, x = prepare_rows(stream, control, w.dtype, keep, final)
	matmul(h, w, epi, control)
	return x


def epilogue(mode: int, out: torch.Tensor, scale: float = 1.0) -> '_dense.Epilogue':
	e = _dense.Epilogue()
	e.mode, e.out, e.ldo, e.scale = mode, ptr(out), out.stride(0), scale
	return e


def linear(x: torch.Tensor, w: torch.Tensor, control: torch.Tensor, out_dtype: Optional[torch.dtype] = None) -> torch.Tensor:
	"""x W^T as [M, N padded to 16], fp32 by default or in the weights' dtype."""
	f32 = out_dtype is None or out_dtype == torch.float32
	out = torch.empty((x.shape[0], padded(w.shape[0])), dtype=torch.float32 if f32 else out_dtype, device=w.device)
	matmul(x, w, epilogue(_dense.EPI_F32 if f32 else _dense.EPI_T, out), control)
	return out


class Norm(nn.Module):
	"""A norm that a projection applies to the stream it reads; weight and bias fp32, padded."""
	kind = _dense.NORM_NONE
	parts = 1

	def __init__(self, weight: torch.Tensor, bias: Optional[torch.Tensor] = None):
		super().__init__()
		n = padded(weight.numel())
		self.register_buffer('weight', pad_to(weight.float(), n))
		self.register_buffer('bias', None if bias is None else pad_to(bias.float(), n))


class LayerNorm(Norm):
	kind = _dense.NORM_LAYER


class RMSNorm(Norm):
	"""x / rms(x) * (offset + weight), by the mean square of the row or of each of `parts` equal parts."""
	kind = _dense.NORM_RMS

	def __init__(self, weight: torch.Tensor, offset: float = 0.0, parts: int = 1):
		if not 1 <= parts <= _dense.MAX_NORM_GROUPS or weight.numel() % parts:
			raise ValueError(f'an RMS norm of {weight.numel()} entries in {parts} parts')
		super().__init__(weight.float() + offset)
		self.parts = parts


class PostNorm(nn.Module):
	"""What joins a sublayer's output y to the stream: x + multiplier * layer_scale * (LayerNorm(y) * weight + bias), folded
	into one gain and one shift per column."""

	def __init__(self, weight: torch.Tensor, bias: torch.Tensor, layer_scale: Optional[torch.Tensor], multiplier: float):
		super().__init__()
		f = multiplier * (1.0 if layer_scale is None else layer_scale.double())
		n = padded(weight.numel())
		self.register_buffer('gain', pad_to((weight.double() * f).float(), n))
		self.register_buffer('shift', pad_to((bias.double() * f).float(), n))

	def join(self, stream: Stream, x: torch.Tensor, y: torch.Tensor) -> Stream:
		return stream.then(x, y, _dense.NORM_LAYER, self.gain, self.shift)


class DenseMLP(nn.Module):
	"""down(act(gate h) * (up h)).  Gate and up rows alternate in groups of eight in one matrix, so that one pass over it
	leaves both factors of an output in the same thread."""

	def __init__(self, gate: torch.Tensor, up: torch.Tensor, down: torch.Tensor, act: str = 'silu'):
		super().__init__()
		ff, width = gate.shape
		f, w = padded(ff), padded(width)
		g, u = pad_to(gate, f, w), pad_to(up, f, w)
		self.act = _dense.ACT_CODE[act]
		self.register_buffer('gate_up', torch.stack([g.view(f // 8, 8, w), u.view(f // 8, 8, w)], dim=1).reshape(2 * f, w).contiguous())
		self.register_buffer('down', pad_to(down, w, f).contiguous())

	def gated(self, out: torch.Tensor) -> '_dense.Epilogue':
		e = epilogue(_dense.EPI_GATED, out)
		e.act = self.act
		return e

	def forward(self, stream: Stream, control: torch.Tensor, norm: Optional[Norm] = None):
		"""Returns (residual stream x, sublayer output y), both fp32."""
		a = torch.empty((stream.rows, self.down.shape[1]), dtype=self.down.dtype, device=self.down.device)
		x = project_stream(stream, self.gate_up, self.gated(a), control, final=norm)
		return x, linear(a, self.down, control)


class TokenSide(nn.Module):
	"""A layer's per-token input: x + RMSNorm(proj(act(gate x) * e)) with e the columns [column, column + dim) of the token's row
	of `table` (all sizes padded)."""

	def __init__(self, gate: torch.Tensor, proj: torch.Tensor, norm_weight: torch.Tensor, column: int, act: str = 'gelu_tanh'):
		super().__init__()
		dim, width = gate.shape
		d, w = padded(dim), padded(width)
		self.column, self.act = column, _dense.ACT_CODE[act]
		self.register_buffer('gate', pad_to(gate, d, w).contiguous())
		self.register_buffer('proj', pad_to(proj, w, d).contiguous())
		self.register_buffer('gain', pad_to(norm_weight.float(), w))

	def gated(self, out: torch.Tensor, table: torch.Tensor, token: torch.Tensor) -> '_dense.Epilogue':
		e = epilogue(_dense.EPI_TABLE, out)
		e.act, e.tab, e.tab_ld, e.tab_rows, e.tab_col, e.tab_token = self.act, ptr(table), table.stride(0), table.shape[0], self.column, ptr(token)
		return e

	def forward(self, stream: Stream, table: torch.Tensor, token: torch.Tensor, control: torch.Tensor) -> Stream:
		a = torch.empty((stream.rows, self.gate.shape[0]), dtype=self.gate.dtype, device=self.gate.device)
		x = project_stream(stream, self.gate, self.gated(a, table, token), control)
		return stream.then(x, linear(a, self.proj, control), _dense.NORM_RMS, self.gain)
