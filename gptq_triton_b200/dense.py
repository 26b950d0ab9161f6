"""Decoder building blocks with dense bf16 or fp32 weights: projections with fused input and output steps, a SiLU-gated MLP,
post-norm residual sublayers with LayerNorm and layer scale.

The residual stream is fp32 throughout.  Feature sizes are padded with zeros to multiples of 16 when weights are loaded, so
the kernels need no edge cases inside a row; sizes that enter a mean stay the true ones.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
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
	"""The residual stream between two sublayers, not yet formed: rows of `table` by token, or
	x (+ LayerNorm(y) * gain + shift).  The next projection (or the row kernel) forms it."""
	width: int
	ld: int
	eps: float
	table: Optional[torch.Tensor] = None
	token: Optional[torch.Tensor] = None
	x: Optional[torch.Tensor] = None
	y: Optional[torch.Tensor] = None
	gain: Optional[torch.Tensor] = None
	shift: Optional[torch.Tensor] = None

	@property
	def rows(self) -> int:
		return self.token.numel() if self.x is None else self.x.shape[0]

	def take(self, index: torch.Tensor) -> 'Stream':
		"""The stream of some rows only."""
		pick = lambda t: None if t is None else t.index_select(0, index)
		return Stream(self.width, self.ld, self.eps, self.table, None if self.token is None else self.token.reshape(-1).index_select(0, index), pick(self.x), pick(self.y),
					  self.gain, self.shift)

	def spec(self, control: torch.Tensor, x_out: Optional[torch.Tensor], final) -> '_dense.Rows':
		r = _dense.Rows()
		if self.x is None:
			r.table, r.token, r.vocab = ptr(self.table), ptr(self.token), self.table.shape[0]
		else:
			r.x_in = ptr(self.x)
		r.x_out, r.y, r.gain, r.shift = ptr(x_out), ptr(self.y), ptr(self.gain), ptr(self.shift)
		if final is not None:
			r.fin_w, r.fin_b = ptr(final.weight), ptr(final.bias)
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
	rc = _dense.lib().dense_matmul(ptr(x), 0 if x is None else x.stride(0), ptr(w), w.stride(0), x.shape[0] if x is not None else M, K, N, _dense.DTYPE_CODE[w.dtype],
								   None if rows is None else ctypes.byref(rows), ctypes.byref(epi), _dense.status_ptr(control), stream_ptr(w.device))
	_dense.check(rc, 'dense_matmul')


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


class LayerNorm(nn.Module):
	"""Weight and bias (fp32, padded) of a LayerNorm that a projection applies to the stream it reads."""

	def __init__(self, weight: torch.Tensor, bias: torch.Tensor):
		super().__init__()
		n = padded(weight.numel())
		self.register_buffer('weight', pad_to(weight.float(), n))
		self.register_buffer('bias', pad_to(bias.float(), n))


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
		return Stream(stream.width, stream.ld, stream.eps, x=x, y=y, gain=self.gain, shift=self.shift)


class DenseMLP(nn.Module):
	"""down(silu(gate h) * (up h)).  Gate and up rows alternate in groups of eight in one matrix, so that one pass over it
	leaves both factors of an output in the same thread."""

	def __init__(self, gate: torch.Tensor, up: torch.Tensor, down: torch.Tensor):
		super().__init__()
		ff, width = gate.shape
		f, w = padded(ff), padded(width)
		g, u = pad_to(gate, f, w), pad_to(up, f, w)
		self.register_buffer('gate_up', torch.stack([g.view(f // 8, 8, w), u.view(f // 8, 8, w)], dim=1).reshape(2 * f, w).contiguous())
		self.register_buffer('down', pad_to(down, w, f).contiguous())

	def forward(self, stream: Stream, control: torch.Tensor):
		"""Returns (residual stream x, sublayer output y), both fp32."""
		a = torch.empty((stream.rows, self.down.shape[1]), dtype=self.down.dtype, device=self.down.device)
		x = project_stream(stream, self.gate_up, epilogue(_dense.EPI_SILU, a), control)
		return x, linear(a, self.down, control)
