"""Selective state-space mixer (Mamba-2): a gated linear recurrence per head behind a short causal convolution.

A sequence carries its state (heads x value entries x state entries, fp32) and the convolution's last inputs from token to
token; nothing else is cached, whatever the length.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn as nn

from . import _dense
from ._lib import ptr, stream_ptr
from .cache import Carried
from .dense import Norm, RMSNorm, Stream, epilogue, pad_to, padded, project_stream


# portions of more rows than this per sequence run in chunks (bf16)
STEP_MAX_ROWS = 8


@dataclass(frozen=True)
class StateSpaceSpec:
	heads: int
	vdim: int
	state: int
	groups: int                 # heads of a group share B and C
	taps: int                   # of the convolution, the current token included
	norm_groups: int            # equal parts of the gated output, each normed on its own

	def __post_init__(self):
		if min(self.heads, self.vdim, self.state, self.groups, self.taps, self.norm_groups) < 1 or self.heads % self.groups or self.inner % self.norm_groups:
			raise ValueError(f'state-space sizes: {self}')
		if self.state > 256 or self.taps > 16 or self.norm_groups > _dense.MAX_NORM_GROUPS:
			raise ValueError(f'the state-space kernels hold states of up to 256 entries per value, 16 taps and {_dense.MAX_NORM_GROUPS} norm groups: {self}')

	@property
	def inner(self) -> int:
		return self.heads * self.vdim

	@property
	def channels(self) -> int:
		"""Channels of the convolution: values, B, C."""
		return self.inner + 2 * self.groups * self.state

	def cache_layout(self):
		return {'ring': Carried((self.taps, padded(self.channels))), 's': Carried((self.heads, self.vdim, self.state))}


class StateSpaceMixer(nn.Module):
	"""w_in: rows [z | x, B, C | dt], every section padded to a multiple of 16."""

	def __init__(self, spec: StateSpaceSpec, w_in, conv, conv_b, dt_bias, a_log, d, norm_w, w_o):
		super().__init__()
		self.spec = spec
		width, w = w_in.shape[1], padded(w_in.shape[1])
		z, xbc, dt = w_in.split([spec.inner, spec.channels, spec.heads])
		self.register_buffer('w_in', torch.cat([pad_to(t, padded(t.shape[0]), w) for t in (z, xbc, dt)]).contiguous())
		self.conv_at = padded(spec.inner)
		self.dt_at = self.conv_at + padded(spec.channels)
		ld = padded(spec.channels)
		self.register_buffer('conv_w', pad_to(conv.float().t(), spec.taps, ld).contiguous())
		self.register_buffer('conv_b', pad_to(conv_b.float(), ld))
		self.register_buffer('dt_bias', dt_bias.float().contiguous())
		self.register_buffer('a', -a_log.double().exp().float().contiguous())
		self.register_buffer('d', d.float().contiguous())
		self.register_buffer('w_o', pad_to(w_o, w, padded(spec.inner)).contiguous())
		self.norm = RMSNorm(norm_w, parts=spec.norm_groups)

	def forward(self, stream: Stream, cache, pos: torch.Tensor, rows_per_seq: int, start: Optional[int], control: torch.Tensor, norm: Optional[Norm] = None):
		"""As GroupedAttention.forward; cache: ring and s, carried on here."""
		s, dev, M, dt = self.spec, control.device, stream.rows, self.w_in.dtype
		chunked = dt == torch.bfloat16 and rows_per_seq > STEP_MAX_ROWS
		n, n_dt = self.dt_at, self.w_in.shape[0] - self.dt_at
		# one matrix product; the step sizes stay fp32 when the rest becomes bf16
		raw = torch.empty((M, n if chunked else n + n_dt), dtype=dt if chunked else torch.float32, device=dev)
		steps = torch.empty((M, n_dt), dtype=torch.float32, device=dev) if chunked else raw[:, n:]
		e = epilogue(_dense.EPI_MIXED if chunked else _dense.EPI_F32, raw)
		if chunked:
			e.n_q, e.n_kv, e.kv_out = n, n_dt, ptr(steps)
		x = project_stream(stream, self.w_in, e, control, final=norm)
		inner = padded(s.inner)
		out = (torch.empty if inner == s.inner else torch.zeros)((M, inner), dtype=raw.dtype, device=dev)
		a = self.arguments(raw, steps, cache, pos, rows_per_seq, out, control)
		lib, st = _dense.lib(), stream_ptr(dev)
		if rows_per_seq == 1:
			_dense.check(lib.dense_ssm_step(ctypes.byref(a), st), 'dense_ssm_step')
		else:
			scratch = self.portion_buffers(a, raw.dtype, chunked)      # noqa: F841 (alive until the launches)
			_dense.check(lib.dense_ssm_conv(ctypes.byref(a), _dense.DTYPE_CODE[raw.dtype], st), 'dense_ssm_conv')
			if chunked:
				kernels = 3 if lib.dense_ssm_chunked_scratch(ctypes.byref(a)) else M // rows_per_seq
				_dense.check(lib.dense_ssm_chunked(ctypes.byref(a), st), 'dense_ssm_chunked', kernels)
			else:
				_dense.check(lib.dense_ssm_scan(ctypes.byref(a), st), 'dense_ssm_scan')
		y = torch.empty((M, self.w_o.shape[0]), dtype=torch.float32, device=dev)
		project_stream(Stream(s.inner, inner, stream.eps, x=out), self.w_o, epilogue(_dense.EPI_F32, y), control, keep=False, final=self.norm)
		return x, y

	def arguments(self, raw, steps, cache, pos, rows_per_seq: int, out, control) -> '_dense.Ssm':
		s, a = self.spec, _dense.Ssm()
		a.M, a.rows_per_seq, a.heads, a.vdim, a.state, a.groups, a.taps = pos.numel(), rows_per_seq, s.heads, s.vdim, s.state, s.groups, s.taps
		a.z_at, a.conv_at, a.conv_ld, a.raw_ld, a.dt_ld = 0, self.conv_at, padded(s.channels), raw.stride(0), steps.stride(0)
		a.raw, a.dt, a.pos, a.conv_w, a.conv_b, a.dt_bias, a.a, a.d = ptr(raw), ptr(steps), ptr(pos), ptr(self.conv_w), ptr(self.conv_b), ptr(self.dt_bias), ptr(self.a), ptr(self.d)
		a.ring, a.s, a.out, a.out_ld, a.status = ptr(cache['ring']), ptr(cache['s']), ptr(out), out.stride(0), _dense.status_ptr(control)
		return a

	def portion_buffers(self, a: '_dense.Ssm', dtype: torch.dtype, chunked: bool):
		"""Scratch of a portion, entered into `a`; returns what must stay alive."""
		s, dev = self.spec, self.w_in.device
		u = torch.empty((a.M, a.conv_ld), dtype=dtype, device=dev)
		a.u = ptr(u)
		if not chunked:
			return (u,)
		if not _dense.lib().dense_ssm_chunked_scratch(ctypes.byref(a)):
			return (u,)
		n = a.M // a.rows_per_seq * ((a.rows_per_seq + _dense.SSM_CHUNK - 1) // _dense.SSM_CHUNK)
		states = torch.empty((n, s.heads, s.vdim, s.state), dtype=torch.float32, device=dev)
		decay = torch.empty((n, s.heads), dtype=torch.float32, device=dev)
		a.chunk_s, a.chunk_decay = ptr(states), ptr(decay)
		return u, states, decay
