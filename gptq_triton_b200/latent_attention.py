"""Latent attention: keys and values of a token live in one low-rank row (a normed latent and one rotated key part that all
heads share), which is all that is cached.

Two forms of the same arithmetic: decode steps and short portions fold the key and value up-projections into the query and
the output (the kernels then work on the cached rows alone); longer bf16 portions expand keys and values of the visible
positions with tensor-core matmuls and run a tcgen05 attention kernel over them.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn as nn

from . import _dense
from ._lib import ptr, stream_ptr
from .dense import Stream, epilogue, linear, matmul, pad_to, padded, project_stream

# portions of more rows than this per sequence use the expanded form (bf16)
ABSORBED_MAX_ROWS = 8


@dataclass(frozen=True)
class LatentAttentionSpec:
	heads: int
	dim: int                    # unrotated query / key entries per head
	rot_dim: int                # rotated ones
	vdim: int
	kv_rank: int
	rot_base: float
	rot_dims: int               # entries of the rotated part that rotate (the rest pass unchanged)
	scale: float
	kv_from: Optional[int] = None

	def __post_init__(self):
		if min(self.heads, self.dim, self.rot_dim, self.vdim, self.kv_rank) < 1 or self.rot_dims % 2 or not 0 < self.rot_dims <= self.rot_dim:
			raise ValueError(f'latent attention sizes: {self}')
		if padded(self.kv_rank) > 1024 or padded(self.rot_dim) > 256:
			raise ValueError(f'the latent attention kernels hold latents of up to 1024 and rotated parts of up to 256 entries: {self}')

	@property
	def row(self) -> int:
		"""Entries of a cache row (padded)."""
		return padded(self.kv_rank) + padded(self.rot_dim)


def interleaved_rope_tables(base: float, dims: int, positions: int, device):
	"""cos, sin fp32 [positions, dims / 2] of p * base^(-2 i / dims), from float64 angles."""
	f = float(base) ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)
	a = torch.arange(positions, dtype=torch.float64)[:, None] * f[None, :]
	return a.cos().float().to(device).contiguous(), a.sin().float().to(device).contiguous()


class LatentAttention(nn.Module):
	"""Weights are packed once: query, down-projection and gate rows in one matrix (one pass over the input), all sizes padded
	to multiples of 16 with zeros."""

	def __init__(self, spec: LatentAttentionSpec, q, uk, uv, g, o, dkv=None, dkv_norm=None):
		super().__init__()
		self.spec = spec
		H, D, R, V, C = spec.heads, spec.dim, spec.rot_dim, spec.vdim, spec.kv_rank
		self.D, self.R, self.V, self.C, self.G = padded(D), padded(R), padded(V), padded(C), padded(H)
		width, w = q.shape[1], padded(q.shape[1])
		qh = q.view(H, D + R, width)
		rows = [torch.cat([pad_to(qh[:, :D], H, self.D, w), pad_to(qh[:, D:], H, self.R, w)], dim=1).reshape(H * (self.D + self.R), w)]
		if dkv is not None:
			rows += [pad_to(dkv[:C], self.C, w), pad_to(dkv[C:], self.R, w)]
			self.register_buffer('kv_norm', pad_to(dkv_norm.float(), self.C))
		else:
			self.kv_norm = None
		rows.append(pad_to(g, self.G, w))
		self.register_buffer('w_in', torch.cat(rows).contiguous())
		self.register_buffer('w_uk', pad_to(uk.view(H, D, C), H, self.D, self.C).reshape(H * self.D, self.C).contiguous())
		self.register_buffer('w_uv', pad_to(uv.view(H, V, C), H, self.V, self.C).reshape(H * self.V, self.C).contiguous())
		self.register_buffer('w_o', pad_to(o.view(width, H, V), w, H, self.V).reshape(w, H * self.V).contiguous())

	def forward(self, stream: Stream, cache: torch.Tensor, pos: torch.Tensor, rows_per_seq: int, start: Optional[int], tables, eps: float, control: torch.Tensor):
		"""stream: M = sequences * rows_per_seq rows at positions pos (int32 [M]); cache [sequences, max_seq, row], written here
		unless the layer shares another's.  start: the portion's first position, None for a decode step (positions are known
		to the device only).  Returns (residual stream x, sublayer output y), both fp32."""
		s, dev, dt = self.spec, cache.device, cache.dtype
		M, H = stream.rows, s.heads
		f32 = dt == torch.float32
		expanded = (start is not None and not f32 and rows_per_seq > ABSORBED_MAX_ROWS and s.scale > 0
					and bool(_dense.lib().dense_latent_prefill_ok(self.D, self.R, self.V)))
		n_q = H * (self.D + self.R)
		cos, sin = tables
		max_seq = cache.shape[1]
		q = torch.empty((M, n_q), dtype=torch.bfloat16 if expanded else torch.float32, device=dev)
		kv = torch.empty((M, s.row), dtype=torch.float32, device=dev) if self.kv_norm is not None else None
		gate = torch.empty((M, self.G), dtype=torch.float32, device=dev)
		e = _dense.Epilogue()
		e.mode, e.n_q, e.head_dim, e.rot_at, e.rot_dims = _dense.EPI_QKV, n_q, self.D + self.R, self.D, s.rot_dims
		e.n_kv, e.n_gate = (s.row if kv is not None else 0), self.G
		e.cos_t, e.sin_t, e.pos, e.max_pos = ptr(cos), ptr(sin), ptr(pos), min(cos.shape[0], max_seq)
		e.q_out, e.q_f32, e.kv_out, e.gate_out, e.status = ptr(q), int(not expanded), ptr(kv), ptr(gate), _dense.status_ptr(control)
		x = project_stream(stream, self.w_in, e, control)

		a = self.arguments(cache, pos, rows_per_seq, tables, eps, control, kv)
		lib, code, st = _dense.lib(), _dense.DTYPE_CODE[dt], stream_ptr(dev)
		out = torch.empty((M, H * self.V), dtype=dt, device=dev)
		if expanded:
			if kv is not None:
				_dense.check(lib.dense_latent_append(ctypes.byref(a), code, st), 'dense_latent_append')
			S = start + rows_per_seq
			for b in range(M // rows_per_seq):
				lo = b * rows_per_seq
				self._expanded(q[lo:lo + rows_per_seq], cache[b, :S], gate[lo:lo + rows_per_seq], out[lo:lo + rows_per_seq], start, control)
		else:
			scratch = self.absorbed_buffers(a, q, gate, out, max_seq if start is None else start + rows_per_seq)      # noqa: F841 (alive until the launches)
			_dense.check(lib.dense_latent_absorb(ctypes.byref(a), code, st), 'dense_latent_absorb')
			_dense.check(lib.dense_latent_attend(ctypes.byref(a), code, st), 'dense_latent_attend')
			_dense.check(lib.dense_latent_value(ctypes.byref(a), code, st), 'dense_latent_value')
		return x, linear(out, self.w_o, control)

	def arguments(self, cache, pos, rows_per_seq: int, tables, eps: float, control, kv) -> '_dense.Latent':
		"""Sizes, positions, tables and cache of a call; kv: raw rows to append, or None."""
		s, a = self.spec, _dense.Latent()
		a.M, a.rows_per_seq, a.heads, a.dim, a.rot_dim, a.vdim, a.kv_rank, a.kv_width = pos.numel(), rows_per_seq, s.heads, self.D, self.R, self.V, self.C, s.kv_rank
		a.rot_dims, a.max_seq, a.splits, a.scale, a.eps = s.rot_dims, cache.shape[1], 1, s.scale, eps
		a.pos, a.cos_t, a.sin_t, a.cache, a.status = ptr(pos), ptr(tables[0]), ptr(tables[1]), ptr(cache), _dense.status_ptr(control)
		a.kv_raw, a.kv_norm = ptr(kv), ptr(self.kv_norm)
		return a

	def absorbed_buffers(self, a: '_dense.Latent', q, gate, out, keys: int):
		"""Scratch of the absorbed form for up to `keys` visible positions, entered into `a`; returns what must stay alive."""
		dev, f32 = q.device, out.dtype == torch.float32
		a.splits = _dense.lib().dense_latent_splits(a.M, a.heads, keys, _dense.DTYPE_CODE[out.dtype])
		qa = torch.empty((1 if f32 else 2, a.M, a.heads, self.spec.row), dtype=out.dtype, device=dev)
		ml = torch.empty((a.M, a.heads, a.splits, 2), dtype=torch.float32, device=dev)
		acc = torch.empty((a.M, a.heads, a.splits, self.C), dtype=torch.float32, device=dev)
		a.q, a.w_uk, a.w_uv, a.part_ml, a.part_acc = ptr(q), ptr(self.w_uk), ptr(self.w_uv), ptr(ml), ptr(acc)
		if f32:
			a.qa_f32 = ptr(qa)
		else:
			a.qa_hi, a.qa_lo = ptr(qa[0]), ptr(qa[1])
		a.gate, a.gate_ld, a.out, a.out_ld = ptr(gate), self.G, ptr(out), out.stride(0)
		return qa, ml, acc

	def _expanded(self, q, rows, gate, out, start: int, control):
		"""One sequence: keys and (transposed) values of the cached rows [S, row], then the tensor-core attention kernel."""
		S, H = rows.shape[0], self.spec.heads
		latent = rows[:, :self.C]
		k = torch.empty((S, H * self.D), dtype=torch.bfloat16, device=rows.device)
		matmul(latent, self.w_uk, epilogue(_dense.EPI_T, k), control)
		vt = torch.empty((H * self.V, padded(S)), dtype=torch.bfloat16, device=rows.device)
		matmul(self.w_uv, latent, epilogue(_dense.EPI_T, vt), control)
		p = _dense.LatentPrefill()
		p.t, p.start, p.S, p.heads, p.dim, p.rot_dim, p.vdim, p.kv_rank, p.scale = q.shape[0], start, S, H, self.D, self.R, self.V, self.C, self.spec.scale
		p.q, p.k, p.vt, p.ldv, p.cache = ptr(q), ptr(k), ptr(vt), vt.stride(0), ptr(rows)
		p.gate, p.gate_ld, p.out, p.out_ld, p.status = ptr(gate), gate.stride(0), ptr(out), out.stride(0), _dense.status_ptr(control)
		_dense.check(_dense.lib().dense_latent_prefill(ctypes.byref(p), stream_ptr(rows.device)), 'dense_latent_prefill')
