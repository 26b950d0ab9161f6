"""Lifinex: decoder-only language models that mix differential attention and state-space layers, with a block of layers that
runs several times on the same weights, learned positions, pre-norm sublayers and a per-token input to every layer.

Configuration, weight names and the engine; the mechanisms are in gqa_attention.py, ssm.py and dense.py, what designs with
dense weights share in dense_model.py.
"""
from __future__ import annotations

import json
from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple, Union

import torch
import torch.nn as nn

from . import _dense
from .dense import DenseMLP, RMSNorm, Stream, TokenSide, epilogue, pad_to, padded, project_stream
from .dense_model import DenseCausalLM, DenseEngine, load_checkpoint
from .gqa_attention import GroupedAttention, GroupedAttentionSpec, diff_lambda
from .ssm import StateSpaceMixer, StateSpaceSpec

ARCHITECTURE = 'Lifinex'


@dataclass(frozen=True)
class LifinexLayerConfig:
	mixer: Union[GroupedAttentionSpec, StateSpaceSpec]
	ff: Optional[int]                    # None: a layer without a feed-forward


@dataclass(frozen=True)
class LoopConfig:
	"""Layers start .. stop - 1 run `times` times in a row."""
	start: int
	stop: int
	times: int


def _mixer(i: int, kind: str, m: dict):
	if kind == 'attention':
		return GroupedAttentionSpec(heads=m['heads'], kv_heads=m['kv_heads'], dim=m['dim'], vdim=m['vdim'], scale=m['scale'], softcap=m.get('softcap'), maps=2, diff=m['diff'])
	if kind == 'mamba2':
		return StateSpaceSpec(heads=m['heads'], vdim=m['vdim'], state=m['state'], groups=m['groups'], taps=m['conv'], norm_groups=m['norm_groups'])
	raise ValueError(f"layer {i}: mixer '{kind}' is not part of this design")


@dataclass(frozen=True)
class LifinexConfig:
	vocab_size: int
	width: int
	layers: List[LifinexLayerConfig]
	norm_eps: float
	max_positions: int
	side_dim: Optional[int] = None
	loop: Optional[LoopConfig] = None

	def __post_init__(self):
		l = self.loop
		if l is not None and not (0 <= l.start < l.stop <= len(self.layers) and l.times >= 1):
			raise ValueError(f'{l} does not fit {len(self.layers)} layers')

	@classmethod
	def from_dict(cls, d: dict) -> 'LifinexConfig':
		layers = []
		for i, layer in enumerate(d['layers']):
			mlp = layer.get('mlp')
			if mlp is not None and mlp['kind'] != 'dense':
				raise ValueError(f"layer {i}: feed-forward '{mlp['kind']}' is not part of this design")
			layers.append(LifinexLayerConfig(_mixer(i, layer['type'], layer['mixer']), None if mlp is None else mlp['ff']))
		side, loop = d.get('token_side'), d.get('loop')
		return cls(d['vocab'], d['width'], layers, d['norm']['eps'], d['max_positions'], None if side is None else side['dim'],
				   None if loop is None else LoopConfig(loop['start'], loop['stop'], loop['times']))

	@classmethod
	def from_json(cls, path) -> 'LifinexConfig':
		return cls.from_dict(json.load(open(path)))

	def runs(self) -> List[Tuple[int, Optional[int]]]:
		"""Layers in the order in which they run: (layer, number of the pass that begins with it, or None)."""
		n, l = len(self.layers), self.loop
		if l is None:
			return [(i, None) for i in range(n)]
		body = [(i, t if i == l.start else None) for t in range(l.times) for i in range(l.start, l.stop)]
		return [(i, None) for i in range(l.start)] + body + [(i, None) for i in range(l.stop, n)]

	def tensor_shapes(self) -> Dict[str, tuple]:
		"""Names and shapes of a checkpoint's tensors."""
		w = self.width
		out = {'embed': (self.vocab_size, w), 'pos': (self.max_positions, w), 'head': (self.vocab_size, w), 'final.norm': (w,)}
		if self.loop is not None:
			out['loop.in'] = (w, 2 * w)
			out['loop.step'] = (self.loop.times, w)
		if self.side_dim is not None:
			out['side.embed'] = (self.vocab_size, len(self.layers) * self.side_dim)
		for i, layer in enumerate(self.layers):
			m, p = layer.mixer, f'l{i}.'
			out[p + 'norm1'] = (w,)
			if isinstance(m, GroupedAttentionSpec):
				out[p + 'mix.q'] = (m.heads * m.maps * m.dim, w)
				out[p + 'mix.k'] = (m.kv_heads * m.maps * m.dim, w)
				out[p + 'mix.v'] = (m.kv_heads * m.vdim, w)
				for n in ('q.norm', 'k.norm', 'lq1', 'lk1', 'lq2', 'lk2'):
					out[p + 'mix.' + n] = (m.dim,)
				out[p + 'mix.o'] = (w, m.heads * m.vdim)
			else:
				out[p + 'mix.in'] = (m.inner + m.channels + m.heads, w)
				out[p + 'mix.conv'] = (m.channels, m.taps)
				out[p + 'mix.conv.b'] = (m.channels,)
				for n in ('dt_bias', 'A_log', 'D'):
					out[p + 'mix.' + n] = (m.heads,)
				out[p + 'mix.norm'] = (m.inner,)
				out[p + 'mix.o'] = (w, m.inner)
			if layer.ff is not None:
				out[p + 'norm2'] = (w,)
				out[p + 'mlp.gate'] = out[p + 'mlp.up'] = (layer.ff, w)
				out[p + 'mlp.down'] = (w, layer.ff)
			if self.side_dim is not None:
				out[p + 'side.gate'] = (self.side_dim, w)
				out[p + 'side.proj'] = (w, self.side_dim)
				out[p + 'side.norm'] = (w,)
		return out


class LifinexLayer(nn.Module):
	"""get: a weight in the model's dtype; get32: in fp32."""

	def __init__(self, i: int, layer: LifinexLayerConfig, config: LifinexConfig, get, get32):
		super().__init__()
		m = layer.mixer
		self.mixer_norm = RMSNorm(get32('norm1'), offset=1.0)
		if isinstance(m, GroupedAttentionSpec):
			lam = diff_lambda(*(get32('mix.' + n) for n in ('lq1', 'lk1', 'lq2', 'lk2')), m.diff)
			self.mixer = GroupedAttention(m, get('mix.q'), get('mix.k'), get('mix.v'), get('mix.o'), get32('mix.q.norm'), get32('mix.k.norm'), lam)
		else:
			self.mixer = StateSpaceMixer(m, get('mix.in'), get32('mix.conv'), get32('mix.conv.b'), get32('mix.dt_bias'), get32('mix.A_log'), get32('mix.D'), get32('mix.norm'),
										 get('mix.o'))
		self.mlp = self.mlp_norm = self.side = None
		if layer.ff is not None:
			self.mlp_norm = RMSNorm(get32('norm2'), offset=1.0)
			self.mlp = DenseMLP(get('mlp.gate'), get('mlp.up'), get('mlp.down'), act='gelu_tanh')
		if config.side_dim is not None:
			self.side = TokenSide(get('side.gate'), get('side.proj'), get32('side.norm'), column=i * padded(config.side_dim))


class LifinexForCausalLM(DenseCausalLM):
	"""Inference weights in the kernels' layout, built from a checkpoint's tensors."""
	architecture = ARCHITECTURE

	def __init__(self, config: LifinexConfig, tensors: Dict[str, torch.Tensor], dtype: torch.dtype = torch.bfloat16, device='cuda'):
		super().__init__(config, tensors, dtype, device)
		get, get32 = self.reader(tensors, device), self.reader(tensors, device, dtype=torch.float32)
		width, w = config.width, padded(config.width)
		self.register_buffer('embed', self.table(get('embed')))
		self.register_buffer('pos', self.table(get('pos')))
		self.register_buffer('head', self.table(get('head')))
		if config.loop is not None:
			# the pass entry W [x; x0] in two halves: the part of the embedding output is the same for every pass
			self.register_buffer('loop_x', pad_to(get('loop.in')[:, :width], w, w).contiguous())
			self.register_buffer('loop_x0', pad_to(get('loop.in')[:, width:], w, w).contiguous())
			self.register_buffer('loop_step', self.table(get32('loop.step')))
		if config.side_dim is not None:
			n, d = len(config.layers), config.side_dim
			self.register_buffer('side', pad_to(get('side.embed').view(config.vocab_size, n, d), config.vocab_size, n, padded(d)).reshape(config.vocab_size, n * padded(d)).contiguous())
		else:
			self.side = None
		self.layers = nn.ModuleList([LifinexLayer(i, layer, config, self.reader(tensors, device, f'l{i}.'), self.reader(tensors, device, f'l{i}.', torch.float32))
									 for i, layer in enumerate(config.layers)])
		self.norm = RMSNorm(get32('final.norm'), offset=1.0)


def load_lifinex(checkpoint, device='cuda', dtype: Optional[torch.dtype] = None) -> LifinexForCausalLM:
	"""Checkpoint directory with config.json and model.safetensors."""
	return load_checkpoint(LifinexForCausalLM, LifinexConfig, checkpoint, device, dtype)


@torch.no_grad()
def synthetic_lifinex(config: LifinexConfig, seed: int = 0, device='cuda', dtype: torch.dtype = torch.bfloat16) -> LifinexForCausalLM:
	"""Random weights of the given configuration, scaled so that activations stay near unit variance."""
	gen = torch.Generator(device=device).manual_seed(seed)
	tensors = {}
	for name, shape in config.tensor_shapes().items():
		t = torch.randn(shape, generator=gen, device=device)
		short = name.split('.', 1)[-1]
		if short == 'mix.dt_bias':
			t = t - 3.0
		elif short == 'mix.A_log':
			t = 0.5 * t + 0.5
		elif short in ('mix.q.norm', 'mix.k.norm', 'mix.norm', 'side.norm', 'mix.D'):
			t = 1.0 + 0.1 * t
		elif len(shape) == 1:
			t = 0.1 * t
		elif name not in ('embed', 'pos', 'side.embed', 'loop.step'):
			t = t * shape[1] ** -0.5
		tensors[name] = t.to(dtype)
	return LifinexForCausalLM(config, tensors, dtype, device)


class LifinexEngine(DenseEngine):
	"""Cached keys and values of attention layers, carried state of state-space layers; a layer that runs several times has its
	own of each run.  Sequences are at most as long as the table of positions."""

	def __init__(self, model: LifinexForCausalLM, batch: int, max_seq: int, use_graph: bool = True):
		cfg = model.config
		max_seq = min(max_seq, cfg.max_positions)
		self.runs = cfg.runs()
		mixers = [cfg.layers[i].mixer for i, _ in self.runs]
		super().__init__(model, batch, max_seq, [m.cache_layout(max_seq) if isinstance(m, GroupedAttentionSpec) else m.cache_layout() for m in mixers], use_graph)

	def _layers(self, token: torch.Tensor, pos: torch.Tensor, rows_per_seq: int, start: Optional[int]) -> Stream:
		m, cfg, ctl = self.model, self.cfg, self.control
		stream = Stream(cfg.width, m.embed.shape[1], cfg.norm_eps, table=m.embed, token=token, pos_table=m.pos, pos=pos)
		project = lambda w: self._plain(stream, w)
		from_x0 = project(m.loop_x0) if cfg.loop is not None else None
		for run, (i, entry) in enumerate(self.runs):
			layer = m.layers[i]
			if entry is not None:
				stream = stream.then(from_x0, project(m.loop_x), shift=m.loop_step[entry])
			x, y = layer.mixer(stream, self.cache[run], pos, rows_per_seq, start, ctl, norm=layer.mixer_norm)
			stream = stream.then(x, y)
			if layer.mlp is not None:
				x, y = layer.mlp(stream, ctl, norm=layer.mlp_norm)
				stream = stream.then(x, y)
			if layer.side is not None:
				stream = layer.side(stream, m.side, token, ctl)
			self._tap(stream)
		return stream

	def _plain(self, stream: Stream, w: torch.Tensor) -> torch.Tensor:
		"""x W^T of the stream itself, fp32 [M, rows of w]."""
		out = torch.empty((stream.rows, w.shape[0]), dtype=torch.float32, device=self.device)
		project_stream(stream, w, epilogue(_dense.EPI_F32, out), self.control, keep=False)
		return out
