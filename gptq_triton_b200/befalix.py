"""Befalix: decoder-only language models with latent attention (per-head output gates, layers that may share an earlier
layer's cached rows), SiLU-gated MLPs, post-norm residual sublayers with LayerNorm and layer scale, tied output embedding.

Configuration, weight names and the engine; the mechanisms are in latent_attention.py and dense.py.
"""
from __future__ import annotations

import json
import warnings
from dataclasses import dataclass
from pathlib import Path
from typing import Dict, List, Optional, Sequence

import torch
import torch.nn as nn

from . import _dense
from ._lib import ptr
from .cache import StaticCache
from .dense import DenseMLP, LayerNorm, PostNorm, Stream, epilogue, pad_to, padded, project_stream
from .engine import StaticEngine
from .latent_attention import LatentAttention, LatentAttentionSpec, interleaved_rope_tables

ARCHITECTURE = 'Befalix'


@dataclass(frozen=True)
class BefalixLayerConfig:
	mixer: LatentAttentionSpec
	ff: Optional[int]                    # None: a layer without a feed-forward


@dataclass(frozen=True)
class BefalixConfig:
	vocab_size: int
	width: int
	layers: List[BefalixLayerConfig]
	norm_eps: float
	residual_mult: float
	logit_scale: float

	@classmethod
	def from_dict(cls, d: dict) -> 'BefalixConfig':
		layers = []
		for i, layer in enumerate(d['layers']):
			if layer['type'] != 'latent_attention':
				raise ValueError(f"layer {i}: mixer '{layer['type']}' is not part of this design")
			m, mlp = layer['mixer'], layer.get('mlp')
			if mlp is not None and mlp['kind'] != 'dense':
				raise ValueError(f"layer {i}: feed-forward '{mlp['kind']}' is not part of this design")
			spec = LatentAttentionSpec(heads=m['heads'], dim=m['dim'], rot_dim=m['rot_dim'], vdim=m['vdim'], kv_rank=m['kv_rank'], rot_base=m['rot']['base'],
									   rot_dims=m['rot']['dims'], scale=m['scale'], kv_from=m.get('kv_from'))
			if spec.kv_from is not None:
				src = layers[spec.kv_from].mixer if 0 <= spec.kv_from < i else None
				if src is None or src.kv_from is not None or (src.kv_rank, src.rot_dim, src.rot_base, src.rot_dims) != (spec.kv_rank, spec.rot_dim, spec.rot_base, spec.rot_dims):
					raise ValueError(f'layer {i} cannot read the cache of layer {spec.kv_from}')
			layers.append(BefalixLayerConfig(spec, None if mlp is None else mlp['ff']))
		return cls(d['vocab'], d['width'], layers, d['norm']['eps'], d['residual_mult'], d['logit_scale'])

	@classmethod
	def from_json(cls, path) -> 'BefalixConfig':
		return cls.from_dict(json.load(open(path)))

	def tensor_shapes(self) -> Dict[str, tuple]:
		"""Names and shapes of a checkpoint's tensors."""
		w = self.width
		out = {'embed': (self.vocab_size, w), 'final.norm': (w,), 'final.norm.b': (w,)}
		for i, layer in enumerate(self.layers):
			m, p = layer.mixer, f'l{i}.'
			out[p + 'mix.q'] = (m.heads * (m.dim + m.rot_dim), w)
			if m.kv_from is None:
				out[p + 'mix.dkv'] = (m.kv_rank + m.rot_dim, w)
				out[p + 'mix.dkv.norm'] = (m.kv_rank,)
			out[p + 'mix.uk'] = (m.heads * m.dim, m.kv_rank)
			out[p + 'mix.uv'] = (m.heads * m.vdim, m.kv_rank)
			out[p + 'mix.g'] = (m.heads, w)
			out[p + 'mix.o'] = (w, m.heads * m.vdim)
			subs = [1]
			if layer.ff is not None:
				out[p + 'mlp.gate'] = out[p + 'mlp.up'] = (layer.ff, w)
				out[p + 'mlp.down'] = (w, layer.ff)
				subs.append(2)
			for n in subs:
				out[f'{p}norm{n}'] = out[f'{p}norm{n}.b'] = out[f'{p}ls{n}'] = (w,)
		return out


class BefalixLayer(nn.Module):
	def __init__(self, layer: BefalixLayerConfig, config: BefalixConfig, get):
		super().__init__()
		own = layer.mixer.kv_from is None
		self.mixer = LatentAttention(layer.mixer, get('mix.q'), get('mix.uk'), get('mix.uv'), get('mix.g'), get('mix.o'),
									 get('mix.dkv') if own else None, get('mix.dkv.norm') if own else None)
		self.mixer_norm = PostNorm(get('norm1'), get('norm1.b'), get('ls1'), config.residual_mult)
		self.mlp = self.mlp_norm = None
		if layer.ff is not None:
			self.mlp = DenseMLP(get('mlp.gate'), get('mlp.up'), get('mlp.down'))
			self.mlp_norm = PostNorm(get('norm2'), get('norm2.b'), get('ls2'), config.residual_mult)


class BefalixForCausalLM(nn.Module):
	"""Inference weights in the kernels' layout, built from a checkpoint's tensors."""
	architecture = ARCHITECTURE

	def __init__(self, config: BefalixConfig, tensors: Dict[str, torch.Tensor], dtype: torch.dtype = torch.bfloat16, device='cuda'):
		super().__init__()
		if dtype not in _dense.DTYPE_CODE:
			raise ValueError(f'{ARCHITECTURE} runs in bfloat16 or float32, not {dtype}')
		self.config, self.dtype = config, dtype
		shapes = config.tensor_shapes()
		missing, extra = sorted(set(shapes) - set(tensors)), sorted(set(tensors) - set(shapes))
		if missing:
			raise ValueError(f'checkpoint tensors do not fit the configuration: missing {missing[:5]}')
		if extra:
			warnings.warn(f'checkpoint tensors that the configuration does not use: {extra[:5]}')

		def get(name):
			if tuple(tensors[name].shape) != shapes[name]:
				raise ValueError(f'{name} has shape {tuple(tensors[name].shape)}, the configuration needs {shapes[name]}')
			return tensors[name].to(device=device, dtype=dtype)
		self.register_buffer('embed', pad_to(get('embed'), config.vocab_size, padded(config.width)).contiguous())
		self.layers = nn.ModuleList([BefalixLayer(layer, config, lambda n, i=i: get(f'l{i}.{n}')) for i, layer in enumerate(config.layers)])
		self.norm = LayerNorm(get('final.norm'), get('final.norm.b'))


def load_befalix(checkpoint, device='cuda', dtype: Optional[torch.dtype] = None) -> BefalixForCausalLM:
	"""Checkpoint directory with config.json and model.safetensors."""
	from safetensors.torch import load_file
	ck = Path(checkpoint)
	return BefalixForCausalLM(BefalixConfig.from_json(ck / 'config.json'), load_file(str(ck / 'model.safetensors')), dtype or torch.bfloat16, device)


@torch.no_grad()
def synthetic_befalix(config: BefalixConfig, seed: int = 0, device='cuda', dtype: torch.dtype = torch.bfloat16) -> BefalixForCausalLM:
	"""Random weights of the given configuration, scaled so that activations stay near unit variance."""
	gen = torch.Generator(device=device).manual_seed(seed)
	tensors = {}
	for name, shape in config.tensor_shapes().items():
		t = torch.randn(shape, generator=gen, device=device)
		if len(shape) == 2:
			t *= shape[1] ** -0.5 if name != 'embed' else 1.0
		elif name.endswith('.b'):
			t *= 0.1
		else:
			t = 1.0 + 0.1 * t
		tensors[name] = t.to(dtype)
	return BefalixForCausalLM(config, tensors, dtype, device)


class BefalixEngine(StaticEngine):
	"""Static cache of latent rows; a layer that shares another's reads that layer's rows.  A decode step of one sequence is
	seven kernels per layer plus one for the logits and the greedy choice."""
	max_portion = 8192

	def __init__(self, model: BefalixForCausalLM, batch: int, max_seq: int, use_graph: bool = True):
		super().__init__(model, batch, max_seq, model.embed.device, use_graph)
		cfg = model.config
		self.cfg = cfg
		mixers = [layer.mixer for layer in cfg.layers]
		self.cache = StaticCache([m.kv_from if m.kv_from is not None else {'rows': (max_seq, m.row)} for m in mixers], batch, model.dtype, self.device)
		tables = {}
		for m in mixers:
			if (m.rot_base, m.rot_dims) not in tables:
				tables[m.rot_base, m.rot_dims] = interleaved_rope_tables(m.rot_base, m.rot_dims, max_seq, self.device)
		self.tables = [tables[m.rot_base, m.rot_dims] for m in mixers]
		# arrival counter and candidates of the greedy choice (8 bytes per row from byte 256), status word at the end
		self.control = _dense.control_buffer(self.device)
		if 256 + 8 * batch > _dense.CONTROL_BYTES - 8:
			raise ValueError(f'batch {batch} is larger than the control buffer provides for')
		self._taps = None          # tests: a list that receives the residual stream after every layer

	def _layers(self, token: torch.Tensor, pos: torch.Tensor, rows_per_seq: int, start: Optional[int]) -> Stream:
		m, cfg = self.model, self.cfg
		stream = Stream(cfg.width, m.embed.shape[1], cfg.norm_eps, table=m.embed, token=token)
		for i, layer in enumerate(m.layers):
			x, y = layer.mixer(stream, self.cache[i]['rows'], pos, rows_per_seq, start, self.tables[i], cfg.norm_eps, self.control)
			stream = layer.mixer_norm.join(stream, x, y)
			if layer.mlp is not None:
				x, y = layer.mlp(stream, self.control)
				stream = layer.mlp_norm.join(stream, x, y)
			if self._taps is not None:
				from .dense import prepare_rows
				self._taps.append(prepare_rows(stream, self.control, m.dtype, True)[1][:, :cfg.width].clone())
		return stream

	def _head(self, stream: Stream, greedy: bool = False) -> torch.Tensor:
		"""Final norm and tied output projection: fp32 logits [M, vocab] (a view of padded rows).  greedy: the same kernel
		also writes self.tok and advances self.pos."""
		m, cfg = self.model, self.cfg
		logits = torch.empty((stream.rows, padded(cfg.vocab_size)), dtype=torch.float32, device=self.device)
		e = epilogue(_dense.EPI_LOGITS, logits, cfg.logit_scale)
		if greedy:
			e.ticket, e.best, e.tok, e.pos_inout = self.control.data_ptr(), self.control.data_ptr() + 256, ptr(self.tok), ptr(self.pos)
		project_stream(stream, m.embed, e, self.control, keep=False, final=m.norm)
		return logits[:, :cfg.vocab_size]

	def _portion(self, input_ids: torch.Tensor, start: int, want: Sequence[int]) -> Optional[torch.Tensor]:
		b, t = input_ids.shape
		pos = torch.arange(start, start + t, device=self.device, dtype=torch.int32).repeat(b)
		stream = self._layers(input_ids.reshape(-1).contiguous(), pos, t, start)
		if not want:
			return None
		index = (torch.arange(b, device=self.device)[:, None] * t + torch.tensor(list(want), device=self.device)[None, :]).reshape(-1)
		return self._head(stream.take(index)).reshape(b, len(want), -1)

	def _step_body(self):
		stream = self._layers(self.tok.view(-1), self.pos.view(-1), 1, None)
		greedy = bool(_dense.lib().dense_decode_rows_ok(self.batch, stream.ld, _dense.DTYPE_CODE[self.model.dtype]))
		self.logits = self._head(stream, greedy).view(self.batch, 1, -1)
		if not greedy:
			self.tok.copy_(self.logits.argmax(-1))
			self.pos.add_(1)
