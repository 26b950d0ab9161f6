"""Befalix: decoder-only language models with latent attention (per-head output gates, layers that may share an earlier
layer's cached rows), SiLU-gated MLPs, post-norm residual sublayers with LayerNorm and layer scale, tied output embedding.

Configuration, weight names and the engine; the mechanisms are in latent_attention.py and dense.py,
what designs with dense weights share in dense_model.py.
"""
from __future__ import annotations

import json
from dataclasses import dataclass
from typing import Dict, List, Optional

import torch
import torch.nn as nn

from .dense import DenseMLP, LayerNorm, PostNorm, Stream
from .dense_model import DenseCausalLM, DenseEngine, load_checkpoint
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


class BefalixForCausalLM(DenseCausalLM):
	"""Inference weights in the kernels' layout, built from a checkpoint's tensors."""
	architecture = ARCHITECTURE

	def __init__(self, config: BefalixConfig, tensors: Dict[str, torch.Tensor], dtype: torch.dtype = torch.bfloat16, device='cuda'):
		super().__init__(config, tensors, dtype, device)
		get = self.reader(tensors, device)
		self.register_buffer('embed', self.table(get('embed')))
		self.layers = nn.ModuleList([BefalixLayer(layer, config, self.reader(tensors, device, f'l{i}.')) for i, layer in enumerate(config.layers)])
		self.norm = LayerNorm(get('final.norm'), get('final.norm.b'))

	@property
	def head(self) -> torch.Tensor:
		return self.embed


def load_befalix(checkpoint, device='cuda', dtype: Optional[torch.dtype] = None) -> BefalixForCausalLM:
	"""Checkpoint directory with config.json and model.safetensors."""
	return load_checkpoint(BefalixForCausalLM, BefalixConfig, checkpoint, device, dtype)


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


class BefalixEngine(DenseEngine):
	"""Static cache of latent rows; a layer that shares another's reads that layer's rows.  A decode step of one sequence is
	seven kernels per layer plus one for the logits and the greedy choice."""

	def __init__(self, model: BefalixForCausalLM, batch: int, max_seq: int, use_graph: bool = True):
		mixers = [layer.mixer for layer in model.config.layers]
		super().__init__(model, batch, max_seq, [m.kv_from if m.kv_from is not None else {'rows': (max_seq, m.row)} for m in mixers], use_graph)
		tables = {}
		for m in mixers:
			if (m.rot_base, m.rot_dims) not in tables:
				tables[m.rot_base, m.rot_dims] = interleaved_rope_tables(m.rot_base, m.rot_dims, max_seq, self.device)
		self.tables = [tables[m.rot_base, m.rot_dims] for m in mixers]

	def _layers(self, token: torch.Tensor, pos: torch.Tensor, rows_per_seq: int, start: Optional[int]) -> Stream:
		m, cfg = self.model, self.cfg
		stream = Stream(cfg.width, m.embed.shape[1], cfg.norm_eps, table=m.embed, token=token)
		for i, layer in enumerate(m.layers):
			x, y = layer.mixer(stream, self.cache[i]['rows'], pos, rows_per_seq, start, self.tables[i], cfg.norm_eps, self.control)
			stream = layer.mixer_norm.join(stream, x, y)
			if layer.mlp is not None:
				x, y = layer.mlp(stream, self.control)
				stream = layer.mlp_norm.join(stream, x, y)
			self._tap(stream)
		return stream
