"""What models with dense weights share: a checkpoint's tensors checked against the configuration, loading from a directory,
and the engine (embedding, layers, logits with the greedy choice) around the layers that each design supplies.
"""
from __future__ import annotations

import warnings
from pathlib import Path
from typing import Callable, Dict, List, Optional, Sequence

import torch
import torch.nn as nn

from . import _dense
from ._lib import ptr
from .cache import StaticCache
from .dense import Stream, epilogue, pad_to, padded, prepare_rows, project_stream
from .engine import StaticEngine


class DenseCausalLM(nn.Module):
	"""Inference weights in the kernels' layout.  A design's class names its `architecture`, takes (config, tensors, dtype, device),
	and leaves `embed` [vocab, padded width], `head` (the same shape; the embedding again when tied) and the final norm `norm`."""
	architecture = ''

	def __init__(self, config, tensors: Dict[str, torch.Tensor], dtype: torch.dtype, device):
		super().__init__()
		if dtype not in _dense.DTYPE_CODE:
			raise ValueError(f'{self.architecture} runs in bfloat16 or float32, not {dtype}')
		self.config, self.dtype = config, dtype
		shapes = config.tensor_shapes()
		missing, extra = sorted(set(shapes) - set(tensors)), sorted(set(tensors) - set(shapes))
		if missing:
			raise ValueError(f'checkpoint tensors do not fit the configuration: missing {missing[:5]}')
		if extra:
			warnings.warn(f'checkpoint tensors that the configuration does not use: {extra[:5]}')
		for name, shape in shapes.items():
			if tuple(tensors[name].shape) != shape:
				raise ValueError(f'{name} has shape {tuple(tensors[name].shape)}, the configuration needs {shape}')

	def reader(self, tensors: Dict[str, torch.Tensor], device, prefix: str = '', dtype: Optional[torch.dtype] = None) -> Callable[[str], torch.Tensor]:
		return lambda name: tensors[prefix + name].to(device=device, dtype=dtype or self.dtype)

	def table(self, t: torch.Tensor) -> torch.Tensor:
		"""Rows of a table or matrix padded to the stream's width."""
		return pad_to(t, t.shape[0], padded(self.config.width)).contiguous()


def load_checkpoint(model_class, config_class, checkpoint, device='cuda', dtype: Optional[torch.dtype] = None) -> DenseCausalLM:
	"""Checkpoint directory with config.json and model.safetensors."""
	from safetensors.torch import load_file
	ck = Path(checkpoint)
	return model_class(config_class.from_json(ck / 'config.json'), load_file(str(ck / 'model.safetensors')), dtype or torch.bfloat16, device)


class DenseEngine(StaticEngine):
	"""A design's engine gives the cache layouts and `_layers`; the configuration has vocab_size, width, norm_eps and (default 1)
	logit_scale."""
	max_portion = 8192
	max_rows = 65535          # rows of a portion over all sequences (a grid dimension of the attention kernels)

	def __init__(self, model: DenseCausalLM, batch: int, max_seq: int, layouts, use_graph: bool = True):
		super().__init__(model, batch, max_seq, model.embed.device, use_graph)
		self.cfg = model.config
		self.max_portion = max(1, min(self.max_portion, self.max_rows // batch))
		self.cache = StaticCache(layouts, batch, model.dtype, self.device)
		# arrival counter and candidates of the greedy choice (8 bytes per row from byte 256), status word at the end
		self.control = _dense.control_buffer(self.device)
		if 256 + 8 * batch > _dense.CONTROL_BYTES - 8:
			raise ValueError(f'batch {batch} is larger than the control buffer provides for')
		self._taps: Optional[List[torch.Tensor]] = None          # tests: receives the residual stream after every layer

	def _carried(self):
		return self.cache.carried

	def _layers(self, token: torch.Tensor, pos: torch.Tensor, rows_per_seq: int, start: Optional[int]) -> Stream:
		"""The residual stream behind the last layer.  token, pos [M], rows_per_seq consecutive rows per sequence; start: the
		portion's first position, None for a decode step (positions are known to the device only)."""
		raise NotImplementedError

	def _tap(self, stream: Stream):
		if self._taps is not None:
			self._taps.append(prepare_rows(stream, self.control, self.model.dtype, True)[1][:, :self.cfg.width].clone())

	def _head(self, stream: Stream, greedy: bool = False) -> torch.Tensor:
		"""Final norm and output projection: fp32 logits [M, vocab] (a view of padded rows).  greedy: the same kernel also
		writes self.tok and advances self.pos."""
		m, cfg = self.model, self.cfg
		logits = torch.empty((stream.rows, padded(cfg.vocab_size)), dtype=torch.float32, device=self.device)
		e = epilogue(_dense.EPI_LOGITS, logits, getattr(cfg, 'logit_scale', 1.0))
		if greedy:
			e.ticket, e.best, e.tok, e.pos_inout = self.control.data_ptr(), self.control.data_ptr() + 256, ptr(self.tok), ptr(self.pos)
		project_stream(stream, m.head, e, self.control, keep=False, final=m.norm)
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
