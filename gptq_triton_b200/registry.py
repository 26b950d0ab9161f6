"""Model registry: which loader and which engine serve a checkpoint, by its config.json."""
from __future__ import annotations

import json
from dataclasses import dataclass
from pathlib import Path
from typing import Callable, Dict, Optional, Tuple

import torch

from . import befalix, lifinex, llama, loader


@dataclass(frozen=True)
class Architecture:
	name: str
	load: Callable                       # (checkpoint, device, dtype) -> model
	engine: Callable                     # (model, batch, max_seq, use_graph=...) -> StaticEngine
	dtypes: Tuple[torch.dtype, ...]      # the first one is the default
	libraries: Tuple[str, ...]           # build targets whose kernels it runs on


ARCHITECTURES: Dict[str, Architecture] = {}


def register(arch: Architecture):
	ARCHITECTURES[arch.name] = arch


register(Architecture('LlamaForCausalLM', lambda ck, device, dtype: loader.load_quant(str(ck), device=device), llama.DecodeEngine, (torch.float16,), ('gptq',)))
register(Architecture(befalix.ARCHITECTURE, befalix.load_befalix, befalix.BefalixEngine, (torch.bfloat16, torch.float32), ('dense',)))
register(Architecture(lifinex.ARCHITECTURE, lifinex.load_lifinex, lifinex.LifinexEngine, (torch.bfloat16, torch.float32), ('dense',)))


def architecture_of(checkpoint) -> Architecture:
	"""config.json names the architecture (`architecture`, or the first of `architectures`); quantised LLaMA checkpoints of the
	reference need not, they are known by their quant_config.json."""
	ck = Path(checkpoint)
	config = json.load(open(ck / 'config.json'))
	name = config.get('architecture') or (config.get('architectures') or [None])[0]
	if name is None and (ck / 'quant_config.json').exists():
		name = 'LlamaForCausalLM'
	if name not in ARCHITECTURES:
		raise ValueError(f'{ck}: architecture {name!r} is not one of {sorted(ARCHITECTURES)}')
	return ARCHITECTURES[name]


def load_model(checkpoint, device='cuda', dtype: Optional[torch.dtype] = None):
	"""Loads any supported checkpoint directory."""
	arch = architecture_of(checkpoint)
	dtype = dtype or arch.dtypes[0]
	if dtype not in arch.dtypes:
		raise ValueError(f'{arch.name} runs in {[str(d) for d in arch.dtypes]}, not {dtype}')
	return arch.load(checkpoint, device, dtype)


def make_engine(model, batch: int, max_seq: int, **kw):
	"""The engine that serves `model` (see StaticEngine)."""
	return ARCHITECTURES[getattr(type(model), 'architecture', 'LlamaForCausalLM')].engine(model, batch=batch, max_seq=max_seq, **kw)
