"""Static per-layer cache of an engine: fixed rows for `batch` sequences of up to `max_seq` positions, written in place, and
recurrent state that a step carries on.

A layer's layout names its tensors and gives their shapes behind the batch dimension (`Carried` for fp32 state that every
token overwrites); a layer that reads what an earlier layer has cached (shared keys and values) gives that layer's number instead
and owns nothing.  A layer that runs several times in one forward pass has an entry per run.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Sequence, Tuple, Union

import torch


@dataclass(frozen=True)
class Carried:
	"""Shape of a recurrent state (fp32)."""
	shape: Tuple[int, ...]


Layout = Union[int, Dict[str, Union[Tuple[int, ...], Carried]]]


class StaticCache:
	def __init__(self, layouts: Sequence[Layout], batch: int, dtype: torch.dtype, device):
		self.layers: List[Dict[str, torch.Tensor]] = []
		self.carried: List[torch.Tensor] = []          # what a step overwrites (running one twice is not the same as once)
		for i, lay in enumerate(layouts):
			if isinstance(lay, int):
				if not 0 <= lay < i or isinstance(layouts[lay], int):
					raise ValueError(f'layer {i} cannot share the cache of layer {lay}: that must be an earlier layer with a cache of its own')
				self.layers.append(self.layers[lay])
			else:
				entry = {}
				for name, shape in lay.items():
					if isinstance(shape, Carried):
						entry[name] = torch.zeros((batch, *shape.shape), dtype=torch.float32, device=device)
						self.carried.append(entry[name])
					else:
						entry[name] = torch.zeros((batch, *shape), dtype=dtype, device=device)
				self.layers.append(entry)

	def __getitem__(self, layer: int) -> Dict[str, torch.Tensor]:
		return self.layers[layer]

	def __len__(self) -> int:
		return len(self.layers)

	def tensors(self, name: str) -> List[torch.Tensor]:
		"""The tensor `name` of every layer (the same object for layers that share)."""
		return [layer[name] for layer in self.layers]

	def nbytes(self) -> int:
		seen = {t.data_ptr(): t.numel() * t.element_size() for layer in self.layers for t in layer.values()}
		return sum(seen.values())
