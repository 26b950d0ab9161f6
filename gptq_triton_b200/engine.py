"""The generation loop that every model of the framework runs in: a static cache, positions and tokens on the device, prompts
in one piece or in portions, decode steps captured in a CUDA graph, greedy sampling on the device.

A model's engine subclasses StaticEngine and supplies the cache layout, `_portion` (several tokens per sequence) and
`_step_body` (one token per sequence, capturable).
"""
from __future__ import annotations

import os
from typing import List, Optional, Sequence

import torch


class StaticEngine:
	# tokens per sequence that one `_portion` call gets at most; longer prompts are cut by feed()
	max_portion = 1 << 30

	def __init__(self, model, batch: int, max_seq: int, device, use_graph: bool = True):
		self.model = model
		self.batch, self.max_seq, self.device = batch, max_seq, device
		self.use_graph = use_graph
		self.pos = torch.zeros((batch, 1), dtype=torch.int32, device=device)          # position of the token being fed
		self.tok = torch.zeros((batch, 1), dtype=torch.int64, device=device)          # token being fed
		self.logits: Optional[torch.Tensor] = None
		self.graph = None
		self.graph_logits: Optional[torch.Tensor] = None
		self.launches_per_step = None
		# captures of the decode step to choose from (see step()); 1 = take the first
		self.graph_candidates = int(os.environ.get('GPTQ_B200_GRAPH_CANDIDATES', '6'))
		self.next_pos = 0          # host-side copy of the position the next step() writes (the cache has max_seq rows)

	# -- what a model supplies ---------------------------------------------------------------------
	def _portion(self, input_ids: torch.Tensor, start: int, want: Sequence[int]) -> Optional[torch.Tensor]:
		"""Runs [b, t] tokens at positions start .. start + t - 1, fills the cache, returns the logits [b, len(want), vocab] at
		the places `want` of the portion (None when nothing is wanted)."""
		raise NotImplementedError

	def _step_body(self):
		"""One decode step: feeds self.tok at self.pos, sets self.logits, then self.tok to the arg-max and self.pos to the next
		position, all on the device."""
		raise NotImplementedError

	def _before_capture(self):
		pass

	def _carried(self) -> List[torch.Tensor]:
		"""Recurrent state that a step overwrites: put back after the trial runs of a capture."""
		return []

	def _restore(self, tok: torch.Tensor, pos: torch.Tensor):
		self.tok.copy_(tok)
		self.pos.copy_(pos)

	# -- the loop ----------------------------------------------------------------------------------
	def reset(self):
		"""Gives the cache rows back: the next tokens start new sequences at position 0.  Rows of earlier sequences are never
		read again, because a query sees positions up to its own only, and recurrent state counts as zero at position 0."""
		self.next_pos = 0
		self.pos.zero_()

	@torch.no_grad()
	def feed(self, input_ids: torch.Tensor, want: Optional[Sequence[int]] = None) -> Optional[torch.Tensor]:
		"""Runs the next tokens [b, t] of every sequence behind what the cache holds.  Returns the logits [b, len(want), vocab]
		at the places `want` among them (default: the last one), None for an empty `want`.  A single token runs as a decode
		step (the captured graph), more as a portion; when the last place is wanted the greedy next token is in self.tok."""
		b, t = input_ids.shape
		if b != self.batch or t < 1:
			raise ValueError(f'feed() takes [{self.batch}, t >= 1] tokens, got {tuple(input_ids.shape)}')
		if self.next_pos + t > self.max_seq:
			raise RuntimeError(f'the static cache holds {self.max_seq} positions; {self.next_pos} are used and {t} more do not fit: build the engine with a larger max_seq')
		want = [t - 1] if want is None else list(want)
		if t == 1:
			self.tok.copy_(input_ids)
			self.step()
			# the graph's output tensor is overwritten by the next step
			return self.logits.reshape(b, 1, -1)[:, [0] * len(want)].clone() if want else None
		order = sorted(range(len(want)), key=want.__getitem__)
		parts = []
		for lo in range(0, t, self.max_portion):
			ids = input_ids[:, lo:lo + self.max_portion].to(self.device)
			local = [want[k] - lo for k in order if lo <= want[k] < lo + ids.shape[1]]
			logits = self._portion(ids, self.next_pos, local)
			self.next_pos += ids.shape[1]
			if logits is not None:
				parts.append(logits)
		self.pos.fill_(self.next_pos)
		if not parts:
			return None
		out = parts[0] if len(parts) == 1 else torch.cat(parts, dim=1)
		if want[order[-1]] == t - 1:
			self.logits = out[:, -1:]
			self.tok.copy_(self.logits.argmax(-1))
		return out if order == list(range(len(want))) else out[:, sorted(range(len(want)), key=order.__getitem__)]

	@torch.no_grad()
	def prefill(self, input_ids: torch.Tensor) -> torch.Tensor:
		"""Starts new sequences with the prompt [b, t], fills the cache, returns the first generated token [b, 1]."""
		self.reset()
		self.feed(input_ids)
		return self.tok.clone()

	@torch.no_grad()
	def step(self) -> torch.Tensor:
		"""Feeds self.tok at self.pos, returns the next token [b, 1] (device tensor)."""
		if self.next_pos >= self.max_seq:
			raise RuntimeError(f'{type(self).__name__}: the static KV cache holds {self.max_seq} positions and is full; build the engine with a larger max_seq')
		self.next_pos += 1
		if not self.use_graph:
			self._step_body()
			return self.tok
		if self.graph is None:
			self._before_capture()
			# warm up on a side stream (allocations, workspaces), then capture
			saved = (self.tok.clone(), self.pos.clone())
			carried = [t.clone() for t in self._carried()]
			s = torch.cuda.Stream()
			s.wait_stream(torch.cuda.current_stream())
			best, best_ms, best_logits = None, None, None
			with torch.cuda.stream(s):
				for _ in range(2):
					self._step_body()
					self._restore(*saved)
				s.synchronize()
				# The activations of a step live in the graph's private memory pool.  Where that pool lands (which physical
				# 2 MB page) decides how fast the few lines that every CTA reads right after a kernel boundary arrive: the same
				# graph replays 7 % faster or slower from one capture to the next (two modes, measured).  So the step is captured several
				# times, every candidate is timed on a few replays, and the fastest one is kept.  The replays write cache rows
				# at the current position onwards, which the real steps write again; token and position are restored.
				n_cand = max(1, self.graph_candidates)          # tensor parallel: every rank replays the same number of times, the choice is per rank
				alive = []          # every candidate keeps its pool until the choice is made: a freed pool would be handed to the next capture
				for _ in range(n_cand):
					g = torch.cuda.CUDAGraph()
					with torch.cuda.graph(g, stream=s):
						self._step_body()
					alive.append(g)
					cand_logits = self.logits          # the capture's own output tensor (it lives in that graph's pool)
					if n_cand == 1:
						best, best_logits = g, cand_logits
						break
					reps = max(1, min(8, self.max_seq - 1 - int(saved[1].max().item())))
					e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
					g.replay()
					e0.record(s)
					for _ in range(reps):
						self.tok.copy_(saved[0]); self.pos.copy_(saved[1])
						g.replay()
					e1.record(s)
					s.synchronize()
					ms = e0.elapsed_time(e1) / reps
					if best_ms is None or ms < best_ms:
						best, best_ms, best_logits = g, ms, cand_logits
				del alive
			torch.cuda.current_stream().wait_stream(s)
			# capture does not execute (and the timed replays started from the saved state): restore it
			self._restore(*saved)
			for t, old in zip(self._carried(), carried):
				t.copy_(old)
			self.graph = best
			self.graph_logits = best_logits
		self.graph.replay()
		self.logits = self.graph_logits
		return self.tok

	@torch.no_grad()
	def generate(self, input_ids: torch.Tensor, steps: int) -> torch.Tensor:
		"""Greedy generation: returns [b, steps] token ids (the first comes from the prefill)."""
		from . import _lib
		out = [self.prefill(input_ids)]
		for _ in range(steps - 1):
			out.append(self.step().clone())
		toks = torch.cat(out, dim=1)
		# the kernels' bounded waits report through a status word instead of hanging: a non-zero word means
		# that some result of this run cannot be trusted
		status = _lib.kernel_status(self.device)
		if status != 0:
			raise _lib.GptqB200Error(f'a decode kernel reported status {status} (see _lib.kernel_status)')
		return toks

	def close(self):
		"""Releases the captured graph."""
		self.graph = None
		self.graph_logits = None
