"""Replays a trace of token ids through a model's engine and writes the logits that the trace asks for.

  bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps.jsonl

A step is one line of JSON on standard input: {"step": n, "entries": [{"id": ..., "tokens": [...], "want": [...]}], "end": [...]}.
An entry brings a request's next tokens; `want` are places among them.  The logits at these places go to DIR/<step>.f32 as
little-endian fp32 rows, and after every step a line "done <step>" is printed.  Requests in `end` give their cache rows back.
Requests run one after the other in the engine's single sequence; a step with more tokens runs as a prompt portion, a single
token as a decode step, with the functions that generation uses.
"""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path


class Replay:
	"""One sequence of an engine, taken by one request at a time."""

	def __init__(self, engine):
		self.engine = engine
		self.live = None

	def run(self, step: dict):
		"""Returns the wanted logits fp32 [wanted, vocab] (None if none are wanted) and frees what ends with the step."""
		import torch
		parts = []
		for entry in step['entries']:
			if not entry['tokens']:
				continue
			if self.live != entry['id']:
				if self.live is not None:
					raise RuntimeError(f"request {entry['id']} begins while {self.live} still holds the sequence")
				self.live = entry['id']
				self.engine.reset()
			logits = self.engine.feed(torch.tensor([entry['tokens']], dtype=torch.int64), entry['want'])
			if logits is not None:
				parts.append(logits[0].float())
		if self.live in step.get('end', []):
			self.live = None
		return torch.cat(parts) if parts else None


def main(argv=None) -> int:
	ap = argparse.ArgumentParser(prog='trace_run', description='replay a trace of token ids through a model and write logits')
	ap.add_argument('--model', required=True, help='checkpoint directory')
	ap.add_argument('--dtype', required=True, choices=['bfloat16', 'float16', 'float32'])
	ap.add_argument('--out', required=True, help='directory for the logits')
	ap.add_argument('--max-tokens', type=int, required=True, help='the most tokens that live requests hold at any time (sizes the cache)')
	args = ap.parse_args(argv)

	import torch
	from . import build, registry
	arch, dtype = registry.architecture_of(args.model), getattr(torch, args.dtype)
	if dtype not in arch.dtypes:
		print(f'{arch.name} does not run in {args.dtype}', file=sys.stderr)
		return 3
	build.build(only=arch.libraries)
	torch.cuda.set_device(0)
	model = registry.load_model(args.model, 'cuda', dtype)
	replay = Replay(registry.make_engine(model, batch=1, max_seq=max(1, args.max_tokens)))
	from . import _lib
	for line in sys.stdin:
		if not line.strip():
			continue
		step = json.loads(line)
		logits = replay.run(step)
		if logits is not None:
			(Path(args.out) / f"{step['step']}.f32").write_bytes(logits.cpu().numpy().astype('<f4').tobytes())
		status = _lib.kernel_status()
		if status != 0:
			raise _lib.GptqB200Error(f'a kernel reported status {status} (see _lib.kernel_status)')
		print(f"done {step['step']}", flush=True)
	replay.engine.close()
	return 0


if __name__ == '__main__':
	sys.exit(main())
