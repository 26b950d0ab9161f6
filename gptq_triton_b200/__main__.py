"""Command line:

  python -m gptq_triton_b200 generate --model DIR --prompt-ids 1,2,3 [--steps N] [--dtype D]     greedy generation, token ids in and out
  python -m gptq_triton_b200 trace --model DIR --dtype D --out DIR --max-tokens N                   see trace.py
"""
from __future__ import annotations

import argparse
import json
import sys


def generate(argv) -> int:
	ap = argparse.ArgumentParser(prog='gptq_triton_b200 generate')
	ap.add_argument('--model', required=True, help='checkpoint directory of any registered architecture')
	ap.add_argument('--prompt-ids', required=True, help='comma-separated token ids; several prompts of equal length separated by semicolons')
	ap.add_argument('--steps', type=int, default=32)
	ap.add_argument('--dtype', default=None, choices=['float16', 'bfloat16', 'float32'])
	ap.add_argument('--no-graph', action='store_true', help='do not capture the decode step in a CUDA graph')
	args = ap.parse_args(argv)
	import torch
	from . import registry
	model = registry.load_model(args.model, 'cuda', getattr(torch, args.dtype) if args.dtype else None)
	prompt = torch.tensor([[int(t) for t in p.split(',')] for p in args.prompt_ids.split(';')], dtype=torch.int64, device='cuda')
	engine = registry.make_engine(model, batch=prompt.shape[0], max_seq=prompt.shape[1] + args.steps + 1, use_graph=not args.no_graph)
	for row in engine.generate(prompt, args.steps).tolist():
		print(json.dumps(row))
	return 0


def main(argv=None) -> int:
	argv = sys.argv[1:] if argv is None else argv
	if argv and argv[0] == 'generate':
		return generate(argv[1:])
	if argv and argv[0] == 'trace':
		from .trace import main as trace
		return trace(argv[1:])
	print(__doc__.strip(), file=sys.stderr)
	return 2


if __name__ == '__main__':
	sys.exit(main())
