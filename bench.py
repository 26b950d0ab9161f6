#!/usr/bin/env python
"""Benchmark of the hot path: greedy decode of a LLaMA-7B-architecture model with 4-bit g128
GPTQ weights (synthetic, random-init) at batch 1 after a 2048-token prompt.

One "step" is one decode step (one token): 32 x (fused QKV+rotary, o_proj, fused gate/up,
down_proj quantised matmuls + attention over the KV cache) + fp16 lm_head + argmax.

  python bench.py [--gpus N] [--steps K] [--warmup W] [--impl reference]

Prints ONE JSON line (rank 0).  `value` is device-timed (CUDA-graph replays, inputs resident
in HBM); `e2e` goes through the public DecodeEngine.step() API with the token fed from pinned
host memory and the result read back every step.  `roofline` is the dominant kernel (fused
gate/up decode kernel) timed live with CUDA events while rotating over all 32 layers' weights
(1.4 GB, larger than L2).  `--impl reference` times the CPU dequantise-then-matmul oracle on the
host cores on a bounded sample of the same workload.
"""
from __future__ import annotations

import argparse
import json
import os
import subprocess
import sys
import threading
import time
from pathlib import Path

ROOT = Path(__file__).resolve().parent
sys.path.insert(0, str(ROOT))

METRIC = 'decode tokens/s (7B-arch, 4-bit g128, 2k ctx)'
UNIT = 'tokens/s'
WORKLOAD = 'llama7b-arch 4-bit g128 greedy decode, batch 1, 2048-token prompt'
PROMPT = 2048
GROUPSIZE = 128


def measured_peaks():
	p = ROOT / 'MEASURED_PEAKS.json'
	if p.exists():
		d = json.load(open(p))
		return float(d['hbm_gbs']), 'measured'
	return 6650.0, 'fallback'


def quantised_bytes(K, N, g=GROUPSIZE):
	return K * N // 2 + (K // g) * N * 2 + (K // g) * N // 2


# ------------------------------------------------------------------------------------------
# reference arm / CPU baseline: the oracle's dequantise-then-matmul path on the host cores
# ------------------------------------------------------------------------------------------
def cpu_model_name() -> str:
	try:
		for line in open('/proc/cpuinfo'):
			if line.lower().startswith('model name'):
				return line.split(':', 1)[1].strip()
	except OSError:
		pass
	return 'unknown'


def cpu_layer_seconds(reps: int):
	"""One decoder layer of the decode step at batch 1 on the host cores through the CPU oracle: the four
	quantised projections at their real shapes (dequantise to fp16 + torch.matmul, the reference's CPU-runnable
	path), attention of one query over a 2112-token fp16 cache, and 1/32 of the fp16 lm_head.
	Returns (median seconds per layer, cores)."""
	import torch
	from gptq_triton_b200 import synth
	from oracle import gptq_oracle as O
	cores = os.cpu_count() or 1
	torch.set_num_threads(cores)
	h, inter, ctx, heads = 4096, 11008, 2112, 32
	shapes = [(h, 3 * h), (h, h), (h, inter), (h, inter), (inter, h)]
	ws = [synth.quant_tensors(K, N, GROUPSIZE, seed=i) for i, (K, N) in enumerate(shapes)]
	xs = [synth.activations((1, K), seed=10 + i) for i, (K, N) in enumerate(shapes)]
	g = torch.Generator().manual_seed(5)
	kc = torch.randn((heads, ctx, 128), generator=g).half()
	vc = torch.randn((heads, ctx, 128), generator=g).half()
	q = torch.randn((heads, 1, 128), generator=g).half()
	lm = (torch.randn((32000 // 32, h), generator=g) * 0.02).half()
	times = []
	for _ in range(reps):
		t0 = time.perf_counter()
		for w, x in zip(ws, xs):
			O.qmatmul_r16(x, w['qweight'], w['qzeros'], w['scales'], GROUPSIZE)
		att = torch.softmax((q.float() @ kc.float().transpose(1, 2)) / 128 ** 0.5, dim=-1)
		(att @ vc.float()).half()
		xs[0] @ lm.t()
		times.append(time.perf_counter() - t0)
	times.sort()
	return times[len(times) // 2], cores


def cpu_config0():
	"""The reference's CPU-runnable case: one 4096 x 4096 g128 QuantLinear, x [1, 512, 4096] through the torch
	dequantise + matmul path; unpack + dequantise and the matmul are timed separately."""
	import torch
	from gptq_triton_b200 import synth
	from oracle import gptq_oracle as O
	cores = os.cpu_count() or 1
	torch.set_num_threads(cores)
	t = synth.quant_tensors(4096, 4096, GROUPSIZE, seed=0)
	x = synth.activations((1, 512, 4096), seed=1)
	d, m = [], []
	for _ in range(3):
		t0 = time.perf_counter()
		w = O.dequant_f16(t['qweight'], t['qzeros'], t['scales'], GROUPSIZE)
		t1 = time.perf_counter()
		torch.matmul(x.view(512, 4096), w)
		t2 = time.perf_counter()
		d.append(t1 - t0)
		m.append(t2 - t1)
	d.sort(); m.sort()
	return {'x': [1, 512, 4096], 'K': 4096, 'N': 4096, 'groupsize': GROUPSIZE, 'dequant_s': d[1], 'matmul_s': m[1], 'total_s': d[1] + m[1],
			'gflops': 2 * 512 * 4096 * 4096 / (d[1] + m[1]) / 1e9, 'cores': cores}


LAYERS = 32


def cpu_baseline_record(reps: int):
	sec, cores = cpu_layer_seconds(reps)
	tok_s = 1.0 / (sec * LAYERS)
	return {'value': tok_s, 'unit': UNIT, 'cores': cores, 'kind': 'port', 'cpu_model': cpu_model_name(),
			'sample': 'one decoder layer of the decode step at batch 1 (4 quantised projections at their real shapes through dequantise + fp16 torch.matmul, '
					  'attention of one query over a 2112-token cache, 1/32 of the lm_head), median of %d; a token = %d such layers' % (reps, LAYERS),
			'extrapolated': True, 'factor': LAYERS, 'layer_s': sec}


def reference_arm(args):
	rank = int(os.environ.get('RANK', '0'))
	if rank != 0:
		return
	for _ in range(max(0, min(args.warmup, 2))):
		cpu_layer_seconds(1)
	rec = cpu_baseline_record(max(1, min(args.steps, 24)))
	tok_s = rec['value']
	line = {
		'impl': 'reference', 'metric': METRIC, 'value': tok_s, 'unit': UNIT, 'n_gpus': args.gpus, 'steps': args.steps, 'warmup': args.warmup,
		'ms_per_step': 1e3 / tok_s, 'higher_is_better': True, 'scaling': 'strong', 'vs_baseline': None, 'dtype': 'f16',
		'data': 'synthetic', 'config': {'workload': WORKLOAD, 'path': 'CPU port of the reference path: unpack + dequantise + torch.matmul fp16 on the host cores'},
		'cpu_baseline': rec,
		'e2e': {'value': tok_s, 'unit': UNIT, 'h2d_bytes_per_step': 0, 'd2h_bytes_per_step': 0},
	}
	print(json.dumps(line))


# ------------------------------------------------------------------------------------------
# clocks
# ------------------------------------------------------------------------------------------
class ClockSampler:
	"""SM clock and clock-event reasons of one GPU, read (never set) every few milliseconds through
	NVML while the timed region runs; falls back to an `nvidia-smi -lms` child process."""
	Q = 'index,clocks.sm,clocks.max.sm,power.draw,clocks_event_reasons.active,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap'
	BITS = {'sw_power_cap': 0x4, 'hw_slowdown': 0x8, 'sw_thermal_slowdown': 0x20, 'hw_thermal_slowdown': 0x40}

	def __init__(self, gpu_index: int, uuid: str = None):
		self.idx = gpu_index
		self.uuid = uuid
		self.proc = None
		self.lines = []
		self.nvml = None
		self.samples = []          # (sm_mhz, reason bits)
		self.stop_flag = False
		self.max_mhz = None

	def start(self):
		try:
			import pynvml
			pynvml.nvmlInit()
			h = None
			if self.uuid:
				try:
					h = pynvml.nvmlDeviceGetHandleByUUID(self.uuid.encode() if hasattr(self.uuid, 'encode') else self.uuid)
				except Exception:
					h = None
			if h is None:
				h = pynvml.nvmlDeviceGetHandleByIndex(self.idx)
			self.max_mhz = float(pynvml.nvmlDeviceGetMaxClockInfo(h, pynvml.NVML_CLOCK_SM))
			reasons_fn = getattr(pynvml, 'nvmlDeviceGetCurrentClocksEventReasons', None) or pynvml.nvmlDeviceGetCurrentClocksThrottleReasons
			self.nvml = (pynvml, h, reasons_fn)
			self.thread = threading.Thread(target=self._poll, daemon=True)
			self.thread.start()
			return
		except Exception:
			self.nvml = None
		try:
			self.proc = subprocess.Popen(['nvidia-smi', '-i', str(self.idx), '--query-gpu=' + self.Q, '--format=csv,noheader,nounits', '-lms', '100'],
										 stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
			self.thread = threading.Thread(target=self._read, daemon=True)
			self.thread.start()
		except Exception:
			self.proc = None

	def _poll(self):
		pynvml, h, reasons_fn = self.nvml
		while not self.stop_flag:
			try:
				self.samples.append((float(pynvml.nvmlDeviceGetClockInfo(h, pynvml.NVML_CLOCK_SM)), int(reasons_fn(h))))
			except Exception:
				pass
			time.sleep(0.005)

	def _read(self):
		for line in self.proc.stdout:
			self.lines.append(line.strip())

	def stop(self):
		if self.nvml is not None:
			self.stop_flag = True
			self.thread.join(timeout=1)
			sm = sorted(s for s, _ in self.samples)
			bits = 0
			for _, r in self.samples:
				bits |= r
			reasons = sorted(n for n, b in self.BITS.items() if bits & b)
			return {'sm_mhz': sm[len(sm) // 2] if sm else None, 'sm_max_mhz': self.max_mhz, 'samples': len(sm), 'reasons': reasons}
		if self.proc is None:
			return {'sm_mhz': None, 'sm_max_mhz': None, 'reasons': ['nvidia-smi unavailable']}
		self.proc.terminate()
		try:
			self.proc.wait(timeout=2)
		except Exception:
			self.proc.kill()
		sm, mx, reasons = [], None, set()
		names = ['hw_slowdown', 'hw_thermal_slowdown', 'sw_thermal_slowdown', 'sw_power_cap']
		for l in self.lines:
			f = [x.strip() for x in l.split(',')]
			if len(f) < 9:
				continue
			try:
				sm.append(float(f[1])); mx = float(f[2])
			except ValueError:
				continue
			for n, v in zip(names, f[5:9]):
				if v.lower().startswith('active'):
					reasons.add(n)
		sm.sort()
		return {'sm_mhz': sm[len(sm) // 2] if sm else None, 'sm_max_mhz': mx, 'samples': len(sm), 'reasons': sorted(reasons)}


# ------------------------------------------------------------------------------------------
# GPU arm
# ------------------------------------------------------------------------------------------
def greedy_reference(model_fn, prompt, steps):
	"""Reference-style greedy decoding (concatenated K/V tuples): tokens [b, steps], logits of the last step and the
	smallest top-1/top-2 margin."""
	import torch
	logits, past = model_fn(prompt, None)
	toks, margin = [], float('inf')
	last = None
	for _ in range(steps):
		last = logits[:, -1, :].float()
		top2 = last.topk(2, dim=-1).values
		margin = min(margin, float((top2[:, 0] - top2[:, 1]).min()))
		nxt = last.argmax(-1, keepdim=True)
		toks.append(nxt)
		logits, past = model_fn(nxt, past)
	return torch.cat(toks, dim=1), last, margin


def parity_check(G, engine_factory, reference, cfg, batch, dev, steps=8):
	"""Greedy tokens and last-step logits of the engine that is about to be timed against `reference`
	(prompt -> (tokens, last logits, margin)).  The prompt is chosen by seed so that every top-1/top-2 margin of
	the reference run is clear of fp16 noise (random-init logits over 32000 entries are nearly flat)."""
	import torch
	best = None
	for seed in range(6):
		prompt = torch.randint(0, cfg.vocab_size, (batch, PROMPT), generator=torch.Generator().manual_seed(500 + seed)).to(dev)
		toks, last, margin = reference(prompt, steps)
		if best is None or margin > best[3]:
			best = (prompt, toks, last, margin)
		if margin > 0.05:
			break
	prompt, ref_toks, ref_last, margin = best
	engine = engine_factory()
	out = [engine.prefill(prompt)]
	for _ in range(steps - 1):
		out.append(engine.step().clone())
	# the logits that produced the last token: those of step `steps - 1`
	got = torch.cat(out, dim=1)
	logits = engine.logits.float().view(batch, -1)
	diff = (got != ref_toks).any(dim=0).nonzero()
	first = int(diff[0]) if diff.numel() else -1
	scale = float(ref_last.abs().max())
	err = float((logits - ref_last.view(batch, -1)).abs().max()) / max(scale, 1e-30) if first < 0 else None
	# Tokens must be identical.  The logits of the last step are compared as max|a - b| / max|b|; both runs round the
	# residual stream and the activations to fp16 at 2 x 32 places with different summation orders (and the twin also
	# rounds the weights to fp16), so the bound is that of accumulated fp16 rounding over 32 layers, not of one op.
	return engine, {'steps': steps, 'first_diff_step': first, 'min_reference_margin': margin, 'last_logits_max_err_over_max': err,
					'tolerance': 2e-2, 'ok': bool(first < 0 and err is not None and err <= 2e-2)}


def prefill_record(G, model, cfg, dev, peak_tflops):
	"""The tcgen05 prefill kernel at M = 512 and 2048 on the model's own weights, rotating over all layers
	(32 x 8 MB / 32 x 43 MB of packed weights: larger than L2), timed with CUDA events."""
	import torch
	layers = model.model.layers
	out = []
	for M in (512, 2048):
		x = (torch.randn((1, M, cfg.hidden_size), device=dev) * 0.5).half()
		for name, fn, flops in (
				('o_proj %dx%d' % (cfg.hidden_size, cfg.hidden_size), lambda l: l.self_attn.o_proj(x), 2.0 * M * cfg.hidden_size * cfg.hidden_size),
				('gate/up %dx2x%d fused' % (cfg.hidden_size, cfg.intermediate_size), lambda l: l.mlp.intermediate(x), 4.0 * M * cfg.hidden_size * cfg.intermediate_size)):
			for l in layers[:3]:
				fn(l)
			torch.cuda.synchronize()
			e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
			e0.record()
			for l in layers:
				fn(l)
			e1.record()
			torch.cuda.synchronize()
			us = e0.elapsed_time(e1) * 1e3 / len(layers)
			tf = flops / us / 1e6
			out.append({'M': M, 'op': name, 'us': us, 'tflops': tf, 'frac': tf / peak_tflops})
	return out


def measure_exchange(G, tp, dev, rank, world, barrier, dist):
	"""The all-reduce that is fused into the row-parallel decode kernel, alone: a projection with a one-chunk K-slice
	(128 rows per rank, 4096 outputs, one row of x) with and without the exchange over peer memory, 64 launches per CUDA
	graph, CUDA events, max over ranks.  The difference is what one exchange adds to a kernel; a 7B decode step has 64."""
	import torch
	from gptq_triton_b200 import synth
	N, K = 4096, 128
	t = synth.quant_tensors(K, N, 128, seed=77 + rank)
	w = tuple(v.to(dev) for v in (t['qweight'], t['scales'], t['qzeros']))
	x = synth.activations((1, K), seed=5).to(dev)
	res = torch.zeros((1, N), dtype=torch.float16, device=dev)
	try:
		ex = tp.PeerExchange(N, rank, world, group=None)
	except RuntimeError:
		return None
	out = {}
	for name, ar in (('with_exchange_us', ex), ('without_exchange_us', None)):
		fn = lambda: G.qmatmul(128, x, *w, residual=res, ar=ar)
		s = torch.cuda.Stream()
		with torch.cuda.stream(s):
			for _ in range(3):
				fn()
			s.synchronize()
			barrier()
			g = torch.cuda.CUDAGraph()
			with torch.cuda.graph(g, stream=s):
				for _ in range(64):
					fn()
			barrier()
			g.replay()
			s.synchronize()
			barrier()
			e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
			e0.record(s)
			for _ in range(5):
				g.replay()
			e1.record(s)
			s.synchronize()
		us = torch.tensor([e0.elapsed_time(e1) * 1e3 / (5 * 64)], device=dev)
		dist.all_reduce(us, op=dist.ReduceOp.MAX)
		out[name] = float(us.item())
		del g
	barrier()
	ex.close()
	out['exchange_us'] = out['with_exchange_us'] - out['without_exchange_us']
	out['what'] = 'o_proj-shaped decode kernel (M = 1, 128 rows per rank -> 4096) inside a CUDA graph, with and without the fused all-reduce'
	return out


def measure_config4(G, tp, dev, rank, world, barrier, dist, steps=16, warmup=4):
	"""Benchmark configuration 4: LLaMA-65B architecture, 4-bit g128, batch 16, 2048-token prompts, greedy decode,
	tensor parallel over the ranks of this run.  Device-timed like the main measurement (barrier, CUDA events, max over
	ranks).  Reports tokens/s over all sequences, the bytes one rank streams per step and the fraction of that rank's
	HBM roofline."""
	import torch
	from gptq_triton_b200 import _lib
	from gptq_triton_b200.llama import LlamaConfig
	cfg = LlamaConfig.llama_65b()
	batch = 16
	model = G.synthetic_quantized_llama(cfg, groupsize=GROUPSIZE, seed=4321, device=dev, fuse=False)
	if world > 1:
		tp.shard_llama(model, rank, world)
	G.make_quant_attn(model)
	G.make_fused_mlp(model)
	torch.cuda.empty_cache()
	engine = G.DecodeEngine(model, batch=batch, max_seq=PROMPT + warmup + steps + 16, use_graph=True)
	prompt = torch.randint(0, cfg.vocab_size, (batch, PROMPT), generator=torch.Generator().manual_seed(77)).to(dev)
	engine.prefill(prompt)
	for _ in range(warmup):
		engine.step()
	barrier()
	e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
	e0.record()
	for _ in range(steps):
		engine.step()
	e1.record()
	barrier()
	t = torch.tensor([e0.elapsed_time(e1)], device=dev)
	if dist is not None:
		dist.all_reduce(t, op=dist.ReduceOp.MAX)
	ms = float(t.item())
	wbytes = 0
	for n, b_ in model.named_buffers():
		if n.endswith(('qweight', 'qzeros', 'scales')):
			wbytes += b_.numel() * b_.element_size()
	wbytes += model.lm_head.weight.numel() * 2
	heads_local = model.model.layers[0].self_attn.num_heads
	ctx = PROMPT + warmup + steps / 2.0
	kv = 2.0 * cfg.num_hidden_layers * batch * heads_local * ctx * 128 * 2
	peak, which = measured_peaks()
	ach = (wbytes + kv) / (ms / steps) / 1e6
	rec = {'workload': 'llama65b-arch 4-bit g128 greedy decode, batch 16, 2048-token prompts, tp%d' % world, 'value': batch * steps / (ms / 1e3), 'unit': UNIT,
		   'ms_per_step': ms / steps, 'steps': steps, 'warmup': warmup, 'weight_bytes_per_rank': wbytes, 'kv_bytes_per_rank_per_step': kv,
		   'achieved_gbs_per_rank': ach, 'hbm_peak_gbs': peak, 'frac_of_rank_roofline': ach / peak, 'peak_source': which,
		   'fused_all_reduce': engine.ar_o is not None, 'kernel_status': _lib.kernel_status(dev)}
	barrier()
	engine.close()
	return rec


def gpu_arm(args):
	import torch
	import torch.distributed as dist

	rank = int(os.environ.get('RANK', '0'))
	local_rank = int(os.environ.get('LOCAL_RANK', '0'))
	world = int(os.environ.get('WORLD_SIZE', '1'))
	if not torch.cuda.is_available():
		raise SystemExit('bench.py needs a CUDA device (B200); there is no CPU path for the product kernels')
	torch.cuda.set_device(local_rank)
	dev = torch.device('cuda', local_rank)
	if world > 1:
		dist.init_process_group('nccl', device_id=dev)

	import gptq_triton_b200 as G
	from gptq_triton_b200 import _lib, loader
	from gptq_triton_b200.llama import LlamaConfig

	from gptq_triton_b200 import tp
	big = args.workload == 'llama65b-b16'
	cfg = LlamaConfig.llama_65b() if big else LlamaConfig.llama_7b()
	batch = 16 if big else 1
	if args.layers:
		cfg.num_hidden_layers = args.layers            # debugging aid only; the default is the full model
	max_seq = PROMPT + args.warmup + 2 * args.steps + 32

	# ---- the model, and the parity check of the engine that is timed below --------------------------------
	# N = 1: against the dequantise-then-matmul twin (fp16 nn.Linear holding the dequantised weights, cuBLAS);
	# N > 1: ONE model, tensor-parallel over the N GPUs (same seed on every rank, each keeps its shards), against the
	# un-sharded engine built on the same rank.
	parity = None
	if world > 1:
		model = G.synthetic_quantized_llama(cfg, groupsize=GROUPSIZE, seed=1234, device=dev, fuse=False)
		tp.shard_llama(model, rank, world)
		G.make_quant_attn(model)
		G.make_fused_mlp(model)
		torch.cuda.empty_cache()
		factory = lambda: G.DecodeEngine(model, batch=batch, max_seq=max_seq, use_graph=not args.no_graph)
		if not big and not args.no_parity:
			whole = G.synthetic_quantized_llama(cfg, groupsize=GROUPSIZE, seed=1234, device=dev)
			def reference(prompt, steps):
				e = G.DecodeEngine(whole, batch=batch, max_seq=PROMPT + steps + 8, use_graph=False)
				toks = [e.prefill(prompt)]
				margin = float('inf')
				for i in range(steps):
					top2 = e.logits.float().view(batch, -1).topk(2, dim=-1).values
					margin = min(margin, float((top2[:, 0] - top2[:, 1]).min()))
					last = e.logits.float().view(batch, -1).clone()
					if i < steps - 1:
						toks.append(e.step().clone())
				return torch.cat(toks, dim=1), last, margin
			engine, parity = parity_check(G, factory, reference, cfg, batch, dev)
			parity['against'] = 'un-sharded engine on the same rank'
			flag = torch.tensor([1 if parity['ok'] else 0], device=dev)
			dist.all_reduce(flag, op=dist.ReduceOp.MIN)
			parity['ok_on_every_rank'] = bool(int(flag.item()))
			del whole
			torch.cuda.empty_cache()
		else:
			engine = factory()
	else:
		model = G.synthetic_quantized_llama(cfg, groupsize=GROUPSIZE, seed=1234, device=dev, fuse=False)
		dense = None if (big or args.no_parity) else loader.dense_reference_copy(model)
		G.make_quant_attn(model)
		G.make_fused_mlp(model)
		factory = lambda: G.DecodeEngine(model, batch=batch, max_seq=max_seq, use_graph=not args.no_graph)
		if dense is not None:
			def model_fn(ids, past):
				return dense(ids, past_key_values=past, use_cache=True)
			engine, parity = parity_check(G, factory, lambda prompt, steps: greedy_reference(model_fn, prompt, steps), cfg, batch, dev)
			parity['against'] = 'dequantise-then-matmul twin (fp16 cuBLAS) of the same model'
			del dense
			torch.cuda.empty_cache()
		else:
			engine = factory()
	gen = torch.Generator().manual_seed(99)
	prompt = torch.randint(0, cfg.vocab_size, (batch, PROMPT), generator=gen).to(dev)
	engine.prefill(prompt)
	torch.cuda.synchronize()

	def barrier():
		torch.cuda.synchronize()
		if world > 1:
			dist.barrier()
		torch.cuda.synchronize()

	# ---- device-timed: K graph replays -------------------------------------------------------
	try:
		gpu_uuid = 'GPU-' + str(torch.cuda.get_device_properties(local_rank).uuid)
	except Exception:
		gpu_uuid = None
	sampler = ClockSampler(local_rank, gpu_uuid)
	if rank == 0:
		sampler.start()           # before the warm-up: the timed region follows the warm-up without a pause
	for _ in range(args.warmup):
		engine.step()
	barrier()
	if rank == 0:
		sampler.samples.clear()
	e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
	torch.cuda.profiler.start()           # lets a profiler restrict itself to the timed region
	e0.record()
	for _ in range(args.steps):
		engine.step()
	e1.record()
	barrier()
	torch.cuda.profiler.stop()
	ms = e0.elapsed_time(e1)
	clocks = sampler.stop() if rank == 0 else None
	t = torch.tensor([ms], device=dev)
	if world > 1:
		dist.all_reduce(t, op=dist.ReduceOp.MAX)
	ms = float(t.item())
	tok_s = batch * args.steps / (ms / 1e3)            # every rank works on the same tokens (tensor parallel)

	# ---- end to end through DecodeEngine.step(): token in from pinned host memory, token out ----
	host_tok = torch.zeros((batch, 1), dtype=torch.int64).pin_memory()
	host_out = torch.zeros((batch, 1), dtype=torch.int64).pin_memory()
	host_tok.copy_(engine.tok.cpu())
	barrier()
	t0 = time.perf_counter()
	for _ in range(args.steps):
		engine.tok.copy_(host_tok, non_blocking=True)       # H2D: the token chosen on the host side
		out = engine.step()
		host_out.copy_(out, non_blocking=True)              # D2H: the next token
		torch.cuda.current_stream().synchronize()
		host_tok.copy_(host_out)
	e2e_s = time.perf_counter() - t0
	t = torch.tensor([e2e_s], device=dev)
	if world > 1:
		dist.all_reduce(t, op=dist.ReduceOp.MAX)
	e2e_tok_s = batch * args.steps / float(t.item())

	# ---- roofline of the dominant kernel: fused gate/up decode kernel, live, rotating weights ----
	roof = None
	status = None
	prefill = None
	if rank == 0:
		layers = model.model.layers
		x = torch.randn((batch, 1, cfg.hidden_size), device=dev, dtype=torch.float16)
		for l in layers[:4]:
			l.mlp.intermediate(x)
		torch.cuda.synchronize()
		reps = max(1, 256 // len(layers))
		k0, k1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
		g = torch.cuda.CUDAGraph()
		s = torch.cuda.Stream()
		s.wait_stream(torch.cuda.current_stream())
		with torch.cuda.stream(s):
			for l in layers:
				l.mlp.intermediate(x)
			s.synchronize()
			with torch.cuda.graph(g, stream=s):
				for l in layers:
					l.mlp.intermediate(x)
			g.replay()
			s.synchronize()
			k0.record(s)
			for _ in range(reps):
				g.replay()
			k1.record(s)
			s.synchronize()
		us = k0.elapsed_time(k1) * 1e3 / (reps * len(layers))
		K, N = cfg.hidden_size, int(layers[0].mlp.gate_proj_qweight.shape[1])      # N is this rank's share under tensor parallelism
		alg = 2 * quantised_bytes(K, N) + batch * (2 * K + 2 * N)           # two weight streams + x + y
		peak, which = measured_peaks()
		ach = alg / us / 1e3
		full = world == 1 and not big
		roof = {'bound': 'hbm', 'kernel': 'skinny_kernel<gate/up, SiLU epilogue> M=%d K=%d N=%d' % (batch, K, N), 'achieved': ach, 'peak': peak, 'unit': 'GB/s',
				'frac': ach / peak, 'peak_source': which, 'us_per_launch': us, 'algorithmic_bytes': alg,
				'traffic': 46.95e6 if full else None,
				'traffic_source': 'ncu capture of the same kernel and shape (dram__bytes_read + dram__bytes_write per launch), profiles/skinny_gateup_m1_ncu_full.md' if full else None}
		if world == 1 and not big and not args.no_prefill:
			tf_peak = 1618.5
			pk = ROOT / 'MEASURED_PEAKS.json'
			if pk.exists():
				tf_peak = float(json.load(open(pk)).get('bf16_tflops', tf_peak))
			prefill = {'bound': 'tensor', 'peak': tf_peak, 'peak_source': 'measured cuBLAS bf16 burst' if pk.exists() else 'fallback', 'unit': 'TFLOP/s',
					   'kernels': prefill_record(G, model, cfg, dev, tf_peak)}
		status = _lib.kernel_status(dev)

	# ---- CPU baseline (rank 0, N=1 only) -----------------------------------------------------------
	cpu = None
	if rank == 0 and world == 1 and not args.no_cpu_baseline:
		cpu = cpu_baseline_record(9)
		cpu['config0'] = cpu_config0()

	exchange = None
	# ---- benchmark configuration 4 as a sub-record: 65B architecture, batch 16, tensor parallel (N >= 2 by default) ----
	config4 = None
	want4 = (args.config4 == 'on') or (args.config4 == 'auto' and world > 1)
	if want4 and not big and not args.layers:
		launches_7b = None
		chain_used = engine.chain is not None
		qa_used = int(engine.used_qkv_attn) + int(engine.used_fused_oproj)
		fused_ar = engine.ar_o is not None
		folded_7b = engine.fuse_norm and batch <= 16 and (world == 1 or engine.ar_o is not None)
		barrier()
		engine.close()
		del engine, model
		torch.cuda.empty_cache()
		exchange = measure_exchange(G, tp, dev, rank, world, barrier, dist) if (world > 1 and fused_ar) else None
		config4 = measure_config4(G, tp, dev, rank, world, barrier, dist if world > 1 else None)
		engine = None
	else:
		chain_used = engine.chain is not None
		qa_used = int(engine.used_qkv_attn) + int(engine.used_fused_oproj)
		fused_ar = engine.ar_o is not None
		folded_7b = engine.fuse_norm and batch <= 16 and (world == 1 or engine.ar_o is not None)

	rc = 0
	if rank == 0:
		# own kernels per rank and step: 4 quantised matmuls + attention per layer (batch 1: the QKV projection and the attention
		# and on one GPU also o_proj are one kernel), embedding + first norm in one kernel,
		# final norm + lm_head + arg-max in one kernel; RMSNorm is otherwise folded into the matmul kernels.  The persistent
		# kernel path: one chain kernel + lm_head.
		if chain_used:
			launches_per_step = 2
		else:
			launches_per_step = ((5 - qa_used) * cfg.num_hidden_layers + 2) if folded_7b else (7 * cfg.num_hidden_layers + 1)
		line = {
			'metric': METRIC, 'value': tok_s, 'unit': UNIT, 'n_gpus': world, 'steps': args.steps, 'warmup': args.warmup,
			'ms_per_step': ms / args.steps, 'higher_is_better': True, 'scaling': 'strong', 'vs_baseline': None, 'dtype': 'f16',
			'data': 'synthetic',
			'config': {'workload': WORKLOAD if not big else 'llama65b-arch 4-bit g128 greedy decode, batch 16, 2048-token prompts', 'layers': cfg.num_hidden_layers, 'hidden': cfg.hidden_size, 'groupsize': GROUPSIZE,
					   'parallelism': (('tp%d: QKV and gate/up by columns, o_proj and down by rows, ' % world) + ('all-reduce fused into those kernels over peer memory' if fused_ar else 'one NCCL all-reduce after each')) if world > 1 else 'single GPU',
					   'step': 'persistent chain kernel' if chain_used else (('attention block (QKV projection, rotary, attention, o_proj, residual) in one kernel, gate/up and down_proj one kernel each, CUDA graph' if qa_used == 2 else 'QKV projection + attention in one kernel, one kernel per other projection, CUDA graph') if qa_used else 'one kernel per projection, CUDA graph'),
					   'l2': 'inputs larger than L2: 3.6 GB of weights + KV cache are streamed every step'},
			'e2e': {'value': e2e_tok_s, 'unit': UNIT, 'h2d_bytes_per_step': 8 * batch, 'd2h_bytes_per_step': 8 * batch},
			'gpu_launches': launches_per_step * args.steps,
			'roofline': roof, 'prefill': prefill, 'parity': parity, 'config4': config4, 'exchange': exchange, 'cpu_baseline': cpu, 'clocks': clocks, 'kernel_status': status,
		}
		print(json.dumps(line), flush=True)
		if config4 is not None and config4.get('kernel_status'):
			status = status or config4['kernel_status']
		if status != 0:
			sys.stderr.write('bench.py: a kernel reported status %d (see gptq_triton_b200._lib.kernel_status)\n' % status)
			rc = 3
	if world > 1:
		# Leave without tearing the communicator down: destroying a process group while CUDA graphs
		# that captured its collectives are alive was seen to block until the NCCL watchdog fired.
		torch.cuda.synchronize()
		dist.barrier()
		sys.stdout.flush()
		os._exit(rc)
	if rc:
		sys.exit(rc)


def kernel_case(args):
	"""Small stand-alone case for profilers: a few launches of one decode kernel over rotating
	weight copies (larger than L2 together), nothing else.  `--kernel-case gateup|qkv|o|down`."""
	import torch
	import gptq_triton_b200 as G
	from gptq_triton_b200 import synth
	dev = torch.device('cuda', 0)
	M = args.m
	if args.kernel_case == 'prefill':
		# tensor-core kernel: M x 4096 x 4096 quantised matmul, three launches
		K, N = 4096, 4096
		t = synth.quant_tensors(K, N, GROUPSIZE, seed=2)
		w = tuple(v.to(dev) for v in (t['qweight'], t['scales'], t['qzeros']))
		x = synth.activations((max(M, 2048), K), seed=1).to(dev)
		for i in range(3):
			G.qmatmul(GROUPSIZE, x, *w)
		torch.cuda.synchronize()
		print(json.dumps({'kernel_case': 'prefill', 'M': int(x.shape[0]), 'launches': 3}))
		return
	if args.kernel_case in ('latent-prefill', 'latent-decode'):
		# latent attention, 2048 tokens: the tensor-core prompt kernel alone / decode steps of two layers (about 2 GB on the device)
		import ctypes
		from gptq_triton_b200 import _dense
		if args.kernel_case == 'latent-prefill':
			ctl = _dense.control_buffer(dev)
			t, H, D, R, V, C = PROMPT, args.heads, 128, 64, 128, 512
			bf = lambda *shape: torch.randn(shape, device=dev).bfloat16()
			q, k, vt, c, g, o = bf(t, H * (D + R)), bf(t, H * D), bf(H * V, t), bf(t, C + R), torch.rand((t, H), device=dev), bf(t, H * V)
			p = _dense.LatentPrefill()
			p.t, p.start, p.S, p.heads, p.dim, p.rot_dim, p.vdim, p.kv_rank, p.scale = t, 0, t, H, D, R, V, C, (D + R) ** -0.5
			p.q, p.k, p.vt, p.ldv, p.cache, p.gate, p.gate_ld = q.data_ptr(), k.data_ptr(), vt.data_ptr(), t, c.data_ptr(), g.data_ptr(), H
			p.out, p.out_ld, p.status = o.data_ptr(), H * V, _dense.status_ptr(ctl).value
			for _ in range(3):
				_dense.check(_dense.lib().dense_latent_prefill(ctypes.byref(p), None), 'dense_latent_prefill')
		else:
			cfg = befalix_config(G, 2, 4096, 11008, 32, 128, 64, 128, 512, vocab=2048)
			e = G.BefalixEngine(G.synthetic_befalix(cfg, device=dev), 1, PROMPT + 16, use_graph=False)
			e.feed(torch.randint(0, cfg.vocab_size, (1, PROMPT), generator=torch.Generator().manual_seed(3)))
			for _ in range(3):
				e.step()
		torch.cuda.synchronize()
		print(json.dumps({'kernel_case': args.kernel_case}))
		return
	if args.kernel_case in ('gqa-prefill', 'ssm-prefill', 'lifinex-decode'):
		# 2048 tokens through the tensor-core kernels of the differential attention / the state-space recurrence alone, or decode steps
		# of two layers (at most 2 GB on the device)
		import ctypes
		from gptq_triton_b200 import _dense
		from gptq_triton_b200.cache import StaticCache
		bf, t = torch.bfloat16, PROMPT
		cfg = lifinex_config(G, 2, args.heads * 128, 11008 if args.kernel_case == 'lifinex-decode' else 256, vocab=2048)
		e = G.LifinexEngine(G.synthetic_lifinex(cfg, device=dev), 1, PROMPT + 16, use_graph=False)
		if args.kernel_case == 'lifinex-decode':
			e.feed(torch.randint(0, cfg.vocab_size, (1, t), generator=torch.Generator().manual_seed(3)))
			for _ in range(3):
				e.step()
		elif args.kernel_case == 'gqa-prefill':
			mx, s = e.model.layers[0].mixer, cfg.layers[0].mixer
			raw, o = torch.randn((t, mx.w_in.shape[0]), device=dev).to(bf), torch.empty((t, s.heads * mx.V), dtype=bf, device=dev)
			pos = torch.arange(t, dtype=torch.int32, device=dev)
			a = mx.arguments(raw, e.cache[0], pos, t, cfg.norm_eps, e.control)
			keep = mx.buffers(a, o, 1)
			_dense.check(_dense.lib().dense_gqa_append(ctypes.byref(a), 0, None), 'dense_gqa_append')
			for _ in range(3):
				_dense.check(_dense.lib().dense_gqa_prefill(ctypes.byref(a), 0, None), 'dense_gqa_prefill')
		else:
			mx, s = e.model.layers[1].mixer, cfg.layers[1].mixer
			raw, steps = torch.randn((t, mx.dt_at), device=dev).to(bf), torch.randn((t, mx.w_in.shape[0] - mx.dt_at), device=dev)
			o, pos = torch.empty((t, s.inner), dtype=bf, device=dev), torch.arange(t, dtype=torch.int32, device=dev)
			a = mx.arguments(raw, steps, e.cache[1], pos, t, o, e.control)
			keep = mx.portion_buffers(a, bf, True)
			_dense.check(_dense.lib().dense_ssm_conv(ctypes.byref(a), 0, None), 'dense_ssm_conv')
			for _ in range(3):
				_dense.check(_dense.lib().dense_ssm_chunked(ctypes.byref(a), None), 'dense_ssm_chunked')
		torch.cuda.synchronize()
		print(json.dumps({'kernel_case': args.kernel_case}))
		return
	if args.kernel_case == 'chain':
		# the persistent decode-step kernel on four layers of the 7B architecture after a 2048-token prompt (about 1 GB on
		# the device): a few steps, nothing else; also prints the step time of both engines
		from gptq_triton_b200.llama import LlamaConfig
		cfg = LlamaConfig(num_hidden_layers=4, max_position_embeddings=4096)
		model = G.synthetic_quantized_llama(cfg, groupsize=GROUPSIZE, seed=1, device=dev)
		prompt = torch.randint(0, cfg.vocab_size, (1, PROMPT), generator=torch.Generator().manual_seed(3)).to(dev)
		out = {'kernel_case': 'chain', 'layers': 4}
		for name, flag in (('chain', '1'), ('kernel_per_projection', '0')):
			os.environ['GPTQ_B200_CHAIN'] = flag
			e = G.DecodeEngine(model, batch=1, max_seq=PROMPT + 64, use_graph=(flag == '0'))
			assert (e.chain is not None) == (flag == '1')
			e.prefill(prompt)
			for _ in range(5):
				e.step()
			torch.cuda.synchronize()
			e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
			e0.record()
			for _ in range(20):
				e.step()
			e1.record()
			torch.cuda.synchronize()
			out[name + '_ms_per_step'] = e0.elapsed_time(e1) / 20
		print(json.dumps(out))
		return
	if args.kernel_case == 'lmhead':
		# final RMSNorm + fp16 lm_head + arg-max: 32000 x 4096 weights (262 MB, larger than L2), timed with CUDA events
		from gptq_triton_b200 import _lib
		L = _lib.lib()
		V, K = 32000, 4096
		h = (torch.randn((M, K), device=dev) * 2).half()
		wn = torch.ones((K,), device=dev, dtype=torch.float16)
		W = (torch.randn((V, K), device=dev) * 0.02).half()
		ss = h.float().pow(2).view(M, K // 32, 32).sum(-1).contiguous()
		logits = torch.zeros((M, V), dtype=torch.float16, device=dev)
		tok = torch.zeros((M,), dtype=torch.int64, device=dev)
		pos = torch.zeros((M,), dtype=torch.int32, device=dev)
		ws = torch.zeros(L.gptq_lm_head_workspace_bytes(M), dtype=torch.uint8, device=dev)
		def run():
			rc = L.gptq_lm_head_argmax(_lib.ptr(h), _lib.ptr(ss), _lib.ptr(wn), _lib.ptr(W), M, K, V, 1e-6, _lib.ptr(logits), _lib.ptr(tok), _lib.ptr(pos),
									   _lib.ptr(ws), ws.numel(), _lib.stream_ptr(dev))
			assert rc == 0
		for _ in range(3):
			run()
		torch.cuda.synchronize()
		e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
		e0.record()
		for _ in range(10):
			run()
		e1.record()
		torch.cuda.synchronize()
		us = e0.elapsed_time(e1) * 100
		x = (h.float() * torch.rsqrt(h.float().pow(2).mean(-1, keepdim=True) + 1e-6)).half()
		t0, t1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
		for _ in range(3):
			(x @ W.t()).argmax(-1)
		t0.record()
		for _ in range(10):
			(x @ W.t()).argmax(-1)
		t1.record()
		torch.cuda.synchronize()
		peak, which = measured_peaks()
		alg = V * K * 2 + M * K * 2 + M * V * 2
		print(json.dumps({'kernel_case': 'lmhead', 'M': M, 'us': us, 'gbs': alg / us / 1e3, 'frac': alg / us / 1e3 / peak, 'peak_source': which,
						  'cublas_plus_argmax_us': t0.elapsed_time(t1) * 100, 'launches': 13}))
		return
	if args.kernel_case == 'attn':
		# single-query attention over rotating caches (together larger than L2) at 2100 tokens of context:
		# --m sequences x --heads heads (1 x 32: the 7B decode step; 16 x 8 / 16 x 16 / 16 x 32: configuration 4 per rank at tp8 / 4 / 2)
		from gptq_triton_b200.fused_attention import attn_decode
		B, H, S, D = M, args.heads, 2200, 128
		per = 2 * B * H * S * D * 2
		ncache = max(2, min(8, (300 << 20) // per + 1))
		caches = [(torch.randn((B, H, S, D), device=dev).half(), torch.randn((B, H, S, D), device=dev).half()) for _ in range(ncache)]
		q = torch.randn((B, 1, H, D), device=dev).half().transpose(1, 2)
		pos = torch.full((B, 1), 2100, dtype=torch.int32, device=dev)
		for i in range(ncache):
			attn_decode(q, caches[i][0], caches[i][1], pos, 2101)
		torch.cuda.synchronize()
		e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
		reps = 4
		e0.record()
		for _ in range(reps):
			for i in range(ncache):
				attn_decode(q, caches[i][0], caches[i][1], pos, 2101)
		e1.record()
		torch.cuda.synchronize()
		us = e0.elapsed_time(e1) * 1e3 / (reps * ncache)
		alg = 2 * B * H * 2101 * D * 2
		peak, which = measured_peaks()
		print(json.dumps({'kernel_case': 'attn', 'batch': B, 'heads': H, 'ctx': 2101, 'us': us, 'gbs': alg / us / 1e3, 'frac': alg / us / 1e3 / peak,
						  'peak_source': which, 'launches': ncache * (reps + 1)}))
		return
	if args.kernel_case == 'qkvattn':
		# decode attention block of one sequence at 2100 tokens of context, 7B shapes: the one-kernel form (projection + rotary +
		# cache append + attention, one cluster per head) against the pair qkv_rope + attn_decode, over rotating copies of the
		# weights and caches (together larger than L2), timed with CUDA events
		from gptq_triton_b200.fused_attention import attn_decode, qkv_attn_decode, qkv_attn_oproj_decode, qkv_attn_oproj_scratch, qkv_rope, rope_tables
		K, H, S, D, ctx = 4096, 32, 2200, 128, 2100
		t = synth.quant_tensors(K, 3 * H * D, GROUPSIZE, seed=2)
		ncopy = 8
		ws = [tuple(v.to(dev).clone() for v in (t['qweight'], t['scales'], t['qzeros'])) for _ in range(ncopy)]
		to = synth.quant_tensors(K, K, GROUPSIZE, seed=3)
		wo = [tuple(v.to(dev).clone() for v in (to['qweight'], to['scales'], to['qzeros'])) for _ in range(ncopy)]
		scratch = qkv_attn_oproj_scratch(H, K, dev)
		ss = torch.zeros(K // 32, dtype=torch.float32, device=dev)
		caches = [(torch.randn((1, H, S, D), device=dev).half(), torch.randn((1, H, S, D), device=dev).half()) for _ in range(ncopy)]
		x = synth.activations((1, 1, K), seed=1).to(dev)
		cos, sin = rope_tables(D, S, 10000.0, device=dev)
		pos = torch.full((1, 1), ctx, dtype=torch.int32, device=dev)
		def one(i):
			qw, sc, qz = ws[i]
			return qkv_attn_decode(GROUPSIZE, x, qw, sc, qz, cos, sin, pos.view(-1), caches[i][0], caches[i][1], H)
		def pair(i):
			qw, sc, qz = ws[i]
			q, _, _ = qkv_rope(GROUPSIZE, x, qw, sc, qz, cos, sin, pos, H, D, kv_cache=caches[i])
			return attn_decode(q, caches[i][0], caches[i][1], pos, ctx + 1)
		def block(i):          # the whole attention block: + o_proj + residual, still one kernel
			qw, sc, qz = ws[i]
			return qkv_attn_oproj_decode(GROUPSIZE, x, qw, sc, qz, cos, sin, pos.view(-1), caches[i][0], caches[i][1], H, GROUPSIZE, wo[i][0], wo[i][1],
										 wo[i][2], scratch, residual=x, sumsq_out=ss)
		def pair_o(i):
			return G.qmatmul(GROUPSIZE, pair(i).view(1, K), *wo[i], residual=x.view(1, K), sumsq_out=ss.view(1, -1))
		out = {'kernel_case': 'qkvattn', 'heads': H, 'ctx': ctx + 1, 'timing': 'eager launches, CUDA events (includes launch gaps)'}
		reps = 4
		for name, fn in (('one_kernel_us', one), ('two_kernels_us', pair), ('block_one_kernel_us', block), ('block_three_kernels_us', pair_o)):
			for i in range(ncopy):
				fn(i)
			torch.cuda.synchronize()
			e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
			e0.record()
			for _ in range(reps):
				for i in range(ncopy):
					fn(i)
			e1.record()
			torch.cuda.synchronize()
			out[name] = e0.elapsed_time(e1) * 1e3 / (reps * ncopy)
		alg = K * 3 * H * D // 2 + (K // GROUPSIZE) * 3 * H * D * 5 // 2 + 2 * H * (ctx + 1) * D * 2
		alg_block = alg + K * K // 2 + (K // GROUPSIZE) * K * 5 // 2
		peak, which = measured_peaks()
		out.update({'alg_bytes_block': alg_block, 'frac_block_one_kernel': alg_block / out['block_one_kernel_us'] / 1e3 / peak, 'alg_bytes': alg, 'frac_one_kernel': alg / out['one_kernel_us'] / 1e3 / peak, 'frac_two_kernels': alg / out['two_kernels_us'] / 1e3 / peak,
					'peak_source': which, 'max_abs_diff': float((one(0).float() - pair(0).float()).abs().max()), 'launches': 8 * ncopy * (reps + 1) + 3})
		from gptq_triton_b200 import _lib
		out['kernel_status'] = _lib.kernel_status()
		print(json.dumps(out))
		return
	if args.kernel_case == 'gateup':
		K, N = 4096, 11008
		g, u = synth.quant_tensors(K, N, GROUPSIZE, seed=2), synth.quant_tensors(K, N, GROUPSIZE, seed=3)
		copies = [tuple(t.to(dev).clone() for t in (g['qweight'], g['scales'], g['qzeros'], u['qweight'], u['scales'], u['qzeros'])) for _ in range(4)]
		x = synth.activations((M, K), seed=1).to(dev)
		for i in range(8):
			G.gateup_silu(GROUPSIZE, x, *copies[i % 4])
	else:
		K, N = {'qkv': (4096, 12288), 'o': (4096, 4096), 'down': (11008, 4096)}[args.kernel_case]
		t = synth.quant_tensors(K, N, GROUPSIZE, seed=2)
		copies = [tuple(v.to(dev).clone() for v in (t['qweight'], t['scales'], t['qzeros'])) for _ in range(8)]
		x = synth.activations((M, K), seed=1).to(dev)
		for i in range(8):
			G.qmatmul(GROUPSIZE, x, *copies[i % 8])
	torch.cuda.synchronize()
	print(json.dumps({'kernel_case': args.kernel_case, 'M': M, 'launches': 8}))


# ------------------------------------------------------------------------------------------
# --workload befalix: prefill and decode of a latent-attention design beside the LLaMA path at equal size
# ------------------------------------------------------------------------------------------
BEFALIX_CASES = (
	# name, layers, hidden, intermediate, heads, head dim (unrotated), rotated, value, latent
	('2048', 8, 2048, 5504, 16, 128, 64, 128, 512),
	('4096', 4, 4096, 11008, 32, 128, 64, 128, 512),
	('8192', 2, 8192, 22016, 64, 128, 64, 128, 512),
)


def graph_us(calls, reps: int = 10) -> float:
	"""Microseconds per call: `calls` (each on its own data, together larger than L2) captured in one CUDA graph, replayed."""
	import torch
	s = torch.cuda.Stream()
	with torch.cuda.stream(s):
		for c in calls:
			c()
		s.synchronize()
		g = torch.cuda.CUDAGraph()
		with torch.cuda.graph(g, stream=s):
			for c in calls:
				c()
		for _ in range(3):
			g.replay()
		e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
		e0.record(s)
		for _ in range(reps):
			g.replay()
		e1.record(s)
		s.synchronize()
	return e0.elapsed_time(e1) * 1e3 / reps / len(calls)


def event_us(calls, reps: int = 3) -> float:
	"""The same without a graph, for calls that may not be captured."""
	import torch
	for c in calls:
		c()
	torch.cuda.synchronize()
	e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
	e0.record()
	for _ in range(reps):
		for c in calls:
			c()
	e1.record()
	torch.cuda.synchronize()
	return e0.elapsed_time(e1) * 1e3 / reps / len(calls)


def engine_rates(engine, vocab: int, steps: int, prompt_len: int = PROMPT):
	"""(prompt tokens/s, decode ms per step after the prompt) of any engine, device-timed."""
	import torch
	prompt = torch.randint(0, vocab, (engine.batch, prompt_len), generator=torch.Generator().manual_seed(3)).to(engine.device)
	for _ in range(3):
		engine.prefill(prompt)
	e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
	torch.cuda.synchronize()
	e0.record()
	for _ in range(3):
		engine.prefill(prompt)
	e1.record()
	torch.cuda.synchronize()
	rate = 3 * prompt.numel() / e0.elapsed_time(e1) * 1e3
	for _ in range(4):
		engine.step()
	torch.cuda.synchronize()
	e0.record()
	for _ in range(steps):
		engine.step()
	e1.record()
	torch.cuda.synchronize()
	return rate, e0.elapsed_time(e1) / steps


def befalix_kernels(G, engine, hbm: float, tflops: float, ctx: int = PROMPT, t: int = PROMPT):
	"""Every kernel of the design alone, on rotating copies of its operands: microseconds, and the fraction of the measured
	copy bandwidth (decode) or of the measured cuBLAS bf16 rate (prompts) that its algorithmic bytes or operations amount to."""
	import ctypes
	import torch
	from gptq_triton_b200 import _dense
	from gptq_triton_b200._lib import stream_ptr
	from gptq_triton_b200.dense import Stream, epilogue, linear, matmul, prepare_rows, project_stream
	m, cfg, dev, ctl = engine.model, engine.cfg, engine.device, engine.control
	lib, sp = _dense.lib(), lambda: stream_ptr(dev)
	layer = m.layers[0]
	mx, spec, W = layer.mixer, layer.mixer.spec, m.embed.shape[1]
	H, D, R, V, C = spec.heads, mx.D, mx.R, mx.V, mx.C
	out = {}

	def copies(w, limit=320e6):
		return [w] + [w.clone() for _ in range(max(3, min(80, int(limit / (w.numel() * w.element_size())))))]

	def record(name, us, nbytes=None, flops=None):
		r = {'us': round(us, 2)}
		if nbytes is not None:
			r['frac_hbm'] = round(nbytes / us / 1e3 / hbm, 3)
		if flops is not None:
			r['frac_tensor'] = round(flops / us / 1e6 / tflops, 3)
		out[name] = r

	x1 = torch.randn((1, W), device=dev)
	s1 = layer.mixer_norm.join(Stream(cfg.width, W, cfg.norm_eps), x1, torch.randn((1, W), device=dev))
	pos = torch.full((1,), ctx, dtype=torch.int32, device=dev)
	q = torch.randn((1, H * (D + R)), device=dev)
	gate = torch.rand((1, mx.G), device=dev)
	kv = torch.randn((1, spec.row), device=dev)
	attn = torch.empty((1, H * V), dtype=m.dtype, device=dev)

	def qkv_epi(M, posv, q_out, kv_out, gate_out, f32):
		e = _dense.Epilogue()
		e.mode, e.n_q, e.head_dim, e.rot_at, e.rot_dims, e.n_kv, e.n_gate = _dense.EPI_QKV, H * (D + R), D + R, D, spec.rot_dims, spec.row, mx.G
		e.cos_t, e.sin_t, e.pos, e.max_pos = engine.tables[0][0].data_ptr(), engine.tables[0][1].data_ptr(), posv.data_ptr(), engine.max_seq
		e.q_out, e.q_f32, e.kv_out, e.gate_out, e.status = q_out.data_ptr(), int(f32), kv_out.data_ptr(), gate_out.data_ptr(), _dense.status_ptr(ctl).value
		return e
	esz = lambda w: w.numel() * w.element_size()
	e = qkv_epi(1, pos, q, kv, gate, True)
	record('decode in-projection', graph_us([lambda w=w: project_stream(s1, w, e, ctl) for w in copies(mx.w_in)]), esz(mx.w_in))
	S = ctx + 1
	caches = [torch.randn((1, engine.max_seq, spec.row), device=dev).to(m.dtype) for _ in range(max(4, min(120, int(320e6 / (S * spec.row * 2)))))]
	args = []
	keep = []
	for w_uk, w_uv, c in zip(copies(mx.w_uk), copies(mx.w_uv), caches):
		a = mx.arguments(c, pos, 1, engine.tables[0], cfg.norm_eps, ctl, kv)
		keep.append((mx.absorbed_buffers(a, q, gate, attn, engine.max_seq), w_uk, w_uv))
		a.w_uk, a.w_uv = w_uk.data_ptr(), w_uv.data_ptr()
		args.append(a)
	call = lambda fn, a: _dense.check(fn(ctypes.byref(a), 0, sp()), 'bench')
	call(lib.dense_latent_absorb, args[0])
	record('decode absorb + cache row', graph_us([lambda a=a: call(lib.dense_latent_absorb, a) for a in args]), esz(mx.w_uk))
	acc_bytes = H * args[0].splits * (C + 2) * 4
	cargs = []
	for c in caches:
		a = mx.arguments(c, pos, 1, engine.tables[0], cfg.norm_eps, ctl, kv)
		keep.append(mx.absorbed_buffers(a, q, gate, attn, engine.max_seq))
		cargs.append(a)
	record('decode attention', graph_us([lambda a=a: call(lib.dense_latent_attend, a) for a in cargs]), S * spec.row * 2)
	record('decode merge + value', graph_us([lambda a=a: call(lib.dense_latent_value, a) for a in args]), esz(mx.w_uv) + acc_bytes)
	record('decode out-projection', graph_us([lambda w=w: linear(attn, w, ctl) for w in copies(mx.w_o)]), esz(mx.w_o))
	gu, down = layer.mlp.gate_up, layer.mlp.down
	act = torch.empty((1, down.shape[1]), dtype=m.dtype, device=dev)
	record('decode gate/up', graph_us([lambda w=w: project_stream(s1, w, layer.mlp.gated(act), ctl) for w in copies(gu)]), esz(gu))
	record('decode down', graph_us([lambda w=w: linear(act, w, ctl) for w in copies(down)]), esz(down))
	logits = torch.empty((1, (cfg.vocab_size + 15) // 16 * 16), device=dev)
	record('decode logits', graph_us([lambda w=w: project_stream(s1, w, epilogue(_dense.EPI_LOGITS, logits), ctl, keep=False, final=m.norm) for w in copies(m.embed)]), esz(m.embed))
	# the attention block as a whole (LLaMA runs it as one kernel)
	parts = ['decode in-projection', 'decode absorb + cache row', 'decode attention', 'decode merge + value', 'decode out-projection']
	record('decode attention block (sum)', sum(out[n]['us'] for n in parts), esz(mx.w_in) + esz(mx.w_uk) + esz(mx.w_uv) + esz(mx.w_o) + S * spec.row * 2)
	# ---- prompt of t tokens ----
	xs = torch.randn((t, W), device=dev)
	st = layer.mixer_norm.join(Stream(cfg.width, W, cfg.norm_eps), xs, torch.randn((t, W), device=dev))
	record('prompt rows (norm, residual)', graph_us([lambda: prepare_rows(st, ctl, m.dtype, True)] * 4), t * W * (4 + 4 + 4 + 2))
	h = torch.randn((t, W), device=dev).to(m.dtype)
	posp = torch.arange(t, dtype=torch.int32, device=dev)
	qp = torch.empty((t, H * (D + R)), dtype=m.dtype, device=dev)
	kvp, gp = torch.randn((t, spec.row), device=dev), torch.rand((t, mx.G), device=dev)
	ep = qkv_epi(t, posp, qp, kvp, gp, False)
	gemm = lambda name, fn, w, M=t: record(name, graph_us(fn), flops=2.0 * M * w.shape[0] * w.shape[1])
	gemm('prompt in-projection', [lambda w=w: matmul(h, w, ep, ctl) for w in copies(mx.w_in)], mx.w_in)
	ap = mx.arguments(caches[0], posp, t, engine.tables[0], cfg.norm_eps, ctl, kvp)
	record('prompt cache rows', graph_us([lambda: call(lib.dense_latent_append, ap)] * 4), t * spec.row * 6)
	lat = caches[0][0, :t, :C]
	k, vt = torch.empty((t, H * D), dtype=m.dtype, device=dev), torch.empty((H * V, (t + 15) // 16 * 16), dtype=m.dtype, device=dev)
	gemm('prompt expand keys', [lambda w=w: matmul(lat, w, epilogue(_dense.EPI_T, k), ctl) for w in copies(mx.w_uk)], mx.w_uk)
	gemm('prompt expand values', [lambda w=w: matmul(w, lat, epilogue(_dense.EPI_T, vt), ctl) for w in copies(mx.w_uv)], mx.w_uv)
	op = torch.empty((t, H * V), dtype=m.dtype, device=dev)
	p = _dense.LatentPrefill()
	p.t, p.start, p.S, p.heads, p.dim, p.rot_dim, p.vdim, p.kv_rank, p.scale = t, 0, t, H, D, R, V, C, spec.scale
	p.q, p.k, p.vt, p.ldv, p.cache, p.gate, p.gate_ld = qp.data_ptr(), k.data_ptr(), vt.data_ptr(), vt.stride(0), caches[0].data_ptr(), gp.data_ptr(), gp.stride(0)
	p.out, p.out_ld, p.status = op.data_ptr(), op.stride(0), _dense.status_ptr(ctl).value
	us = graph_us([lambda: _dense.check(lib.dense_latent_prefill(ctypes.byref(p), sp()), 'bench')] * 4)
	record('prompt attention', us, flops=float(t) * (t + 1) * H * (D + R + V))
	gemm('prompt out-projection', [lambda w=w: linear(op, w, ctl) for w in copies(mx.w_o)], mx.w_o)
	actp = torch.empty((t, down.shape[1]), dtype=m.dtype, device=dev)
	gemm('prompt gate/up', [lambda w=w: matmul(h, w, layer.mlp.gated(actp), ctl) for w in copies(gu)], gu)
	gemm('prompt down', [lambda w=w: linear(actp, w, ctl) for w in copies(down)], down)
	return out


def llama_kernels(G, engine, hbm: float, tflops: float, ctx: int = PROMPT, t: int = PROMPT):
	"""The like kernels of the 4-bit LLaMA engine, the same way (weights rotate over the layers)."""
	import torch
	import torch.nn.functional as F
	from gptq_triton_b200.fused_attention import qkv_attn_oproj_decode, qkv_attn_oproj_scratch
	from gptq_triton_b200.llama import causal_mask
	cfg, dev = engine.cfg, engine.device
	L = engine.model.model.layers
	hid, inter, H = cfg.hidden_size, cfg.intermediate_size, cfg.num_attention_heads
	out = {}

	def record(name, us, nbytes=None, flops=None):
		out[name] = {'us': round(us, 2), **({'frac_hbm': round(nbytes / us / 1e3 / hbm, 3)} if nbytes is not None else {'frac_tensor': round(flops / us / 1e6 / tflops, 3)})}
	x1 = torch.randn((1, 1, hid), device=dev).half()
	ss = x1.float().pow(2).view(1, hid // 32, 32).sum(-1).contiguous()
	pos = torch.full((1,), ctx, dtype=torch.int32, device=dev)
	rot = [l for _ in range(max(1, 16 // len(L))) for l in L]
	layers = list(enumerate(L))
	if engine._one_kernel_attention(L[0].self_attn):
		cos, sin = L[0].self_attn.tables(dev, engine.max_seq)
		scratch = qkv_attn_oproj_scratch(H, hid, dev)
		def block(i, l):
			a, o = l.self_attn, l.self_attn.o_proj
			qw, _, _ = a.qkv_proj.kernel_operands()
			return qkv_attn_oproj_decode(a.qkv_proj.groupsize, x1, qw, a.qkv_proj.scales, a.qkv_proj.qzeros, cos, sin, pos, engine.kcache[i], engine.vcache[i], H,
										 o.groupsize, o.qweight, o.scales, o.qzeros, scratch, residual=x1, sumsq_out=engine.ss_attn, rms_weight=l.input_layernorm.weight,
										 rms_eps=1e-6, sumsq_in=ss)
		record('decode attention block (qkv, attention, o)', graph_us([lambda i=i, l=l: block(i, l) for i, l in layers]),
			   quantised_bytes(hid, 3 * hid) + quantised_bytes(hid, hid) + 2 * H * (ctx + 1) * 256)
	y1 = torch.randn((1, 1, inter), device=dev).half()
	record('decode gate/up', graph_us([lambda l=l: l.mlp.intermediate(x1, rms_weight=l.post_attention_layernorm.weight, rms_eps=1e-6, sumsq_in=ss) for l in rot]), quantised_bytes(hid, 2 * inter))
	record('decode down', graph_us([lambda l=l: l.mlp.down_proj(y1, residual=x1, sumsq_out=engine.ss_mlp) for l in rot]), quantised_bytes(inter, hid))
	record('decode o', graph_us([lambda l=l: l.self_attn.o_proj(x1, residual=x1, sumsq_out=engine.ss_attn) for l in rot]), quantised_bytes(hid, hid))
	from gptq_triton_b200.fused_attention import attn_decode
	q1 = torch.randn((1, H, 1, 128), device=dev).half()
	kcs = [(torch.randn_like(engine.kcache[0]), torch.randn_like(engine.vcache[0])) for _ in range(max(4, int(320e6 / (2 * H * ctx * 256))))]
	record('decode attention', graph_us([lambda k=k, v=v: attn_decode(q1, k, v, pos, ctx + 1) for k, v in kcs]), 2 * H * (ctx + 1) * 256)
	xp = (torch.randn((1, t, hid), device=dev) * 0.5).half()
	yp = (torch.randn((1, t, inter), device=dev) * 0.5).half()
	pp = torch.arange(t, device=dev, dtype=torch.int32)[None]
	record('prompt qkv', event_us([lambda i=i, l=l: l.self_attn.project_qkv(xp, pp, kv_cache=(engine.kcache[i], engine.vcache[i])) for i, l in layers]), flops=2.0 * t * hid * 3 * hid)
	record('prompt o', event_us([lambda l=l: l.self_attn.o_proj(xp) for l in rot]), flops=2.0 * t * hid * hid)
	record('prompt gate/up', event_us([lambda l=l: l.mlp.intermediate(xp) for l in rot]), flops=4.0 * t * hid * inter)
	record('prompt down', event_us([lambda l=l: l.mlp.down_proj(yp) for l in rot]), flops=2.0 * t * hid * inter)
	q, k, v = (torch.randn((1, H, t, 128), device=dev).half() for _ in range(3))
	mask = causal_mask(t, 0, dev)
	record('prompt attention', event_us([lambda: F.scaled_dot_product_attention(q, k, v, attn_mask=mask)] * 4), flops=float(t) * (t + 1) * H * 256)
	return out


def befalix_config(G, layers, hid, inter, H, D, R, V, C, vocab=32000):
	layer = {'type': 'latent_attention', 'mlp': {'kind': 'dense', 'ff': inter},
			 'mixer': {'heads': H, 'dim': D, 'rot_dim': R, 'vdim': V, 'kv_rank': C, 'scale': (D + R) ** -0.5, 'rot': {'base': 10000.0, 'dims': R}}}
	return G.BefalixConfig.from_dict({'vocab': vocab, 'width': hid, 'norm': {'eps': 1e-6}, 'residual_mult': 1.0, 'logit_scale': 1.0, 'layers': [layer] * layers})


def befalix_work(model, layers: int, ctx: int, t: int):
	"""(bytes of a decode step at context ctx, operations of a prompt of t tokens)."""
	s = model.layers[0].mixer.spec
	nbytes = sum(b.numel() * b.element_size() for b in model.buffers()) + layers * ctx * s.row * 2
	return nbytes, t * 2.0 * sum(b.numel() for l in model.layers for b in l.buffers() if b.dim() == 2) + layers * float(t) * (t + 1) * s.heads * (s.dim + s.rot_dim + s.vdim)


def befalix_arm(args):
	"""Prints one JSON line: per size, prompt tokens/s and decode ms per step of a Befalix model (bf16 weights, random) and of a
	4-bit LLaMA with the same hidden size, MLP, heads and number of layers, and every kernel's fraction of its roofline."""
	import torch
	import gptq_triton_b200 as G
	from gptq_triton_b200 import _lib
	from gptq_triton_b200.llama import LlamaConfig
	torch.cuda.set_device(0)
	dev = torch.device('cuda', 0)
	hbm, source = measured_peaks()
	peaks = ROOT / 'MEASURED_PEAKS.json'
	tflops = float(json.load(open(peaks))['bf16_tflops']) if peaks.exists() else 1590.0
	sampler = ClockSampler(0, None)
	sampler.start()
	cases = {}
	for name, layers, hid, inter, H, D, R, V, C in BEFALIX_CASES:
		if args.case and name not in args.case.split(','):
			continue
		max_seq = PROMPT + args.steps + 64
		cfg = befalix_config(G, layers, hid, inter, H, D, R, V, C)
		model = G.synthetic_befalix(cfg, seed=1, device=dev)
		engine = G.BefalixEngine(model, batch=1, max_seq=max_seq)
		rate, ms = engine_rates(engine, cfg.vocab_size, args.steps)
		nbytes, flops = befalix_work(model, layers, PROMPT + args.steps // 2, PROMPT)
		rec = {'hidden': hid, 'intermediate': inter, 'heads': H, 'layers': layers,
			   'befalix': {'prefill_tokens_s': round(rate), 'decode_ms_per_step': round(ms, 4), 'decode_tokens_s': round(1e3 / ms, 1), 'decode_frac_hbm': round(nbytes / ms / 1e6 / hbm, 3),
						   'prefill_frac_tensor': round(flops * rate / PROMPT / 1e12 / tflops, 3), 'kernels': befalix_kernels(G, engine, hbm, tflops)}}
		engine.close()
		del engine, model
		torch.cuda.empty_cache()
		lcfg = LlamaConfig(hidden_size=hid, intermediate_size=inter, num_hidden_layers=layers, num_attention_heads=H, max_position_embeddings=max_seq)
		model = G.synthetic_quantized_llama(lcfg, groupsize=GROUPSIZE, seed=1, device=dev)
		engine = G.DecodeEngine(model, batch=1, max_seq=max_seq)
		rate, ms = engine_rates(engine, lcfg.vocab_size, args.steps)
		nbytes = layers * (quantised_bytes(hid, 4 * hid) + quantised_bytes(hid, 2 * inter) + quantised_bytes(inter, hid) + 2 * H * (PROMPT + args.steps // 2) * 256) + hid * 32000 * 2
		flops = PROMPT * 2.0 * layers * (4 * hid * hid + 3 * hid * inter) + layers * float(PROMPT) * (PROMPT + 1) * H * 256
		rec['llama_4bit'] = {'prefill_tokens_s': round(rate), 'decode_ms_per_step': round(ms, 4), 'decode_tokens_s': round(1e3 / ms, 1), 'decode_frac_hbm': round(nbytes / ms / 1e6 / hbm, 3),
							 'prefill_frac_tensor': round(flops * rate / PROMPT / 1e12 / tflops, 3), 'kernels': llama_kernels(G, engine, hbm, tflops)}
		engine.close()
		del engine, model
		torch.cuda.empty_cache()
		cases[name] = rec
	print(json.dumps({'workload': 'befalix', 'prompt': PROMPT, 'batch': 1, 'data': 'synthetic', 'weights': 'befalix bf16, llama 4-bit g128 (random)', 'hbm_gbs': hbm, 'bf16_tflops': tflops,
					  'peak_source': source, 'kernel_status': _lib.kernel_status(dev), 'clocks': sampler.stop(), 'cases': cases}))


# ------------------------------------------------------------------------------------------
# --workload lifinex: differential attention and state-space layers beside the latent-attention design at equal size
# ------------------------------------------------------------------------------------------
def lifinex_config(G, runs, hid, inter, vocab=32000, max_positions=4096):
	"""`runs` layer runs, attention and state-space layers in turn (runs = 8: six layers, two of them run twice)."""
	ff = {'kind': 'dense', 'ff': inter}
	H = hid // 128
	att = {'type': 'attention', 'mlp': ff, 'mixer': {'heads': H, 'kv_heads': H // 4, 'dim': 64, 'vdim': 128, 'scale': 0.125, 'softcap': 25.0, 'diff': 0.4}}
	ssm = {'type': 'mamba2', 'mlp': ff, 'mixer': {'heads': hid // 32, 'vdim': 64, 'state': 128, 'groups': 8, 'conv': 4, 'norm_groups': 8}}
	layers, loop = {8: ([att, ssm] * 3, (2, 4, 2)), 4: ([ssm, att, ssm], (1, 2, 2)), 2: ([att, ssm], (0, 1, 1))}[runs]
	return G.LifinexConfig.from_dict({'vocab': vocab, 'width': hid, 'layers': layers, 'norm': {'eps': 1e-6}, 'max_positions': max_positions, 'token_side': {'dim': 256},
									  'loop': dict(zip(('start', 'stop', 'times'), loop))})


def lifinex_work(model, ctx: int, t: int):
	"""(bytes of a decode step at context ctx, operations of a prompt of t tokens) that the design needs: weights as often as
	their layers run, cache rows, carried state (read and written); products, both attention maps, the recurrence's state
	update and output."""
	cfg = model.config
	size = lambda m: sum(b.numel() * b.element_size() for b in m.buffers())
	mats = lambda m: sum(b.numel() for b in m.buffers() if b.dim() == 2 and b.shape[0] > 32)
	nbytes, flops = model.head.numel() * 2, 0.0
	for i, entry in cfg.runs():
		layer, s = model.layers[i], cfg.layers[i].mixer
		nbytes += size(layer)
		flops += 2.0 * t * mats(layer)
		if entry is not None:
			nbytes += model.loop_x.numel() * 2
			flops += 2.0 * t * model.loop_x.numel()
		if hasattr(s, 'softcap'):
			nbytes += ctx * s.kv_heads * (s.maps * s.dim + s.vdim) * 2
			flops += float(t) * (t + 1) * s.heads * s.maps * (s.dim + s.vdim)
		else:
			nbytes += 2 * s.heads * s.vdim * s.state * 4
			flops += 4.0 * t * s.heads * s.vdim * s.state
	if cfg.loop is not None:
		nbytes += model.loop_x0.numel() * 2
		flops += 2.0 * t * model.loop_x0.numel()
	return nbytes, flops


def lifinex_kernels(G, engine, hbm: float, tflops: float, ctx: int = PROMPT, t: int = PROMPT):
	"""Every kernel of the design alone, on rotating copies of its operands (see befalix_kernels)."""
	import ctypes
	import torch
	from gptq_triton_b200 import _dense
	from gptq_triton_b200._lib import stream_ptr
	from gptq_triton_b200.cache import StaticCache
	from gptq_triton_b200.dense import Stream, epilogue, linear, matmul, padded, prepare_rows, project_stream
	m, cfg, dev, ctl = engine.model, engine.cfg, engine.device, engine.control
	lib, sp = _dense.lib(), lambda: stream_ptr(dev)
	W, bf = m.embed.shape[1], torch.bfloat16
	att = next(l for l in m.layers if hasattr(l.mixer, 'lam'))
	ssm = next(l for l in m.layers if not hasattr(l.mixer, 'lam'))
	out = {}

	def record(name, us, nbytes=None, flops=None):
		r = {'us': round(us, 2)}
		if nbytes is not None:
			r['frac_hbm'] = round(nbytes / us / 1e3 / hbm, 3)
		if flops is not None:
			r['frac_tensor'] = round(flops / us / 1e6 / tflops, 3)
		out[name] = r
	esz = lambda *ws: sum(w.numel() * w.element_size() for w in ws)
	copies = lambda w, limit=320e6: [w] + [w.clone() for _ in range(max(3, min(80, int(limit / esz(w)))))]
	call = lambda fn, *a: _dense.check(fn(*a, sp()), 'bench')

	def rows(M):
		return Stream(cfg.width, W, cfg.norm_eps).then(torch.randn((M, W), device=dev), torch.randn((M, W), device=dev))
	for M, phase in ((1, 'decode'), (t, 'prompt')):
		decode = M == 1
		st = rows(M)
		h = torch.randn((M, W), device=dev).to(bf)
		start = ctx if decode else 0
		pos = torch.arange(start, start + M, dtype=torch.int32, device=dev)

		def gemm(name, w, epi, norm=None, x=None):
			if decode and x is None:          # the kernel forms its rows itself
				fns = [lambda c=c: project_stream(st, c, epi, ctl, final=norm) for c in copies(w)]
			else:
				xin = h if x is None else x
				fns = [lambda c=c: matmul(xin, c, epi, ctl) for c in copies(w)]
			record(f'{phase} {name}', graph_us(fns), **({'nbytes': esz(w)} if decode else {'flops': 2.0 * M * w.numel()}))
		f32 = lambda n: torch.empty((M, n), device=dev)
		if not decode:
			record('prompt rows (residual, norm)', graph_us([lambda: prepare_rows(st, ctl, bf, True, att.mixer_norm)] * 4), t * W * (4 + 4 + 4 + 2))
		# ---- attention ----
		mx, s = att.mixer, att.mixer.spec
		raw = torch.randn((M, mx.w_in.shape[0]), device=dev).to(torch.float32 if decode else bf)
		gemm('attention in-projection', mx.w_in, epilogue(_dense.EPI_F32 if decode else _dense.EPI_T, raw), att.mixer_norm)
		n = max(2, min(80, int(320e6 / (ctx * s.kv_heads * (s.maps * mx.D + mx.V) * 2)))) if decode else 2
		caches = [{k: torch.randn_like(v.float()).to(bf) for k, v in StaticCache([s.cache_layout(engine.max_seq)], 1, bf, dev)[0].items()} for _ in range(n)]
		o = torch.empty((M, s.heads * mx.V), dtype=bf, device=dev)
		keep, args = [], []
		for c in caches:
			a = mx.arguments(raw, c, pos, M, cfg.norm_eps, ctl)
			keep.append(mx.buffers(a, o, engine.max_seq if decode else 1))
			args.append(a)
		row = s.kv_heads * (s.maps * mx.D + mx.V)
		if decode:
			call(lib.dense_gqa_append, ctypes.byref(args[0]), 0)
			record('decode attention norms, cache row', graph_us([lambda a=a: call(lib.dense_gqa_append, ctypes.byref(a), 0) for a in args]), esz(raw) * 2)
			for a in args:
				call(lib.dense_gqa_append, ctypes.byref(a), 0)
			record('decode attention', graph_us([lambda a=a: call(lib.dense_gqa_attend, ctypes.byref(a), 0) for a in args]), (ctx + 1) * row * 2)
			record('decode attention merge', graph_us([lambda a=a: call(lib.dense_gqa_merge, ctypes.byref(a), 0) for a in args]),
				   s.heads * s.maps * args[0].splits * (mx.V + 2) * 4)
		else:
			record('prompt attention norms, cache rows', graph_us([lambda a=a: call(lib.dense_gqa_append, ctypes.byref(a), 0) for a in args] * 2), esz(raw) + M * (row + s.heads * s.maps * mx.D) * 2)
			record('prompt attention', graph_us([lambda a=a: call(lib.dense_gqa_prefill, ctypes.byref(a), 0) for a in args] * 2), flops=float(t) * (t + 1) * s.heads * s.maps * (s.dim + s.vdim))
		y = f32(W)
		gemm('attention out-projection', mx.w_o, epilogue(_dense.EPI_F32, y), x=o)
		if decode:
			parts = ['decode attention in-projection', 'decode attention norms, cache row', 'decode attention', 'decode attention merge', 'decode attention out-projection']
			record('decode attention block (sum)', sum(out[k]['us'] for k in parts), esz(mx.w_in, mx.w_o) + (ctx + 1) * row * 2)
		# ---- state space ----
		mx, s = ssm.mixer, ssm.mixer.spec
		if decode:
			raw = torch.randn((M, mx.w_in.shape[0]), device=dev)
			steps, e = raw[:, mx.dt_at:], epilogue(_dense.EPI_F32, raw)
		else:
			raw, steps = torch.randn((M, mx.dt_at), device=dev).to(bf), torch.randn((M, mx.w_in.shape[0] - mx.dt_at), device=dev)
			e = epilogue(_dense.EPI_MIXED, raw)
			e.n_q, e.n_kv, e.kv_out = mx.dt_at, steps.shape[1], steps.data_ptr()
		gemm('state-space in-projection', mx.w_in, e, ssm.mixer_norm)
		state = 4 * s.heads * s.vdim * s.state
		g = torch.randn((M, padded(s.inner)), device=dev).to(raw.dtype)
		args = []
		for _ in range(max(2, min(80, int(320e6 / state))) if decode else 2):
			c = StaticCache([s.cache_layout()], 1, bf, dev)[0]
			a = mx.arguments(raw, steps, c, pos, M, g, ctl)
			keep.append((c, None if decode else mx.portion_buffers(a, bf, True)))
			args.append(a)
		if decode:
			record('decode state-space step', graph_us([lambda a=a: call(lib.dense_ssm_step, ctypes.byref(a)) for a in args]), 2 * state + esz(raw, g) + 4 * (s.taps + 1) * a.conv_ld)
		else:
			record('prompt state-space convolution', graph_us([lambda a=a: call(lib.dense_ssm_conv, ctypes.byref(a), 0) for a in args] * 2), M * a.conv_ld * 4)
			record('prompt state-space recurrence', graph_us([lambda a=a: call(lib.dense_ssm_chunked, ctypes.byref(a)) for a in args] * 2), M * a.conv_ld * 2 + M * s.inner * 4 + esz(steps) + 2 * state)
			gs = Stream(s.inner, padded(s.inner), cfg.norm_eps, x=g)
			record('prompt state-space norm', graph_us([lambda: prepare_rows(gs, ctl, bf, False, mx.norm)] * 4), M * s.inner * 4)
		if decode:
			gs = Stream(s.inner, padded(s.inner), cfg.norm_eps, x=g)
			record('decode state-space norm, out-projection', graph_us([lambda c=c: project_stream(gs, c, epilogue(_dense.EPI_F32, y), ctl, keep=False, final=mx.norm) for c in copies(mx.w_o)]),
				   esz(mx.w_o))
		else:
			gemm('state-space out-projection', mx.w_o, epilogue(_dense.EPI_F32, y), x=g)
		# ---- feed-forward, side input, pass entry, logits ----
		act = torch.empty((M, att.mlp.down.shape[1]), dtype=bf, device=dev)
		gemm('gate/up', att.mlp.gate_up, att.mlp.gated(act), att.mlp_norm)
		gemm('down', att.mlp.down, epilogue(_dense.EPI_F32, y), x=act)
		tok = torch.arange(M, device=dev) % cfg.vocab_size
		side = torch.empty((M, att.side.gate.shape[0]), dtype=bf, device=dev)
		gemm('side gate', att.side.gate, att.side.gated(side, m.side, tok))
		gemm('side projection', att.side.proj, epilogue(_dense.EPI_F32, y), x=side)
		gemm('pass entry', m.loop_x, epilogue(_dense.EPI_F32, y))
		if decode:
			logits = torch.empty((1, padded(cfg.vocab_size)), device=dev)
			record('decode logits', graph_us([lambda w=w: project_stream(st, w, epilogue(_dense.EPI_LOGITS, logits), ctl, keep=False, final=m.norm) for w in copies(m.head)]), esz(m.head))
	return out


def lifinex_arm(args):
	"""Prints one JSON line: per size, prompt tokens/s and decode ms per step of a Lifinex model and of a Befalix model (both
	bf16, random weights) with the same hidden size, MLP and number of layer runs, and every kernel's fraction of its roofline."""
	import torch
	import gptq_triton_b200 as G
	from gptq_triton_b200 import _lib
	torch.cuda.set_device(0)
	dev = torch.device('cuda', 0)
	hbm, source = measured_peaks()
	peaks = ROOT / 'MEASURED_PEAKS.json'
	tflops = float(json.load(open(peaks))['bf16_tflops']) if peaks.exists() else 1590.0
	sampler = ClockSampler(0, None)
	sampler.start()
	cases = {}
	for name, runs, hid, inter, H, D, R, V, C in BEFALIX_CASES:
		if args.case and name not in args.case.split(','):
			continue
		max_seq = PROMPT + args.steps + 64
		cfg = lifinex_config(G, runs, hid, inter)
		engine = G.LifinexEngine(G.synthetic_lifinex(cfg, seed=1, device=dev), batch=1, max_seq=max_seq)
		rate, ms = engine_rates(engine, cfg.vocab_size, args.steps)
		nbytes, flops = lifinex_work(engine.model, PROMPT + args.steps // 2, PROMPT)
		rec = {'hidden': hid, 'intermediate': inter, 'layer_runs': runs,
			   'lifinex': {'prefill_tokens_s': round(rate), 'decode_ms_per_step': round(ms, 4), 'decode_tokens_s': round(1e3 / ms, 1), 'decode_frac_hbm': round(nbytes / ms / 1e6 / hbm, 3),
						   'prefill_frac_tensor': round(flops * rate / PROMPT / 1e12 / tflops, 3), 'kernels': lifinex_kernels(G, engine, hbm, tflops)}}
		engine.close()
		del engine
		torch.cuda.empty_cache()
		cfg = befalix_config(G, runs, hid, inter, H, D, R, V, C)
		engine = G.BefalixEngine(G.synthetic_befalix(cfg, seed=1, device=dev), batch=1, max_seq=max_seq)
		rate, ms = engine_rates(engine, cfg.vocab_size, args.steps)
		nbytes, flops = befalix_work(engine.model, runs, PROMPT + args.steps // 2, PROMPT)
		rec['befalix'] = {'prefill_tokens_s': round(rate), 'decode_ms_per_step': round(ms, 4), 'decode_tokens_s': round(1e3 / ms, 1), 'decode_frac_hbm': round(nbytes / ms / 1e6 / hbm, 3),
						  'prefill_frac_tensor': round(flops * rate / PROMPT / 1e12 / tflops, 3), 'kernels': befalix_kernels(G, engine, hbm, tflops)}
		engine.close()
		del engine
		torch.cuda.empty_cache()
		cases[name] = rec
	print(json.dumps({'workload': 'lifinex', 'prompt': PROMPT, 'batch': 1, 'data': 'synthetic', 'weights': 'bf16 (random)', 'hbm_gbs': hbm, 'bf16_tflops': tflops,
					  'peak_source': source, 'kernel_status': _lib.kernel_status(dev), 'clocks': sampler.stop(), 'cases': cases}))


def main():
	ap = argparse.ArgumentParser()
	ap.add_argument('--gpus', type=int, default=1)
	ap.add_argument('--steps', type=int, default=64)
	ap.add_argument('--warmup', type=int, default=8)
	ap.add_argument('--impl', default='b200', choices=['b200', 'reference'])
	ap.add_argument('--layers', type=int, default=0, help='debug: fewer decoder layers')
	ap.add_argument('--no-cpu-baseline', action='store_true')
	ap.add_argument('--no-parity', action='store_true', help='skip the greedy-decoding parity check before the timed region')
	ap.add_argument('--no-prefill', action='store_true', help='skip the prefill-kernel record')
	ap.add_argument('--config4', default='auto', choices=['auto', 'on', 'off'], help='also measure the 65B-architecture batch-16 configuration as a sub-record (auto: with 2 or more GPUs)')
	ap.add_argument('--workload', default='llama7b', choices=['llama7b', 'llama65b-b16', 'befalix', 'lifinex'],
					help='llama65b-b16: 65B architecture, batch 16 (tensor-parallel runs); befalix: latent-attention models beside LLaMA at equal sizes; lifinex: '
						 'differential attention and state-space layers beside befalix at equal sizes')
	ap.add_argument('--case', default='', help='befalix, lifinex: sizes to run (2048, 4096, 8192), separated by commas')
	ap.add_argument('--no-graph', action='store_true', help='do not capture the decode step in a CUDA graph')
	ap.add_argument('--kernel-case', default=None, choices=['gateup', 'qkv', 'o', 'down', 'prefill', 'attn', 'lmhead', 'chain', 'qkvattn', 'latent-prefill', 'latent-decode', 'gqa-prefill', 'ssm-prefill', 'lifinex-decode'], help='profiling aid: run a few launches of one kernel and exit')
	ap.add_argument('--m', type=int, default=1, help='batch rows for --kernel-case')
	ap.add_argument('--heads', type=int, default=32, help='heads for --kernel-case attn, latent-prefill and gqa-prefill')
	args = ap.parse_args()
	if args.kernel_case:
		kernel_case(args)
	elif args.workload == 'befalix':
		befalix_arm(args)
	elif args.workload == 'lifinex':
		lifinex_arm(args)
	elif args.impl == 'reference':
		reference_arm(args)
	else:
		gpu_arm(args)


if __name__ == '__main__':
	main()
