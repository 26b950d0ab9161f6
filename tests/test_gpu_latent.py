"""Latent-attention models on the GPU against the plain CPU oracle: every kernel alone, prompts, portions, decode steps, reuse of
the cache, single keys that stand out at every kind of border, greedy generation through the engine, command line and replay."""
import ctypes
import json
import os
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import latent_models as LM
from oracle import latent_oracle as O

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
F32, B16 = torch.float32, torch.bfloat16
REL = {F32: 2e-6, B16: 6e-3}          # of the largest result: fp32 sums; one bf16 rounding of operands or result


@pytest.fixture(scope='module')
def control():
	from gptq_triton_b200 import _dense
	return _dense.control_buffer(torch.device('cuda', 0))


@pytest.fixture(autouse=True)
def healthy():
	yield
	from gptq_triton_b200 import _lib
	assert _lib.kernel_status() == 0


def rnd(*shape, seed=0, dtype=F32):
	return torch.randn(shape, generator=torch.Generator().manual_seed(seed)).to(dtype)


def close(got, want, rel):
	want = want.double()
	return float((got.double().cpu() - want).abs().max()) <= rel * float(want.abs().max())


# ---- the kernels alone ---------------------------------------------------------------------------------------------------

@pytest.mark.parametrize('dtype', [F32, B16])
@pytest.mark.parametrize('M,K,N', [(1, 48, 80), (2, 1040, 33), (5, 272, 528), (8, 2080, 16), (9, 64, 48), (130, 336, 515), (300, 1088, 272),
									 (1, 4112, 40), (3, 8208, 256), (6, 2064, 144), (1200, 2064, 200), (2500, 1040, 500), (9, 1040, 16)])
def test_projection(control, dtype, M, K, N):
	from gptq_triton_b200 import _dense
	from gptq_triton_b200.dense import epilogue, linear, matmul
	x, w = rnd(M, K, seed=1, dtype=dtype), rnd(N, K, seed=2, dtype=dtype) * K ** -0.5
	ref = x.double() @ w.double().T
	y = linear(x.cuda(), w.cuda(), control)
	assert y.dtype == F32 and close(y[:, :N], ref, 2e-6)          # fp32 accumulation of exact products in both formats
	y = linear(x.cuda(), w.cuda(), control, out_dtype=dtype)
	assert y.dtype == dtype and close(y[:, :N], ref, REL[dtype])
	wide = torch.zeros((N, K + 16), dtype=dtype, device='cuda')       # weights that are columns of a wider matrix
	wide[:, :K] = w.cuda()
	out = torch.zeros((M, (N + 15) // 16 * 16), device='cuda')
	matmul(x.cuda(), wide[:, :K], epilogue(_dense.EPI_F32, out, 0.5), control)
	assert close(out[:, :N], 0.5 * ref, 2e-6)


@pytest.mark.parametrize('dtype', [F32, B16])
@pytest.mark.parametrize('M', [1, 2, 3, 8, 40, 200])
def test_mlp_sublayer(control, dtype, M):
	"""Row preparation (residual, post-norm), fused gate/up, down."""
	from gptq_triton_b200.dense import DenseMLP, PostNorm, Stream, padded
	width, ff, eps = 90, 77, 1e-4
	g, u, d = (rnd(*s, seed=i, dtype=B16) * s[1] ** -0.5 for i, s in enumerate([(ff, width), (ff, width), (width, ff)]))
	nw, nb, ls = 1 + 0.2 * rnd(width, seed=5), 0.1 * rnd(width, seed=6), 1 + 0.2 * rnd(width, seed=7)
	x, y = rnd(M, width, seed=8), 3 * rnd(M, width, seed=9) + 2          # a mean that is not small
	pad = lambda t: torch.nn.functional.pad(t, (0, padded(width) - width)).cuda()
	norm = PostNorm(nw, nb, ls, 0.7).cuda()
	stream = norm.join(Stream(width, padded(width), eps), pad(x), pad(y))
	mlp = DenseMLP(g.to(dtype), u.to(dtype), d.to(dtype)).cuda()
	got_x, got_y = mlp(stream, control)
	ref_x = x.double() + 0.7 * O.layer_norm(y.double(), nw.double(), nb.double(), eps) * ls.double()
	assert close(got_x[:, :width], ref_x, 2e-6)
	assert got_x.shape[1] == width or float(got_x[:, width:].abs().max()) == 0
	assert close(got_y[:, :width], O.dense_ff(ref_x, g.double(), u.double(), d.double()), REL[dtype] * 2)


@pytest.mark.parametrize('dtype', [F32, B16])
@pytest.mark.parametrize('M', [1, 2, 7])
@pytest.mark.parametrize('width', [50, 4100])          # rows shorter and longer than the registers of a CTA hold
def test_rows_and_logits(control, dtype, M, width):
	"""Embedding lookup, final norm, logits and greedy choice, formed inside the projection or ahead of it."""
	from gptq_triton_b200 import _dense
	from gptq_triton_b200.dense import LayerNorm, PostNorm, Stream, epilogue, pad_to, padded, prepare_rows, project_stream
	V, eps = 83, 1e-6
	table = rnd(V, width, seed=1, dtype=B16)
	fw, fb = 1 + 0.2 * rnd(width, seed=2), 0.3 * rnd(width, seed=3)
	y = rnd(M, width, seed=4)
	tok = torch.arange(M) * 11 % V
	dev_table = pad_to(table.to(dtype), V, padded(width)).cuda()
	one = PostNorm(torch.ones(width), torch.zeros(width), None, 0.5).cuda()
	s = Stream(width, padded(width), eps, table=dev_table, token=tok.cuda())
	h, x = prepare_rows(s, control, dtype, True)
	assert torch.equal(x[:, :width].cpu(), table[tok].float()) and torch.equal(h[:, :width].cpu(), table[tok].to(dtype))
	s2 = one.join(s, x, pad_to(y, M, padded(width)).cuda())
	ref_x = table[tok].double() + 0.5 * O.layer_norm(y.double(), torch.ones(width).double(), torch.zeros(width).double(), eps)
	ref_h = O.layer_norm(ref_x, fw.double(), fb.double(), eps)
	final = LayerNorm(fw, fb).cuda()
	h, x2 = prepare_rows(s2, control, dtype, True, final)
	assert close(x2[:, :width], ref_x, 2e-6) and close(h[:, :width], ref_h, 3e-6 if dtype == F32 else 4e-3)
	logits = torch.empty((M, padded(V)), device='cuda')
	nxt, pos = torch.zeros((M, 1), dtype=torch.int64, device='cuda'), torch.full((M, 1), 4, dtype=torch.int32, device='cuda')
	e = epilogue(_dense.EPI_LOGITS, logits, 1.5)
	e.ticket, e.best, e.tok, e.pos_inout = control.data_ptr(), control.data_ptr() + 256, nxt.data_ptr(), pos.data_ptr()
	for _ in range(2):          # the counters must be left as they were found
		project_stream(s2, dev_table, e, control, keep=False, final=final)
	assert close(logits[:, :V], 1.5 * (ref_h @ table.double().T), 3e-6 if dtype == F32 else 6e-3)
	assert torch.equal(nxt.cpu(), logits[:, :V].argmax(-1, keepdim=True).cpu()) and pos.unique().tolist() == [6]


def test_greedy_choice_takes_the_lowest_index_of_equal_logits(control):
	from gptq_triton_b200 import _dense
	from gptq_triton_b200.dense import epilogue, matmul
	w = torch.zeros((70, 16), dtype=B16, device='cuda')
	w[[33, 12, 66], 0] = 1.0
	x = torch.zeros((2, 16), dtype=B16, device='cuda')
	x[:, 0] = torch.tensor([2.0, -2.0])
	logits = torch.empty((2, 80), device='cuda')
	tok, pos = torch.zeros(2, dtype=torch.int64, device='cuda'), torch.zeros(2, dtype=torch.int32, device='cuda')
	e = epilogue(_dense.EPI_LOGITS, logits)
	e.ticket, e.best, e.tok, e.pos_inout = control.data_ptr(), control.data_ptr() + 256, tok.data_ptr(), pos.data_ptr()
	matmul(x, w, e, control)
	assert tok.tolist() == [12, 0] and pos.tolist() == [1, 1]


def attention_case(dtype, H, D, R, V, C, t, start, seed=0):
	"""A mixer on its own with bf16 weights, latents that the cache already holds for `start` positions, and the stream rows of
	t further tokens."""
	from gptq_triton_b200.latent_attention import LatentAttention, LatentAttentionSpec, interleaved_rope_tables
	width = 64
	spec = LatentAttentionSpec(H, D, R, V, C, 1000.0, R, 0.4)
	shapes = {'q': (H * (D + R), width), 'dkv': (C + R, width), 'dkv.norm': (C,), 'uk': (H * D, C), 'uv': (H * V, C), 'g': (H, width), 'o': (width, H * V)}
	W = {k: (rnd(*s, seed=seed + i, dtype=B16) * (s[-1] ** -0.5 if len(s) == 2 else 0.5)) for i, (k, s) in enumerate(shapes.items())}
	mix = LatentAttention(spec, *(W[k].to(dtype) for k in ('q', 'uk', 'uv', 'g', 'o', 'dkv', 'dkv.norm'))).cuda()
	mixer = {'heads': H, 'dim': D, 'rot_dim': R, 'vdim': V, 'kv_rank': C, 'rot': {'base': 1000.0, 'dims': R}, 'scale': 0.4}
	h = rnd(start + t, width, seed=seed + 50, dtype=B16)
	return spec, mix, mixer, {k: v.double() for k, v in W.items()}, h, interleaved_rope_tables(1000.0, R, start + t + 5, 'cuda')


def run_mixer(mix, cache, h, start, tables, control, decode=False, eps=1e-5):
	from gptq_triton_b200.dense import Stream
	stream = Stream(h.shape[1], h.shape[1], eps, x=h.float().cuda())
	pos = torch.arange(start, start + h.shape[0], dtype=torch.int32, device='cuda')
	return mix(stream, cache, pos, h.shape[0], None if decode else start, tables, eps, control)[1]


@pytest.mark.parametrize('dtype', [F32, B16])
@pytest.mark.parametrize('H,D,R,V,C', [(3, 20, 10, 24, 40), (17, 64, 32, 80, 72), (2, 130, 70, 144, 520), (16, 32, 16, 16, 256), (1, 16, 128, 200, 1000)])
def test_mixer_prompt_portions_and_steps(control, dtype, H, D, R, V, C):
	t = 300
	spec, mix, mixer, W, h, tables = attention_case(dtype, H, D, R, V, C, t, 0)
	ref, latent, key_rot = O.latent_attention(h.double(), W, mixer, 1e-5, torch.arange(t))
	for cuts in ([300], [1, 2, 9, 100, 128, 52, 8]):
		cache = torch.zeros((1, t + 5, spec.row), dtype=dtype, device='cuda')
		out, p = [], 0
		for n in cuts:
			out.append(run_mixer(mix, cache, h[p:p + n], p, tables, control, decode=n == 1))
			p += n
		assert close(torch.cat(out)[:, :64], ref, 5e-6 if dtype == F32 else 1.5e-2), cuts
	from gptq_triton_b200.dense import padded
	assert close(cache[0, :t, :C], latent, 2e-6 if dtype == F32 else 5e-3)
	assert close(cache[0, :t, padded(C):padded(C) + R], key_rot, 2e-6 if dtype == F32 else 5e-3)
	assert float(cache[0, t:].abs().max()) == 0 and float(cache[..., C:padded(C)].abs().max() if padded(C) > C else 0) == 0


@pytest.mark.parametrize('dtype', [F32, B16])
@pytest.mark.parametrize('key', [0, 1, 31, 32, 127, 128, 129, 255, 256, 511, 639, 640, 641, 700])
def test_one_key_that_stands_out(control, dtype, key):
	"""One cached key's score is made far larger than all others: its value is the whole output of every query that may see it
	and no part of those before it, in the tensor-core kernel (prompts) and the absorbed one (steps), wherever its tile lies."""
	H, D, R, V, C, S = 2, 32, 16, 48, 64, 701
	spec, mix, mixer, W, h, tables = attention_case(dtype, H, D, R, V, C, S, 0, seed=7)
	latent = rnd(S, C, seed=90).double()
	latent /= latent.pow(2).mean(-1, keepdim=True).sqrt()
	key_rot = 0.1 * rnd(S, R, seed=91).double()
	w_q = W['q'].clone().reshape(H, D + R, 64)
	h = h.clone()
	h[:, 0] = 4.0                                                             # a constant input feature ...
	direction = torch.stack([W['uk'][n * D:(n + 1) * D] @ latent[key] for n in range(H)])
	w_q[:, :D, 0] = direction / direction.norm(dim=-1, keepdim=True) * 6      # ... that turns every query towards this key
	W = {**W, 'q': w_q.reshape(H * (D + R), 64).bfloat16().double()}
	from gptq_triton_b200.latent_attention import LatentAttention
	mix = LatentAttention(spec, *(W[k].to(dtype) for k in ('q', 'uk', 'uv', 'g', 'o')), None, None).cuda()      # reads the cache, writes none
	cache = torch.zeros((1, S + 5, spec.row), dtype=dtype, device='cuda')
	cache[0, :S, :C] = latent.to(dtype).cuda()
	cache[0, :S, C:C + R] = key_rot.to(dtype).cuda()
	stored = cache[0, :S].double().cpu()
	ref, _, _ = O.latent_attention(h.double(), W, mixer, 1e-5, torch.arange(S), stored[:, :C], stored[:, C:C + R])
	# scores reach 80: rounding queries and keys to bf16 alone moves them by up to 80 / 512, the output by 2.5 % (a lost or an
	# extra key moves it by all of it)
	tol = 2e-5 if dtype == F32 else 3.5e-2
	got = run_mixer(mix, cache, h, 0, tables, control)
	assert close(got[:, :64], ref, tol)
	for start, n in ((max(0, key - 3), 8), (key, 200), (min(key + 1, 600), 100)):          # portions that begin before, at and behind the key
		n = min(n, S - start)
		assert close(run_mixer(mix, cache, h[start:start + n], start, tables, control)[:, :64], ref[start:start + n], tol), start
	for p in sorted({max(0, key - 1), key, min(key + 1, S - 1), S - 1}):
		assert close(run_mixer(mix, cache, h[p:p + 1], p, tables, control, decode=True)[:, :64], ref[p:p + 1], tol), p


def test_prompt_kernel_rescales_when_later_keys_score_higher(control):
	"""Scores that grow along the sequence by far more than the kernel's rescale threshold, and ones that fall."""
	H, D, R, V, C, S = 2, 32, 16, 48, 64, 520
	for sign in (1.0, -1.0):
		spec, mix, mixer, W, h, tables = attention_case(B16, H, D, R, V, C, S, 0, seed=3)
		h = h.clone()
		h[:, 0] = 4.0
		axis = rnd(C, seed=4).double()
		axis /= axis.norm()
		latent = rnd(S, C, seed=5).double() * 0.3 + sign * (torch.arange(S).double()[:, None] / 40) * axis
		w_q = W['q'].clone().reshape(H, D + R, 64)
		d = torch.stack([W['uk'][n * D:(n + 1) * D] @ axis for n in range(H)])
		w_q[:, :D, 0] = 3 * d / d.norm(dim=-1, keepdim=True)
		W = {**W, 'q': w_q.reshape(H * (D + R), 64).bfloat16().double()}
		from gptq_triton_b200.latent_attention import LatentAttention
		mix = LatentAttention(spec, *(W[k].to(B16) for k in ('q', 'uk', 'uv', 'g', 'o')), None, None).cuda()
		cache = torch.zeros((1, S, spec.row), dtype=B16, device='cuda')
		cache[0, :, :C] = latent.to(B16).cuda()
		stored = cache[0].double().cpu()
		ref, _, _ = O.latent_attention(h.double(), W, mixer, 1e-5, torch.arange(S), stored[:, :C], stored[:, C:C + R])
		assert close(run_mixer(mix, cache, h, 0, tables, control)[:, :64], ref, 2e-2)
		for p in (40, 519):
			assert close(run_mixer(mix, cache, h[p:p + 1], p, tables, control, decode=True)[:, :64], ref[p:p + 1], 2e-2)


# ---- whole models ------------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize('dtype', [F32, B16])
@pytest.mark.parametrize('name', list(LM.CONFIGS))
def test_prompts_of_every_kind_of_length(name, dtype):
	"""Whole prompts from one token up, layer by layer; the same engine serves them in turn, longer and shorter ones."""
	n = 290
	ref, taps = LM.oracle_logits(name, n)
	eng = LM.engine(LM.CONFIGS[name], dtype, n)
	toks = LM.tokens(LM.CONFIGS[name], n)
	for t in (290, 1, 2, 3, 8, 9, 16, 17, 127, 128, 129, 256, 257):
		eng.reset()
		eng._taps = []
		got = eng.feed(toks[None, :t], list(range(t)))[0]
		assert LM.error(got, ref[:t]) <= LM.LIMIT[dtype], t
		if t > 1:          # (a single token runs as a captured step)
			for a, b in zip(eng._taps, taps):
				scale = float(b[:t].abs().max())
				assert float((a.double().cpu() - b[:t]).abs().max()) <= (1e-5 if dtype == F32 else 5e-2) * scale, t


@pytest.mark.parametrize('dtype', [F32, B16])
@pytest.mark.parametrize('name', list(LM.CONFIGS))
@pytest.mark.parametrize('cuts', ['ones', 'twos', 'mixed', 'borders', 'tail'])
def test_portions_give_the_whole_prompts_logits(name, dtype, cuts):
	n = 290
	ref, _ = LM.oracle_logits(name, n)
	sizes = {'ones': [1] * 290, 'twos': [2] * 145, 'mixed': [100, 7, 2, 1, 50, 9, 1, 1, 64, 3, 2, 40, 8, 2], 'borders': [31, 1, 1, 94, 1, 1, 126, 2, 1, 32], 'tail': [258] + [1] * 32}[cuts]
	eng = LM.engine(LM.CONFIGS[name], dtype, n)
	assert LM.error(LM.feed_all(eng, LM.tokens(LM.CONFIGS[name], n), sizes), ref) <= LM.LIMIT[dtype]


@pytest.mark.parametrize('dtype', [F32, B16])
def test_cache_rows_are_used_again(dtype):
	"""Requests of different lengths, one after the other on one engine: none sees what an earlier one left."""
	eng = LM.engine(LM.ODD, dtype, 200)
	for seed, cuts in ((0, [150, 1, 1, 30]), (1, [3, 1, 1]), (2, [1] * 5 + [60, 2]), (3, [200]), (4, [2])):
		toks = LM.tokens(LM.ODD, sum(cuts), seed)
		eng.reset()
		assert LM.error(LM.feed_all(eng, toks, cuts), O.forward(LM.ODD, LM.tensors(LM.ODD), toks)) <= LM.LIMIT[dtype], seed


@pytest.mark.parametrize('dtype', [F32, B16])
@pytest.mark.parametrize('batch', [2, 3, 9])
def test_sequences_of_a_batch_do_not_mix(dtype, batch):
	cfg = LM.ODD
	n = 60
	toks = torch.stack([LM.tokens(cfg, n, seed) for seed in range(batch)])
	eng = LM.engine(cfg, dtype, n, batch=batch)
	got, p = [], 0
	for c in (20, 3, 1, 1, 12, 2, 1, 20):
		got.append(eng.feed(toks[:, p:p + c], list(range(c))).clone())
		p += c
	got = torch.cat(got, dim=1)
	for b in range(batch):
		assert LM.error(got[b], O.forward(cfg, LM.tensors(cfg), toks[b])) <= LM.LIMIT[dtype], b


def greedy_reference(cfg, prompt, steps):
	toks, margins = prompt.tolist(), []
	W = LM.tensors(cfg)
	for _ in range(steps):
		top = O.forward(cfg, W, toks)[-1].topk(2)
		margins.append(float(top.values[0] - top.values[1]))
		toks.append(int(top.indices[0]))
	return toks[len(prompt):], margins


@pytest.mark.parametrize('dtype', [F32, B16])
@pytest.mark.parametrize('name', ['odd', 'partial'])
def test_greedy_generation(name, dtype):
	"""engine.generate against greedy decoding with the oracle; a prompt is used as far as the oracle's choice is clear."""
	cfg, steps = LM.CONFIGS[name], 24
	compared = 0
	for seed in range(3):
		prompt = LM.tokens(cfg, 5 + 9 * seed, seed)
		want, margins = greedy_reference(cfg, prompt, steps)
		clear = next((i for i, m in enumerate(margins) if m < (1e-3 if dtype == F32 else 0.3)), steps)
		for graph in (False, True):
			eng = LM.engine(cfg, dtype, len(prompt) + steps, use_graph=graph)
			got = eng.generate(prompt[None], steps)[0].tolist()
			assert got[:clear] == want[:clear]
		compared += clear
	assert compared >= 8


def test_long_decoding_crosses_every_tile_and_split():
	"""1200 decode steps with given tokens (the absorbed kernel's key ranges change with the length) against one prompt."""
	cfg, n = LM.PARTIAL, 1200
	toks = LM.tokens(cfg, n)
	ref = O.forward(cfg, LM.tensors(cfg), toks)
	eng = LM.engine(cfg, B16, n)
	got = LM.feed_all(eng, toks, [1] * n)
	assert LM.error(got, ref) <= LM.LIMIT[B16]
	with pytest.raises(RuntimeError, match='max_seq'):
		eng.feed(toks[None, :1])
	eng.reset()
	assert LM.error(eng.feed(toks[None], list(range(n)))[0], ref) <= LM.LIMIT[B16]


def test_graph_and_eager_steps_are_identical():
	outs = []
	for graph in (False, True):
		eng = LM.engine(LM.WIDE, B16, 64, use_graph=graph)
		toks = eng.generate(LM.tokens(LM.WIDE, 20)[None], 12)
		outs.append((toks.cpu(), eng.logits.clone().cpu(), eng.pos.cpu()))
	assert all(torch.equal(a, b) for a, b in zip(*outs))


def test_a_token_outside_the_vocabulary_is_reported():
	from gptq_triton_b200 import _lib
	eng = LM.engine(LM.PARTIAL, B16, 8, use_graph=False)
	eng.feed(torch.tensor([[3, LM.PARTIAL['vocab'], 1]]))
	assert _lib.kernel_status() == 4
	_lib.clear_kernel_status()


def write_checkpoint(path, cfg, seed=0):
	from safetensors.torch import save_file
	(path / 'config.json').write_text(json.dumps(cfg))
	save_file(LM.tensors(cfg, seed), str(path / 'model.safetensors'))


@pytest.mark.parametrize('dtype', ['bfloat16', 'float32'])
def test_replay_program(tmp_path, dtype):
	"""bin/trace_run as a user calls it: requests one after the other in portions and steps."""
	write_checkpoint(tmp_path, LM.ODD)
	(tmp_path / 'out').mkdir()
	toks = LM.tokens(LM.ODD, 40).tolist()
	steps = [{'step': 0, 'entries': [{'id': 'x', 'tokens': toks[:25], 'want': [0, 24]}], 'end': []},
			 {'step': 1, 'entries': [{'id': 'x', 'tokens': toks[25:26], 'want': []}], 'end': []},
			 {'step': 2, 'entries': [{'id': 'x', 'tokens': toks[26:27], 'want': [0]}], 'end': []},
			 {'step': 3, 'entries': [{'id': 'x', 'tokens': toks[27:30], 'want': [2, 1]}], 'end': ['x']},
			 {'step': 4, 'entries': [{'id': 'y', 'tokens': toks[30:31], 'want': [0]}], 'end': []},
			 {'step': 5, 'entries': [{'id': 'y', 'tokens': toks[31:40], 'want': [0, 8]}], 'end': ['y']}]
	r = subprocess.run([str(ROOT / 'bin' / 'trace_run'), '--model', str(tmp_path), '--dtype', dtype, '--out', str(tmp_path / 'out'), '--max-tokens', '30'],
					   input=''.join(json.dumps(s) + '\n' for s in steps), capture_output=True, text=True, timeout=300)
	assert r.returncode == 0, r.stderr
	assert [l for l in r.stdout.split('\n') if l.startswith('done')] == [f'done {i}' for i in range(6)]
	W = LM.tensors(LM.ODD)
	x, y = O.forward(LM.ODD, W, toks[:30]), O.forward(LM.ODD, W, toks[30:])
	want = {0: x[[0, 24]], 2: x[[26]], 3: x[[29, 28]], 4: y[[0]], 5: y[[1, 9]]}
	assert sorted(int(f[:-4]) for f in os.listdir(tmp_path / 'out')) == sorted(want)
	for step, ref in want.items():
		got = torch.frombuffer(bytearray((tmp_path / 'out' / f'{step}.f32').read_bytes()), dtype=F32).view(len(ref), -1)
		d = got.double() - ref
		assert float((d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt().max() / x.std()) <= LM.LIMIT[getattr(torch, dtype)], step


def test_command_line_generates(tmp_path):
	write_checkpoint(tmp_path, LM.PARTIAL)
	prompt = LM.tokens(LM.PARTIAL, 6)
	r = subprocess.run([sys.executable, '-m', 'gptq_triton_b200', 'generate', '--model', str(tmp_path), '--prompt-ids', ','.join(map(str, prompt.tolist())), '--steps', '5', '--dtype', 'float32'],
					   capture_output=True, text=True, timeout=300, cwd=ROOT)
	assert r.returncode == 0, r.stderr
	assert json.loads(r.stdout) == LM.engine(LM.PARTIAL, F32, 16).generate(prompt[None], 5)[0].tolist()


# ---- the same loop serves the quantised models --------------------------------------------------------------------------------

def test_llama_engine_takes_prompts_in_portions():
	import gptq_triton_b200 as G
	from gptq_triton_b200.llama import LlamaConfig
	cfg = LlamaConfig(hidden_size=512, intermediate_size=1408, num_hidden_layers=2, num_attention_heads=4, vocab_size=512, max_position_embeddings=128)
	model = G.synthetic_quantized_llama(cfg, groupsize=128, seed=3, device='cuda')
	eng = G.make_engine(model, batch=1, max_seq=96)
	assert isinstance(eng, G.DecodeEngine)
	toks = torch.randint(0, 512, (1, 80), generator=torch.Generator().manual_seed(2)).cuda()
	whole = eng.feed(toks, list(range(80)))[0].float()
	eng.reset()
	parts = LM.feed_all(eng, toks[0], [30, 1, 1, 17, 2, 29]).float()
	assert (parts - whole).abs().max() <= 2e-2 * whole.abs().max()


def test_mistakes_that_the_comparisons_must_see():
	"""Each mechanism changed in the oracle (never in a kernel) moves the logits far beyond the limits used above."""
	cfg, n = LM.ODD, 120
	W, toks = LM.tensors(cfg), LM.tokens(cfg, n)
	ref = O.forward(cfg, W, toks)

	def changed(edit_cfg=None, edit_w=None):
		c = json.loads(json.dumps(cfg))
		w = dict(W)
		if edit_cfg:
			edit_cfg(c)
		if edit_w:
			edit_w(w)
		return LM.error(O.forward(c, w, toks), ref)
	cases = {
		'kv_from': changed(lambda c: c['layers'][3]['mixer'].update(kv_from=1, scale=c['layers'][3]['mixer']['scale'] * 1.3)),
		'rotation base': changed(lambda c: [l['mixer']['rot'].update(base=l['mixer']['rot']['base'] * 1.5) for l in c['layers']]),
		'multiplier': changed(lambda c: c.update(residual_mult=0.9)),
		'gate': changed(edit_w=lambda w: w.update({'l0.mix.g': -w['l0.mix.g']})),
		'latent norm': changed(edit_w=lambda w: w.update({'l1.mix.dkv.norm': torch.ones_like(w['l1.mix.dkv.norm'])})),
		'layer scale': changed(edit_w=lambda w: w.update({'l2.ls2': torch.ones_like(w['l2.ls2'])})),
		'norm bias': changed(edit_w=lambda w: w.update({'l3.norm1.b': -w['l3.norm1.b']})),
	}
	assert all(v > 1.5 * LM.LIMIT[B16] for v in cases.values()), cases
