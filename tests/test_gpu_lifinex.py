"""Lifinex models on the GPU against the plain CPU oracle: every mechanism alone, prompts, portions, decode steps, state and cache
rows that are used again, single keys and single inputs that stand out at every kind of border, greedy generation through the
engine, command line and replay."""
import json
import os
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import lifinex_models as LM
from oracle import lifinex_oracle as O

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
F32, B16 = torch.float32, torch.bfloat16
REL = {F32: 3e-6, B16: 7e-3}          # of the largest result: fp32 sums; one bf16 rounding of operands or result


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


def err(got, want):
	"""Largest error in units of the largest wanted value."""
	want = want.double()
	return float((got.double().cpu() - want).abs().max() / want.abs().max())


def pad_cols(t):
	from gptq_triton_b200.dense import pad_to, padded
	return pad_to(t, t.shape[0], padded(t.shape[1])).cuda()


def rows_of(stream, dtype, control, final=None):
	"""(new residual, prepared rows) by the row kernel, and the prepared rows again as a projection with the unit matrix sees them."""
	from gptq_triton_b200 import _dense
	from gptq_triton_b200.dense import epilogue, prepare_rows, project_stream
	parts = final is not None and final.parts > 1
	h, x = prepare_rows(stream, control, dtype, not parts, final)
	eye = torch.eye(stream.ld, dtype=dtype, device='cuda')
	out = torch.empty((stream.rows, stream.ld), device='cuda')
	project_stream(stream, eye, epilogue(_dense.EPI_F32, out), control, keep=False, final=final)
	assert torch.equal(out, h.float())
	return x, h


# ---- the mechanisms alone --------------------------------------------------------------------------------------------------

@pytest.mark.parametrize('dtype', [F32, B16])
@pytest.mark.parametrize('M', [1, 2, 7])
@pytest.mark.parametrize('width', [50, 4100])          # rows shorter and longer than the registers of a CTA hold
def test_rows(control, dtype, M, width):
	"""Embedding with positions, plain residual with a shift, RMS-normed residual, RMS norm with an offset weight."""
	from gptq_triton_b200.dense import RMSNorm, Stream, padded
	eps, V, P = 1e-4, 37, 19
	table, where = rnd(V, width, seed=1, dtype=B16), rnd(P, width, seed=2, dtype=B16)
	tok, pos = torch.arange(M) * 11 % V, (torch.arange(M) * 7 + 3) % P
	s = Stream(width, padded(width), eps, table=pad_cols(table.to(dtype)), token=tok.cuda(), pos_table=pad_cols(where.to(dtype)), pos=pos.int().cuda())
	ref = table[tok].double() + where[pos].double()
	x, h = rows_of(s, dtype, control)
	assert err(x[:, :width], ref) <= 1e-7 and err(h[:, :width], ref) <= REL[dtype]
	assert torch.equal(s.take(torch.tensor([M - 1], device='cuda')).pos.cpu(), pos[-1:].int())
	y, shift, w = 3 * rnd(M, width, seed=3) + 1, rnd(1, width, seed=4), 0.3 * rnd(width, seed=5)
	norm = RMSNorm(w, offset=1.0).cuda()
	for stream, want in ((s.then(x, pad_cols(y), shift=pad_cols(shift)), ref + y + shift),
						 (s.then(x, pad_cols(y), 2, pad_cols(w[None])), ref + O.rms_norm(y.double(), w.double(), eps)),
						 (s.then(x, pad_cols(y)), ref + y)):
		new, h = rows_of(stream, dtype, control, norm)
		assert err(new[:, :width], want) <= 1e-6 and err(h[:, :width], O.rms_norm_centred(want.double(), w.double(), eps)) <= REL[dtype]
		assert new.shape[1] == width or float(new[:, width:].abs().max()) == 0 and float(h[:, width:].abs().max()) == 0


@pytest.mark.parametrize('dtype', [F32, B16])
@pytest.mark.parametrize('M', [1, 2, 5])
@pytest.mark.parametrize('n,parts', [(96, 1), (96, 2), (35, 7), (33, 11), (60, 20), (4160, 8), (90, 5), (512, 256), (6144, 3)])
def test_norm_of_equal_parts(control, dtype, M, n, parts):
	"""Parts that end inside a 16-byte unit, parts shorter than one, more and fewer parts than warps; their sizes differ a lot."""
	from gptq_triton_b200.dense import RMSNorm, Stream, padded
	x, w = rnd(M, n, seed=1), 1 + 0.2 * rnd(n, seed=2)
	x = x * torch.exp(2 * rnd(M, parts, seed=3)).repeat_interleave(n // parts, 1)
	got = rows_of(Stream(n, padded(n), 1e-5, x=pad_cols(x)), dtype, control, RMSNorm(w, parts=parts).cuda())[1]
	assert err(got[:, :n], O.rms_norm_parts(x.double(), w.double(), parts, 1e-5)) <= REL[dtype]


@pytest.mark.parametrize('dtype', [F32, B16])
@pytest.mark.parametrize('M,width', [(1, 90), (2, 90), (3, 90), (8, 90), (40, 90), (200, 90), (1, 4200), (2, 6200), (5, 4200), (140, 4200)])
def test_gated_mlp_and_token_side(control, dtype, M, width):
	"""Also rows so long that the narrow projections share them over several CTAs."""
	from gptq_triton_b200.dense import DenseMLP, RMSNorm, Stream, TokenSide, padded, pad_to
	ff, dim, V, L, eps = 77, 21, 31, 3, 1e-4
	g, u, d = (rnd(*s, seed=i, dtype=B16) * 2 * s[1] ** -0.5 for i, s in enumerate([(ff, width), (ff, width), (width, ff)]))
	x, y = rnd(M, width, seed=8), rnd(M, width, seed=9)
	w = 0.2 * rnd(width, seed=5)
	stream = Stream(width, padded(width), eps).then(pad_cols(x), pad_cols(y))
	mlp = DenseMLP(g.to(dtype), u.to(dtype), d.to(dtype), act='gelu_tanh').cuda()
	got_x, got_y = mlp(stream, control, norm=RMSNorm(w, offset=1.0).cuda())
	ref = (x + y).double()
	assert err(got_x[:, :width], ref) <= 1e-6
	assert err(got_y[:, :width], O.dense_ff(O.rms_norm_centred(ref, w.double(), eps), g.double(), u.double(), d.double())) <= REL[dtype] * 2
	# the side input of the last of three layers, on the stream itself
	sg, sp, sn = rnd(dim, width, seed=11, dtype=B16) * width ** -0.5 * 3, rnd(width, dim, seed=12, dtype=B16), 1 + 0.2 * rnd(width, seed=13)
	table, tok = rnd(V, L * dim, seed=14, dtype=B16), torch.arange(M) * 5 % V
	packed = pad_to(table.view(V, L, dim), V, L, padded(dim)).reshape(V, -1).to(dtype).contiguous().cuda()
	side = TokenSide(sg.to(dtype), sp.to(dtype), sn, column=2 * padded(dim)).cuda()
	out = side(stream, packed, tok.cuda(), control)
	got = rows_of(out, F32, control)[0][:, :width]
	want = ref + O.token_side(ref, table[tok][:, 2 * dim:].double(), sg.double(), sp.double(), sn.double(), eps)
	assert err(got, want) <= REL[dtype] * 2


def test_gelu_over_its_whole_range(control):
	"""The gate of the MLP as a function, from values where it vanishes to values where it is the identity."""
	from gptq_triton_b200 import _dense
	from gptq_triton_b200.dense import matmul, epilogue
	z = torch.linspace(-30, 30, 64 * 16).view(64, 16)
	w = torch.zeros((32, 16))
	for i in range(16):          # gate rows: unit matrix in groups of eight; up rows read a constant one
		w[i // 8 * 16 + i % 8, i] = 1.0
		w[i // 8 * 16 + 8 + i % 8, i] = 1.0
	out = torch.empty((64, 16), device='cuda')
	e = epilogue(_dense.EPI_GATED, out)
	e.act = _dense.ACT_CODE['gelu_tanh']
	matmul(z.cuda(), w.cuda(), e, control)
	want = O.gelu_tanh(z.double()) * z.double()
	assert float(((out.double().cpu() - want).abs() / (want.abs() + 1e-6)).max()) <= 2e-6


def gqa_case(H, G, D, V, t, maps=2, scale=0.7, cap=6.0, seed=0, width=64):
	from gptq_triton_b200.gqa_attention import GroupedAttentionSpec
	spec = GroupedAttentionSpec(H, G, D, V, scale, cap, maps, 0.35)
	shapes = {'q': (H * maps * D, width), 'k': (G * maps * D, width), 'v': (G * V, width), 'o': (width, H * V), 'q.norm': (D,), 'k.norm': (D,),
			  'lq1': (D,), 'lk1': (D,), 'lq2': (D,), 'lk2': (D,)}
	W = {}
	for i, (k, s) in enumerate(shapes.items()):
		r = rnd(*s, seed=seed + i)
		W[k] = (r * s[1] ** -0.5 if len(s) == 2 else 1 + 0.3 * r if 'norm' in k else 0.3 * r).bfloat16()
	mixer = {'heads': H, 'kv_heads': G, 'dim': D, 'vdim': V, 'scale': scale, 'softcap': cap, 'diff': 0.35}
	return spec, W, mixer, rnd(t, width, seed=seed + 50, dtype=B16)


def build_gqa(spec, W, dtype):
	from gptq_triton_b200.gqa_attention import GroupedAttention, diff_lambda
	lam = diff_lambda(W['lq1'], W['lk1'], W['lq2'], W['lk2'], spec.diff)
	return GroupedAttention(spec, *(W[k].to(dtype) for k in 'qkvo'), W['q.norm'], W['k.norm'], lam).cuda()


def new_cache(spec, max_seq, dtype, batch=1):
	from gptq_triton_b200.cache import StaticCache
	return StaticCache([spec.cache_layout(max_seq) if hasattr(spec, 'softcap') else spec.cache_layout()], batch, dtype, 'cuda')[0]


def run_mixer(mix, cache, h, start, control, eps=1e-5, decode=False):
	from gptq_triton_b200.dense import Stream, padded
	stream = Stream(h.shape[1], padded(h.shape[1]), eps, x=pad_cols(h.float()))
	pos = torch.arange(start, start + h.shape[0], dtype=torch.int32, device='cuda')
	return mix(stream, cache, pos, h.shape[0], None if decode else start, control)[1][:, :h.shape[1]]


def double(W):
	return {k: v.double() for k, v in W.items()}


GQA_SHAPES = [(3, 1, 20, 24), (6, 2, 40, 40), (24, 2, 16, 80), (4, 4, 64, 128), (17, 1, 130, 144), (2, 1, 256, 256), (1, 1, 16, 520 - 8), (8, 2, 64, 64), (2, 2, 300, 16)]


@pytest.mark.parametrize('dtype', [F32, B16])
@pytest.mark.parametrize('maps', [1, 2])
@pytest.mark.parametrize('H,G,D,V', GQA_SHAPES)
def test_attention_prompt_portions_and_steps(control, dtype, maps, H, G, D, V):
	t = 300
	spec, W, mixer, h = gqa_case(H, G, D, V, t, maps, scale=min(0.7, 3 / D ** 0.5), cap=6.0 if maps == 2 else None)
	ref = (O.differential_attention if maps == 2 else O.plain_attention)(h.double(), double(W), mixer, 1e-5)
	mix = build_gqa(spec, W, dtype)
	for cuts in ([300], [1, 2, 9, 100, 128, 52, 8]):
		cache = new_cache(spec, t + 5, dtype)
		out, p = [], 0
		for n in cuts:
			out.append(run_mixer(mix, cache, h[p:p + n], p, control, decode=n == 1))
			p += n
		# (the normed difference of two maps magnifies the rounding of each)
		assert err(torch.cat(out), ref) <= (1e-5 if dtype == F32 else 2.5e-2), cuts
	q, k, v = O.normed_qkv(h.double(), double(W), mixer, 1e-5, maps)
	assert err(cache['k'][0, :t].view(t, G, maps, -1)[..., :D], k) <= (3e-6 if dtype == F32 else 6e-3)
	assert err(cache['v'][0, :t].view(t, G, -1)[..., :V], v) <= (3e-6 if dtype == F32 else 6e-3)
	assert float(cache['k'][0, t:].abs().max()) == 0 and float(cache['v'][0, t:].abs().max()) == 0


@pytest.mark.parametrize('dtype', [F32, B16])
@pytest.mark.parametrize('which', [0, 1])
@pytest.mark.parametrize('key', [0, 1, 31, 32, 63, 64, 127, 128, 129, 255, 256, 511, 639, 640, 641, 700])
def test_one_key_that_stands_out(control, dtype, which, key):
	"""In one map, one cached key scores far above all others for every query that may see it: that map's output is the key's value
	from there on and has nothing of it before, in prompts and steps, wherever the key's tile lies."""
	H, G, D, V, S, width = 4, 2, 128, 48, 701, 64
	spec, W, mixer, h = gqa_case(H, G, D, V, S, cap=40.0, scale=0.3, seed=7)
	h = h.clone()
	h[:, 0] = 0.0
	h[:, 1] = 3.0                                     # a constant feature turns the queries of this map ...
	h[key, 0] = 30.0                                  # ... and a feature that only this token has turns its key the same way
	wq, wk = W['q'].clone().view(H, 2, D, width), W['k'].clone().view(G, 2, D, width)
	axis = rnd(D, seed=90)
	wq[:, which, :, 1] += 3 * axis.bfloat16()
	wk[:, which, :, 0] = (3 * axis).bfloat16()
	W = {**W, 'q': wq.view(-1, width), 'k': wk.view(-1, width)}
	ref = O.differential_attention(h.double(), double(W), mixer, 1e-5)
	a = O.attention_maps(*O.normed_qkv(h.double(), double(W), mixer, 1e-5), mixer['scale'], mixer['softcap'])[:, :, which]
	v = O.normed_qkv(h.double(), double(W), mixer, 1e-5)[2].repeat_interleave(H // G, 1)
	assert float((a[key:] - v[key]).abs().max()) < 0.05 * float(v[key].abs().max())          # the key does stand out
	mix = build_gqa(spec, W, dtype)
	tol = 2e-5 if dtype == F32 else 4e-2
	cache = new_cache(spec, S + 3, dtype)
	assert err(run_mixer(mix, cache, h, 0, control), ref) <= tol
	for start, n in ((max(0, key - 3), 8), (key, 200), (min(key + 1, 600), 100)):          # portions that begin before, at and behind the key
		n = min(n, S - start)
		assert err(run_mixer(mix, cache, h[start:start + n], start, control), ref[start:start + n]) <= tol, start
	for p in sorted({max(0, key - 1), key, min(key + 1, S - 1), S - 1}):
		assert err(run_mixer(mix, cache, h[p:p + 1], p, control, decode=True), ref[p:p + 1]) <= tol, p


@pytest.mark.parametrize('dtype', [F32, B16])
def test_scores_beyond_the_cap_and_growing_scores(control, dtype):
	"""Raw scores from far below to far above the cap; and scores that grow or fall along the sequence by much more than a softmax
	that keeps an old reference point would bear."""
	H, G, D, V, S, width = 2, 1, 32, 48, 520, 64
	for cap, scale, grow in ((2.0, 3.0, 0.0), (0.5, 30.0, 0.0), (300.0, 8.0, 1.0), (300.0, 8.0, -1.0), (1e4, 0.05, 0.0)):
		spec, W, mixer, h = gqa_case(H, G, D, V, S, cap=cap, scale=scale, seed=3)
		if grow:
			h = h.clone()
			h[:, 0] = 2.0
			h[:, 1] = (grow * torch.linspace(-6, 6, S)).bfloat16()
			axis = rnd(D, seed=4).bfloat16()
			for n in ('q', 'k'):
				w = W[n].clone().view(-1, 2, D, width)
				w[..., :2] = 0
				w[..., 0 if n == 'q' else 1] = axis
				W = {**W, n: w.view(-1, width)}
		ref = O.differential_attention(h.double(), double(W), mixer, 1e-5)
		mix = build_gqa(spec, W, dtype)
		cache = new_cache(spec, S, dtype)
		# (with scores of hundreds the rounding of queries and keys to bf16 alone moves a map by several percent)
		tol = 1e-4 if dtype == F32 else 0.12 if scale * cap > 500 else 4e-2
		assert err(run_mixer(mix, cache, h, 0, control), ref) <= tol, (cap, grow)
		for p in (40, 519):
			assert err(run_mixer(mix, cache, h[p:p + 1], p, control, decode=True), ref[p:p + 1]) <= tol, (cap, grow, p)


def ssm_case(H, P, N, G, taps, parts, t, seed=0, width=64):
	from gptq_triton_b200.ssm import StateSpaceSpec
	spec = StateSpaceSpec(H, P, N, G, taps, parts)
	W = {'in': rnd(spec.inner + spec.channels + H, width, seed=seed) * width ** -0.5, 'conv': rnd(spec.channels, taps, seed=seed + 1) * taps ** -0.5,
		 'conv.b': 0.3 * rnd(spec.channels, seed=seed + 2), 'dt_bias': rnd(H, seed=seed + 3) - 2.0, 'A_log': rnd(H, seed=seed + 4) - 1.0, 'D': 1 + 0.3 * rnd(H, seed=seed + 5),
		 'norm': 1 + 0.2 * rnd(spec.inner, seed=seed + 6), 'o': rnd(width, spec.inner, seed=seed + 7) * spec.inner ** -0.5}
	mixer = {'heads': H, 'vdim': P, 'state': N, 'groups': G, 'norm_groups': parts}
	return spec, {k: v.bfloat16() for k, v in W.items()}, mixer, rnd(t, width, seed=seed + 50, dtype=B16)


def build_ssm(spec, W, dtype):
	from gptq_triton_b200.ssm import StateSpaceMixer
	return StateSpaceMixer(spec, W['in'].to(dtype), *(W[k] for k in ('conv', 'conv.b', 'dt_bias', 'A_log', 'D', 'norm')), W['o'].to(dtype)).cuda()


SSM_SHAPES = [(2, 16, 16, 1, 1, 1), (6, 20, 24, 3, 4, 5), (5, 7, 40, 1, 2, 7), (4, 64, 128, 2, 4, 4), (3, 33, 200, 3, 3, 1), (6, 48, 32, 3, 3, 4), (2, 80, 256, 1, 7, 2), (1, 5, 3, 1, 16, 1),
			  (4, 128, 64, 4, 4, 1), (16, 32, 64, 2, 4, 16)]


@pytest.mark.parametrize('dtype', [F32, B16])
@pytest.mark.parametrize('H,P,N,G,taps,parts', SSM_SHAPES)
def test_state_space_prompt_portions_and_steps(control, dtype, H, P, N, G, taps, parts):
	t = 333
	spec, W, mixer, h = ssm_case(H, P, N, G, taps, parts, t)
	ref = O.mamba2(h.double(), double(W), mixer, 1e-5)
	mix = build_ssm(spec, W, dtype)
	for cuts in ([333], [1] * 20 + [2, 3, 9, 64, 1, 65, 127, 2, 1, 1] + [38], [200, 1, 132], [2] * 166 + [1]):
		cache = new_cache(spec, t, dtype)
		for c in cache.values():
			c.fill_(float('nan'))          # what an earlier request has left does not count at position 0
		out, p = [], 0
		for n in cuts:
			out.append(run_mixer(mix, cache, h[p:p + n], p, control, decode=n == 1))
			p += n
		assert err(torch.cat(out), ref) <= (1e-5 if dtype == F32 else 3e-2), cuts


@pytest.mark.parametrize('dtype', [F32, B16])
@pytest.mark.parametrize('at', [0, 1, 15, 16, 31, 32, 63, 64, 65, 127, 128, 200])
def test_one_input_that_the_state_must_keep(control, dtype, at):
	"""Every token but one writes almost nothing to a state that hardly decays: what later tokens read is that one input, carried
	through prompts, portions and steps that begin and end around it."""
	H, P, N, G, taps, t, width = 4, 24, 32, 2, 4, 400, 64
	spec, W, mixer, h = ssm_case(H, P, N, G, taps, 2, t, seed=20)
	h = h.clone()
	h[:, 0] = 0.0
	h[at, 0] = 12.0
	w_in = W['in'].clone()
	w_in[-H:] = 0
	w_in[-H:, 0] = 1.0                                             # dt is large at this token only
	bias = W['conv.b'].clone()
	bias[H * P:] = 1.5                                             # B and C point the same way: their product does not vanish by chance
	W = {**W, 'in': w_in, 'conv.b': bias, 'dt_bias': torch.full((H,), -9.0).bfloat16(), 'A_log': torch.full((H,), -9.0).bfloat16(), 'D': torch.zeros(H).bfloat16()}
	ref = O.mamba2(h.double(), double(W), mixer, 1e-5)
	quiet = O.mamba2(torch.cat([h[:at], h[at:at + 1] * 0, h[at + 1:]]).double(), double(W), mixer, 1e-5)
	assert at > 390 or float((ref - quiet)[-1].abs().max()) > 0.5 * float(ref[-1].abs().max())
	mix = build_ssm(spec, W, dtype)
	for cuts in ([400], [at, 2, 130, 1, 1] if at > 1 else [2, 130, 1, 1], [at + 1, 1, 1, 3, 64] if at > 0 else [1, 1, 1, 3, 64]):
		cuts = cuts + [t - sum(cuts)] if sum(cuts) < t else cuts
		cache = new_cache(spec, t, dtype)
		out, p = [], 0
		for n in cuts:
			out.append(run_mixer(mix, cache, h[p:p + n], p, control, decode=n == 1))
			p += n
		assert err(torch.cat(out), ref) <= (2e-5 if dtype == F32 else 3e-2), cuts


@pytest.mark.parametrize('dtype', [F32, B16])
def test_states_that_forget_at_once_and_never(control, dtype):
	"""Decays from exp(-1e-5) to exp(-1e3) per token: products of decays must neither overflow nor lose the recent tokens."""
	H, P, N, t = 6, 16, 48, 260
	spec, W, mixer, h = ssm_case(H, P, N, 1, 4, 3, t, seed=40)
	W = {**W, 'A_log': torch.tensor([-10.0, -4.0, 0.0, 3.0, 6.0, 7.0]).bfloat16(), 'dt_bias': torch.tensor([1.0, 0.0, -1.0, 2.0, -3.0, 3.0]).bfloat16()}
	ref = O.mamba2(h.double(), double(W), mixer, 1e-5)
	mix = build_ssm(spec, W, dtype)
	for cuts in ([260], [100, 1, 2, 157]):
		cache = new_cache(spec, t, dtype)
		out, p = [], 0
		for n in cuts:
			out.append(run_mixer(mix, cache, h[p:p + n], p, control, decode=n == 1))
			p += n
		assert err(torch.cat(out), ref) <= (2e-5 if dtype == F32 else 4e-2), cuts


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
		assert not LM.wrong(got, ref[:t], dtype), t
		if t > 1:          # (a single token runs as a captured step)
			assert len(eng._taps) == len(taps)
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
	assert not LM.wrong(LM.feed_all(eng, LM.tokens(LM.CONFIGS[name], n), sizes), ref, dtype)


@pytest.mark.parametrize('dtype', [F32, B16])
@pytest.mark.parametrize('name', ['odd', 'looped'])
def test_cache_and_state_are_used_again(name, dtype):
	"""Requests of different lengths, one after the other on one engine: none sees what an earlier one left."""
	cfg = LM.CONFIGS[name]
	eng = LM.engine(cfg, dtype, 200)
	for seed, cuts in ((0, [150, 1, 1, 30]), (1, [3, 1, 1]), (2, [1] * 5 + [60, 2]), (3, [200]), (4, [2]), (5, [1, 1])):
		toks = LM.tokens(cfg, sum(cuts), seed)
		eng.reset()
		assert not LM.wrong(LM.feed_all(eng, toks, cuts), O.forward(cfg, LM.tensors(cfg), toks), dtype), seed


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
		assert not LM.wrong(got[b], O.forward(cfg, LM.tensors(cfg), toks[b]), dtype), b


@pytest.mark.parametrize('dtype', [F32, B16])
def test_long_portions_are_cut(dtype):
	"""A prompt longer than a portion may be: the state and the cache carry over."""
	cfg = LM.LOOPED
	n = 150
	eng = LM.engine(cfg, dtype, n)
	eng.max_portion = 64
	assert not LM.wrong(eng.feed(LM.tokens(cfg, n)[None], list(range(n)))[0], LM.oracle_logits('looped', 290)[0][:n], dtype)


def greedy_reference(cfg, prompt, steps):
	toks, margins = prompt.tolist(), []
	W = LM.tensors(cfg)
	for _ in range(steps):
		top = O.forward(cfg, W, toks)[-1].topk(2)
		margins.append(float(top.values[0] - top.values[1]))
		toks.append(int(top.indices[0]))
	return toks[len(prompt):], margins


@pytest.mark.parametrize('dtype', [F32, B16])
@pytest.mark.parametrize('name', ['odd', 'plain'])
def test_greedy_generation(name, dtype):
	"""engine.generate against greedy decoding with the oracle; a prompt is used as far as the oracle's choice is clear."""
	cfg, steps = LM.CONFIGS[name], 10
	compared = 0
	for seed in range(6):
		prompt = LM.tokens(cfg, 1 + 7 * seed, seed)
		want, margins = greedy_reference(cfg, prompt, steps)
		clear = next((i for i, m in enumerate(margins) if m < (1e-3 if dtype == F32 else 0.12)), steps)
		for graph in (False, True):
			eng = LM.engine(cfg, dtype, len(prompt) + steps, use_graph=graph)
			got = eng.generate(prompt[None], steps)[0].tolist()
			assert got[:clear] == want[:clear]
		compared += clear
	assert compared >= 8


def test_long_decoding():
	"""1200 decode steps with given tokens against one prompt; the sequence ends with the table of positions."""
	cfg, n = {**LM.LOOPED, 'max_positions': 1200}, 1200
	toks = LM.tokens(cfg, n)
	ref = O.forward(cfg, LM.tensors(cfg), toks)
	eng = LM.engine(cfg, B16, n + 50)
	assert eng.max_seq == n
	assert not LM.wrong(LM.feed_all(eng, toks, [1] * n), ref, B16)
	with pytest.raises(RuntimeError, match='max_seq'):
		eng.feed(toks[None, :1])
	eng.reset()
	assert not LM.wrong(eng.feed(toks[None], list(range(n)))[0], ref, B16)


def test_graph_and_eager_steps_are_identical():
	"""Trial runs of the capture leave the carried state as it was."""
	outs = []
	for graph in (False, True):
		eng = LM.engine(LM.WIDE, B16, 64, use_graph=graph)
		toks = eng.generate(LM.tokens(LM.WIDE, 20)[None], 12)
		outs.append((toks.cpu(), eng.logits.clone().cpu(), eng.pos.cpu(), *(t.cpu() for t in eng.cache.carried)))
	assert all(torch.equal(a, b) for a, b in zip(*outs))


def test_a_token_outside_the_vocabulary_is_reported():
	from gptq_triton_b200 import _lib
	eng = LM.engine(LM.LOOPED, B16, 8, use_graph=False)
	eng.feed(torch.tensor([[3, LM.LOOPED['vocab'], 1]]))
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
		assert float((d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt().max() / x.std()) <= LM.LIMIT[getattr(torch, dtype)][0], step


def test_command_line_generates(tmp_path):
	write_checkpoint(tmp_path, LM.PLAIN)
	prompt = LM.tokens(LM.PLAIN, 6)
	r = subprocess.run([sys.executable, '-m', 'gptq_triton_b200', 'generate', '--model', str(tmp_path), '--prompt-ids', ','.join(map(str, prompt.tolist())), '--steps', '5', '--dtype', 'float32'],
					   capture_output=True, text=True, timeout=300, cwd=ROOT)
	assert r.returncode == 0, r.stderr
	assert json.loads(r.stdout) == LM.engine(LM.PLAIN, F32, 16).generate(prompt[None], 5)[0].tolist()
