"""Small random Lifinex models for the tests: configurations, checkpoint tensors, engines, comparison with the oracle."""
import torch

from gptq_triton_b200.lifinex import LifinexConfig, LifinexEngine, LifinexForCausalLM
from latent_models import error, feed_all, tokens          # noqa: F401
from oracle import lifinex_oracle as O

# error of the logits (mean taken off, rms over the vocabulary, relative to the logits' spread) that rounding causes: (largest of any
# position, mean).  Perturbing the weights by a relative e moves the logits of these models by 2 to 7 e at most positions and by up to
# 90 e at single ones (where the difference of two maps, or a part of a gated output, is small before it is normed); the
# mistakes of planted_mistakes() move some position by more than 0.4.
LIMIT = {torch.float32: (6e-5, 5e-6), torch.bfloat16: (0.2, 2.5e-2)}


def wrong(got, ref, dtype):
	"""None, or what exceeds the limits."""
	d = got.double().cpu() - ref
	d = (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / ref.std()
	worst, mean = float(d.max()), float(d.mean())
	return None if worst <= LIMIT[dtype][0] and mean <= LIMIT[dtype][1] else f'largest error {worst:.2e} at {int(d.argmax())}, mean {mean:.2e}'


def attention(heads, kv_heads, dim, vdim, ff, diff=0.4, scale=None, softcap=20.0):
	mixer = {'heads': heads, 'kv_heads': kv_heads, 'dim': dim, 'vdim': vdim, 'diff': diff, 'scale': scale if scale is not None else dim ** -0.5, 'softcap': softcap}
	return {'type': 'attention', 'mixer': mixer, 'mlp': None if ff is None else {'kind': 'dense', 'ff': ff}}


def mamba2(heads, vdim, state, groups, conv, norm_groups, ff):
	mixer = {'heads': heads, 'vdim': vdim, 'state': state, 'groups': groups, 'conv': conv, 'norm_groups': norm_groups}
	return {'type': 'mamba2', 'mixer': mixer, 'mlp': None if ff is None else {'kind': 'dense', 'ff': ff}}


def config(layers, loop=None, side=None, width=72, vocab=101, eps=1e-5, max_positions=1300):
	out = {'architecture': 'Lifinex', 'layers': layers, 'width': width, 'vocab': vocab, 'norm': {'eps': eps}, 'max_positions': max_positions}
	if loop is not None:
		out['loop'] = dict(zip(('start', 'stop', 'times'), loop))
	if side is not None:
		out['token_side'] = {'dim': side}
	return out


# every size its own, none a multiple of 16; both kinds of layer inside the loop and outside, layers without feed-forward
ODD = config([attention(6, 2, 20, 24, 56, diff=0.55, scale=0.5, softcap=7.0), mamba2(6, 20, 24, 3, 4, 5, 33), attention(3, 3, 9, 27, None, scale=0.8, softcap=3.0),
			  mamba2(7, 18, 40, 1, 2, 7, None), attention(4, 1, 34, 40, 90, diff=0.2)], loop=(1, 4, 2), side=22, width=88)
# aligned sizes, several row and column tiles of every kernel; the loop begins with the first layer and has a single layer
WIDE = config([mamba2(8, 64, 128, 2, 4, 8, 336), attention(24, 2, 64, 128, 208), mamba2(4, 48, 144, 4, 3, 1, None), attention(8, 8, 80, 176, 320, softcap=50.0)],
			  loop=(0, 1, 3), side=48, width=320, vocab=515, max_positions=600)
# neither loop nor side input; a single tap; the whole stack runs once
PLAIN = config([mamba2(2, 16, 16, 2, 1, 2, 48), attention(2, 1, 16, 16, None, diff=0.7)], width=48, vocab=64, eps=1e-3)
# all layers inside the loop, the attention comes last
LOOPED = config([mamba2(3, 30, 50, 1, 5, 3, 40), attention(5, 5, 18, 33, 44)], loop=(0, 2, 3), side=16, width=60, vocab=77)
CONFIGS = {'odd': ODD, 'wide': WIDE, 'plain': PLAIN, 'looped': LOOPED}


def tensors(cfg, seed=0):
	gen = torch.Generator().manual_seed(seed)
	out = {}
	for name, shape in LifinexConfig.from_dict(cfg).tensor_shapes().items():
		t = torch.randn(shape, generator=gen)
		short = name.split('.', 1)[-1]
		if short == 'mix.dt_bias':
			t = t - 2.0
		elif short == 'mix.A_log':
			t = t - 1.0                     # states that remember for a few and for hundreds of tokens
		elif short in ('mix.q.norm', 'mix.k.norm'):
			t = 1.5 + 0.3 * t
		elif short in ('mix.norm', 'side.norm', 'mix.D'):
			t = 0.7 + 0.2 * t
		elif short in ('norm1', 'norm2', 'mix.conv.b') or name == 'final.norm':
			t = 0.2 * t
		elif short in ('mix.lq1', 'mix.lk1', 'mix.lq2', 'mix.lk2'):
			t = 0.2 * t
		elif name == 'loop.step':
			t = 0.5 * t
		elif name not in ('embed', 'pos', 'side.embed'):
			t = t * shape[1] ** -0.5
		out[name] = t.bfloat16()
	return out


def engine(cfg, dtype, max_seq, batch=1, seed=0, **kw):
	return LifinexEngine(LifinexForCausalLM(LifinexConfig.from_dict(cfg), tensors(cfg, seed), dtype, 'cuda'), batch, max_seq, **kw)


_oracle = {}


def oracle_logits(name, n, seed=0):
	"""Logits and per-layer residual streams of CONFIGS[name] (weights and tokens of `seed`), computed once."""
	key = (name, n, seed)
	if key not in _oracle:
		taps = []
		_oracle[key] = (O.forward(CONFIGS[name], tensors(CONFIGS[name], seed), tokens(CONFIGS[name], n, seed), collect=taps), taps)
	return _oracle[key]


def planted_mistakes():
	"""name -> error of the logits when one mechanism is changed in the oracle (never in a kernel)."""
	import json
	cfg, n = ODD, 120
	W, toks = tensors(cfg), tokens(cfg, n)
	ref = O.forward(cfg, W, toks)

	def changed(edit_cfg=None, edit_w=None):
		c, w = json.loads(json.dumps(cfg)), dict(W)
		if edit_cfg:
			edit_cfg(c)
		if edit_w:
			edit_w(w)
		return error(O.forward(c, w, toks), ref)
	att, ssm = [0, 2, 4], [1, 3]
	mixers = lambda c, idx: [c['layers'][i]['mixer'] for i in idx]
	w_edit = lambda names, f: lambda w: w.update({n: f(w[n]) for n in names})
	return {
		'soft cap': changed(lambda c: [m.update(softcap=1e6) for m in mixers(c, att)]),
		'constant of lambda and output factor': changed(lambda c: [m.update(diff=m['diff'] + 0.1) for m in mixers(c, att)]),
		'second map': changed(edit_w=w_edit([f'l{i}.mix.lq2' for i in att], lambda t: 0 * t - 3)),
		'query norm': changed(edit_w=w_edit([f'l{i}.mix.q.norm' for i in att], torch.ones_like)),
		'norm parts': changed(lambda c: [m.update(norm_groups=1) for m in mixers(c, ssm)]),
		'decay': changed(edit_w=w_edit([f'l{i}.mix.A_log' for i in ssm], lambda t: t + 1)),
		'convolution bias': changed(edit_w=w_edit([f'l{i}.mix.conv.b' for i in ssm], lambda t: -t)),
		'oldest tap': changed(edit_w=w_edit([f'l{i}.mix.conv' for i in ssm], lambda t: torch.cat([0 * t[:, :1], t[:, 1:]], 1))),
		'skip': changed(edit_w=w_edit([f'l{i}.mix.D' for i in ssm], lambda t: 0 * t)),
		'one pass less': changed(lambda c: c['loop'].update(times=1)),
		'vector of the pass': changed(edit_w=w_edit(['loop.step'], lambda t: t.flip(0))),
		'embedding in the pass entry': changed(edit_w=w_edit(['loop.in'], lambda t: torch.cat([t[:, :88], 0 * t[:, 88:]], 1))),
		'positions': changed(edit_w=w_edit(['pos'], lambda t: t.roll(1, 0))),
		'side part of another layer': changed(edit_w=w_edit(['side.embed'], lambda t: t.roll(22, 1))),
		'final norm offset': changed(edit_w=w_edit(['final.norm'], lambda t: t - 1)),
	}
