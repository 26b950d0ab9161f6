"""Small random latent-attention models for the tests: configurations, checkpoint tensors, comparison with the oracle."""
import torch

from gptq_triton_b200.befalix import BefalixConfig, BefalixEngine, BefalixForCausalLM
from oracle import latent_oracle as O

# error of the logits (mean taken off, rms over the vocabulary, relative to the logits' spread) that rounding causes
LIMIT = {torch.float32: 1e-5, torch.bfloat16: 4.5e-2}


def layer(heads, dim, rot_dim, vdim, kv_rank, ff, base=10000.0, scale=None, kv_from=None, rot_dims=None):
	mixer = {'heads': heads, 'dim': dim, 'rot_dim': rot_dim, 'vdim': vdim, 'kv_rank': kv_rank, 'rot': {'base': base, 'dims': rot_dims or rot_dim},
			 'scale': scale if scale is not None else (dim + rot_dim) ** -0.5}
	if kv_from is not None:
		mixer['kv_from'] = kv_from
	return {'type': 'latent_attention', 'mixer': mixer, 'mlp': None if ff is None else {'kind': 'dense', 'ff': ff}}


def config(layers, width=72, vocab=101, eps=1e-5, residual_mult=0.8, logit_scale=1.7):
	return {'architecture': 'Befalix', 'layers': layers, 'width': width, 'vocab': vocab, 'norm': {'eps': eps}, 'residual_mult': residual_mult, 'logit_scale': logit_scale}


# every size its own, none a multiple of 16; a layer without feed-forward; two layers on one cache, one of them not next to it;
# scores large enough that single keys matter
ODD = config([layer(3, 20, 12, 24, 40, 56, scale=0.5), layer(5, 34, 6, 18, 28, None, base=300.0), layer(2, 50, 12, 74, 40, 90, kv_from=0), layer(7, 9, 6, 11, 28, 33, base=300.0, kv_from=1)])
# aligned sizes, two head tiles, several chunks of every kernel
WIDE = config([layer(17, 80, 48, 112, 208, 336, scale=0.25), layer(6, 144, 64, 96, 304, 208, base=1e5), layer(20, 32, 48, 48, 208, None, kv_from=0)], width=320, vocab=515,
			  residual_mult=1.0, logit_scale=1.0)
# part of the rotated entries pass unchanged, one head, one layer
PARTIAL = config([layer(1, 16, 32, 16, 16, 16, rot_dims=20, scale=1.0)], width=48, vocab=64, eps=1e-3)
CONFIGS = {'odd': ODD, 'wide': WIDE, 'partial': PARTIAL}


def tensors(cfg, seed=0):
	gen = torch.Generator().manual_seed(seed)
	out = {}
	for name, shape in BefalixConfig.from_dict(cfg).tensor_shapes().items():
		t = torch.randn(shape, generator=gen)
		if len(shape) == 2:
			t *= shape[1] ** -0.5 if name != 'embed' else 1.0
		elif name.endswith('.b'):
			t *= 0.1
		else:
			t = 1.0 + 0.2 * t
		out[name] = t.bfloat16()
	return out


def tokens(cfg, n, seed=0):
	return torch.randint(0, cfg['vocab'], (n,), generator=torch.Generator().manual_seed(1000 + seed))


def engine(cfg, dtype, max_seq, batch=1, seed=0, **kw):
	return BefalixEngine(BefalixForCausalLM(BefalixConfig.from_dict(cfg), tensors(cfg, seed), dtype, 'cuda'), batch, max_seq, **kw)


_oracle = {}


def oracle_logits(name, n, seed=0):
	"""Logits and per-layer residual streams of CONFIGS[name] (weights and tokens of `seed`), computed once."""
	key = (name, n, seed)
	if key not in _oracle:
		taps = []
		_oracle[key] = (O.forward(CONFIGS[name], tensors(CONFIGS[name], seed), tokens(CONFIGS[name], n, seed), collect=taps), taps)
	return _oracle[key]


def error(got, ref):
	"""Largest error over the positions, in units of the logits' standard deviation."""
	d = got.double().cpu() - ref
	d = d - d.mean(-1, keepdim=True)
	return float(d.pow(2).mean(-1).sqrt().max() / ref.std())


def feed_all(eng, toks, cuts):
	"""Feeds one sequence in portions of the given sizes; all logits [t, vocab]."""
	assert sum(cuts) == len(toks)
	out, p = [], 0
	for n in cuts:
		out.append(eng.feed(toks[None, p:p + n], list(range(n)))[0].clone())
		p += n
	return torch.cat(out)
