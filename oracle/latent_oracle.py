"""CPU restatement of the latent-attention decoder (Befalix designs), one function per mechanism.

Plain and slow on purpose: whole sequences, no cache, expanded keys and values, python loops over heads, one
dtype throughout (float64 by default).  Test infrastructure only; it shares no code with the product path.
`weights` is a dict of tensors under their checkpoint names, `config` the parsed config.json.
"""
from __future__ import annotations

import math

import torch


def layer_norm(x, w, b, eps):
	"""(x - mean) / sqrt(mean((x - mean)^2) + eps) * w + b over the last dimension."""
	d = x - x.mean(-1, keepdim=True)
	return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def rms_norm(x, w, eps):
	return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def rotate_interleaved(x, positions, base, dims):
	"""Rotates the pairs (0,1), (2,3), ... of the first `dims` entries of x [t, n] by positions * base^(-2i/dims)."""
	i = torch.arange(dims // 2, dtype=x.dtype)
	ang = positions.to(x.dtype)[:, None] * torch.pow(torch.tensor(float(base), dtype=x.dtype), -2.0 * i / dims)[None, :]
	c, s = torch.cos(ang), torch.sin(ang)
	out = x.clone()
	u, v = x[:, 0:dims:2], x[:, 1:dims:2]
	out[:, 0:dims:2] = u * c - v * s
	out[:, 1:dims:2] = v * c + u * s
	return out


def latent_rows(h, w_dkv, norm_w, mixer, eps, positions):
	"""What a layer with its own down projection caches: the normed latent [t, kv_rank] and the rotated shared key [t, rot_dim]."""
	y = h @ w_dkv.T
	r = mixer['kv_rank']
	return rms_norm(y[:, :r], norm_w, eps), rotate_interleaved(y[:, r:], positions, mixer['rot']['base'], mixer['rot']['dims'])


def causal_softmax_attention(scores, values):
	"""scores [t, t] of queries against keys of the same positions, values [t, n]."""
	t = scores.shape[0]
	visible = torch.arange(t)[None, :] <= torch.arange(t)[:, None]
	s = scores.masked_fill(~visible, -math.inf)
	p = torch.exp(s - s.max(-1, keepdim=True).values)
	return (p / p.sum(-1, keepdim=True)) @ values


def latent_attention(h, w, mixer, eps, positions, latent=None, key_rot=None):
	"""w: this layer's mixer tensors by short name ('q', 'uk', ...).  Returns (output [t, width], latent, key_rot)."""
	H, D, R, V = mixer['heads'], mixer['dim'], mixer['rot_dim'], mixer['vdim']
	if latent is None:
		latent, key_rot = latent_rows(h, w['dkv'], w['dkv.norm'], mixer, eps, positions)
	q = (h @ w['q'].T).reshape(-1, H, D + R)
	gate = torch.sigmoid(h @ w['g'].T)
	heads = []
	for n in range(H):
		qn = q[:, n, :D]
		qr = rotate_interleaved(q[:, n, D:], positions, mixer['rot']['base'], mixer['rot']['dims'])
		k = latent @ w['uk'][n * D:(n + 1) * D].T
		v = latent @ w['uv'][n * V:(n + 1) * V].T
		scores = (qn @ k.T + qr @ key_rot.T) * mixer['scale']
		heads.append(causal_softmax_attention(scores, v) * gate[:, n:n + 1])
	return torch.cat(heads, -1) @ w['o'].T, latent, key_rot


def dense_ff(h, w_gate, w_up, w_down):
	z = h @ w_gate.T
	return (z * torch.sigmoid(z) * (h @ w_up.T)) @ w_down.T


def forward(config, weights, tokens, dtype=torch.float64, collect=None):
	"""Logits [t, vocab] of one sequence; with a list `collect`, the residual stream after every layer is appended."""
	W = {k: v.to(dtype) for k, v in weights.items()}
	eps, m = config['norm']['eps'], config['residual_mult']
	tokens = torch.as_tensor(tokens)
	positions = torch.arange(len(tokens))
	x = W['embed'][tokens]
	rows = {}
	for i, layer in enumerate(config['layers']):
		pre = f'l{i}.'
		mix = {k[len(pre) + 4:]: v for k, v in W.items() if k.startswith(pre + 'mix.')}
		mx = layer['mixer']
		shared = rows[mx['kv_from']] if mx.get('kv_from') is not None else (None, None)
		y, latent, key_rot = latent_attention(x, mix, mx, eps, positions, *shared)
		rows[i] = (latent, key_rot)
		x = x + m * (layer_norm(y, W[pre + 'norm1'], W[pre + 'norm1.b'], eps) * W[pre + 'ls1'])
		if layer['mlp'] is not None:
			y = dense_ff(x, W[pre + 'mlp.gate'], W[pre + 'mlp.up'], W[pre + 'mlp.down'])
			x = x + m * (layer_norm(y, W[pre + 'norm2'], W[pre + 'norm2.b'], eps) * W[pre + 'ls2'])
		if collect is not None:
			collect.append(x.clone())
	x = layer_norm(x, W['final.norm'], W['final.norm.b'], eps)
	return x @ W['embed'].T * config['logit_scale']
