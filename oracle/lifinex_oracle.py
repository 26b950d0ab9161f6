"""CPU restatement of the Lifinex decoder, one function per mechanism.

Plain and slow on purpose: whole sequences, no cache and no carried state, python loops over heads, maps and tokens, one
dtype throughout (float64 by default).  Test infrastructure only; it shares no code with the product path.
`weights` is a dict of tensors under their checkpoint names, `config` the parsed config.json.
"""
from __future__ import annotations

import math

import torch


def unit_rms(x, eps):
	"""x over its root mean square along the last dimension."""
	return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
	return unit_rms(x, eps) * w


def rms_norm_centred(x, w, eps):
	"""RMS norm whose weight is stored as its distance from one."""
	return unit_rms(x, eps) * (1 + w)


def rms_norm_parts(x, w, parts, eps):
	"""Each of `parts` equal slices of the last dimension by its own root mean square."""
	t, n = x.shape
	return unit_rms(x.reshape(t, parts, n // parts), eps).reshape(t, n) * w


def silu(z):
	return z / (1 + torch.exp(-z))


def gelu_tanh(z):
	return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
	return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def soft_cap(s, cap):
	return s if cap is None else cap * torch.tanh(s / cap)


def causal_softmax(s):
	t = s.shape[0]
	s = s.masked_fill(torch.arange(t)[None, :] > torch.arange(t)[:, None], -math.inf)
	p = torch.exp(s - s.max(-1, keepdim=True).values)
	return p / p.sum(-1, keepdim=True)


def diff_lambda(w, mixer):
	return torch.exp((w['lq1'] * w['lk1']).sum()) - torch.exp((w['lq2'] * w['lk2']).sum()) + mixer['diff']


def attention_maps(q, k, v, scale, cap):
	"""q [t, heads, maps, dim], k [t, kv_heads, maps, dim], v [t, kv_heads, vdim] -> every map's output [t, heads, maps, vdim]."""
	t, H, n, _ = q.shape
	G = k.shape[1]
	out = torch.empty((t, H, n, v.shape[2]), dtype=q.dtype)
	for h in range(H):
		g = h // (H // G)
		for m in range(n):
			out[:, h, m] = causal_softmax(soft_cap(q[:, h, m] @ k[:, g, m].T * scale, cap)) @ v[:, g]
	return out


def normed_qkv(h, w, mixer, eps, maps=2):
	t, H, G, D, V = h.shape[0], mixer['heads'], mixer['kv_heads'], mixer['dim'], mixer['vdim']
	q = rms_norm((h @ w['q'].T).reshape(t, H, maps, D), w['q.norm'], eps)
	k = rms_norm((h @ w['k'].T).reshape(t, G, maps, D), w['k.norm'], eps)
	return q, k, (h @ w['v'].T).reshape(t, G, V)


def combine_maps(a, lam, diff, eps):
	"""a [t, heads, 2, vdim] -> [t, heads * vdim]."""
	return (unit_rms(a[:, :, 0] - lam * a[:, :, 1], eps) * (1 - diff)).flatten(1)


def differential_attention(h, w, mixer, eps):
	a = attention_maps(*normed_qkv(h, w, mixer, eps), mixer['scale'], mixer['softcap'])
	return combine_maps(a, diff_lambda(w, mixer), mixer['diff'], eps) @ w['o'].T


def plain_attention(h, w, mixer, eps):
	"""The same with a single map per head."""
	return attention_maps(*normed_qkv(h, w, mixer, eps, 1), mixer['scale'], mixer['softcap']).flatten(1) @ w['o'].T


def causal_conv(u, w, b):
	"""Per channel: out[t] = b + sum_k w[k] u[t - (taps - 1) + k], u = 0 before the start."""
	t, taps = u.shape[0], w.shape[1]
	padded = torch.cat([torch.zeros((taps - 1, u.shape[1]), dtype=u.dtype), u])
	out = b.expand(t, -1).clone()
	for k in range(taps):
		out = out + padded[k:k + t] * w[:, k]
	return out


def state_space_scan(x, B, C, dt, A_log, D, groups):
	"""x [t, heads, vdim], B and C [t, groups, state], dt [t, heads] -> y [t, heads, vdim]."""
	t, H, P = x.shape
	y = torch.empty_like(x)
	for n in range(H):
		g = n // (H // groups)
		S = torch.zeros((B.shape[2], P), dtype=x.dtype)
		for i in range(t):
			S = torch.exp(-torch.exp(A_log[n]) * dt[i, n]) * S + dt[i, n] * torch.outer(B[i, g], x[i, n])
			y[i, n] = S.T @ C[i, g] + D[n] * x[i, n]
	return y


def mamba2(h, w, mixer, eps):
	t, H, P, N, G = h.shape[0], mixer['heads'], mixer['vdim'], mixer['state'], mixer['groups']
	inner, bc = H * P, G * N
	z, xbc, dt = (h @ w['in'].T).split([inner, inner + 2 * bc, H], dim=1)
	xbc = silu(causal_conv(xbc, w['conv'], w['conv.b']))
	x, B, C = xbc.split([inner, bc, bc], dim=1)
	y = state_space_scan(x.reshape(t, H, P), B.reshape(t, G, N), C.reshape(t, G, N), softplus(dt + w['dt_bias']), w['A_log'], w['D'], G)
	y = rms_norm_parts(y.reshape(t, inner) * silu(z), w['norm'], mixer['norm_groups'], eps)
	return y @ w['o'].T


MIXERS = {'attention': differential_attention, 'mamba2': mamba2}


def dense_ff(h, w_gate, w_up, w_down):
	return (gelu_tanh(h @ w_gate.T) * (h @ w_up.T)) @ w_down.T


def token_side(x, e, w_gate, w_proj, norm_w, eps):
	"""What a layer adds for its own part e [t, dim] of a per-token table."""
	return rms_norm((gelu_tanh(x @ w_gate.T) * e) @ w_proj.T, norm_w, eps)


def loop_entry(x, x0, w_in, step):
	"""Start of a pass over the looped layers: both streams mixed, and the pass's own vector."""
	return torch.cat([x, x0], -1) @ w_in.T + step


def layer_runs(config):
	"""(layer, pass or None) in the order in which layers run; pass is given at the first layer of every pass."""
	n, loop = len(config['layers']), config.get('loop')
	if not loop:
		return [(i, None) for i in range(n)]
	runs = [(i, None) for i in range(loop['start'])]
	for t in range(loop['times']):
		runs += [(i, t if i == loop['start'] else None) for i in range(loop['start'], loop['stop'])]
	return runs + [(i, None) for i in range(loop['stop'], n)]


def run_layer(x, W, i, layer, tokens, config):
	pre, eps = f'l{i}.', config['norm']['eps']
	mix = {k[len(pre) + 4:]: v for k, v in W.items() if k.startswith(pre + 'mix.')}
	x = x + MIXERS[layer['type']](rms_norm_centred(x, W[pre + 'norm1'], eps), mix, layer['mixer'], eps)
	if layer['mlp'] is not None:
		x = x + dense_ff(rms_norm_centred(x, W[pre + 'norm2'], eps), W[pre + 'mlp.gate'], W[pre + 'mlp.up'], W[pre + 'mlp.down'])
	if config.get('token_side'):
		d = config['token_side']['dim']
		x = x + token_side(x, W['side.embed'][tokens][:, i * d:(i + 1) * d], W[pre + 'side.gate'], W[pre + 'side.proj'], W[pre + 'side.norm'], eps)
	return x


def forward(config, weights, tokens, dtype=torch.float64, collect=None):
	"""Logits [t, vocab] of one sequence; with a list `collect`, the residual stream after every layer run is appended."""
	W = {k: v.to(dtype) for k, v in weights.items()}
	tokens = torch.as_tensor(tokens)
	x = x0 = W['embed'][tokens] + W['pos'][:len(tokens)]
	for i, t in layer_runs(config):
		if t is not None:
			x = loop_entry(x, x0, W['loop.in'], W['loop.step'][t])
		x = run_layer(x, W, i, config['layers'][i], tokens, config)
		if collect is not None:
			collect.append(x.clone())
	return rms_norm_centred(x, W['final.norm'], config['norm']['eps']) @ W['head'].T
