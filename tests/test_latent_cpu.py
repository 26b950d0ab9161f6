"""Host side of the latent-attention models: configuration, weight layout, registry, cache sharing, portions, trace replay."""
import ctypes
import json
import re
from pathlib import Path

import pytest
import torch

import latent_models as LM
from gptq_triton_b200 import _dense, registry
from gptq_triton_b200.befalix import BefalixConfig, BefalixForCausalLM
from gptq_triton_b200.cache import StaticCache
from gptq_triton_b200.dense import padded
from gptq_triton_b200.engine import StaticEngine
from oracle import latent_oracle as O

ROOT = Path(__file__).resolve().parent.parent


@pytest.fixture(scope='module')
def lib():
	from gptq_triton_b200 import build
	build.build(only=['dense'])
	return _dense.lib()


def test_header_binding_and_library_agree(lib):
	text = re.sub(r'/\*.*?\*/', '', (ROOT / 'include' / 'dense_b200.h').read_text(), flags=re.S)
	declared = sorted(set(re.findall(r'\b(dense_[a-z0-9_]+)\s*\(', text)))
	assert declared == sorted(_dense.exported_symbols())
	for n in declared:
		assert hasattr(lib, n)


def test_struct_layouts_match_the_header(tmp_path):
	"""sizeof and the last member's offset of every argument block, as the C compiler lays them out."""
	import subprocess
	structs = {'dense_rows_t': (_dense.Rows, 'status'), 'dense_epilogue_t': (_dense.Epilogue, 'tab_token'), 'dense_latent_t': (_dense.Latent, 'status'),
			   'dense_latent_prefill_t': (_dense.LatentPrefill, 'status'), 'dense_gqa_t': (_dense.Gqa, 'status'), 'dense_ssm_t': (_dense.Ssm, 'status')}
	src = '#include <stdio.h>\n#include "dense_b200.h"\nint main(void) {' + ''.join(
		f'printf("%zu %zu\\n", sizeof({n}), offsetof({n}, {last}));' for n, (_, last) in structs.items()) + 'return 0; }'
	(tmp_path / 's.c').write_text(src)
	subprocess.run(['gcc', '-I', str(ROOT / 'include'), str(tmp_path / 's.c'), '-o', str(tmp_path / 's')], check=True)
	lines = subprocess.run([str(tmp_path / 's')], capture_output=True, text=True, check=True).stdout.split('\n')
	for (_, (cls, last)), line in zip(structs.items(), lines):
		assert [int(v) for v in line.split()] == [ctypes.sizeof(cls), getattr(cls, last).offset]


def test_arguments_are_refused_on_the_host(lib):
	e, r, a = _dense.Epilogue(), _dense.Rows(), _dense.Latent()
	p = ctypes.c_void_p(0x1000)
	assert lib.dense_matmul(None, 64, p, 64, 1, 64, 16, 0, None, ctypes.byref(e), None, p, None) == -1          # neither rows nor x
	assert lib.dense_matmul(p, 64, p, 64, 1, 60, 16, 0, None, ctypes.byref(e), None, p, None) == -2             # K not a multiple of 16
	assert lib.dense_matmul(p, 64, ctypes.c_void_p(0x1004), 64, 1, 64, 16, 0, None, ctypes.byref(e), None, p, None) == -4
	assert lib.dense_matmul(p, 64, p, 64, 1, 64, 16, 0, None, ctypes.byref(e), None, p, None) == -1             # no output
	assert lib.dense_matmul(p, 64, p, 64, 0, 64, 16, 0, None, ctypes.byref(e), None, p, None) == 0              # no rows: nothing to do
	assert lib.dense_prepare_rows(ctypes.byref(r), 1, p, 64, 0, None) == -1
	assert lib.dense_latent_absorb(ctypes.byref(a), 0, None) == -1
	assert lib.dense_latent_prefill(None, None) == -1
	assert lib.dense_decode_rows_ok(8, 4096, 0) == 1 and lib.dense_decode_rows_ok(9, 4096, 0) == 0
	assert lib.dense_decode_rows_ok(8, 22016, 0) == 0 and lib.dense_decode_rows_ok(1, 22016, 1) == 1
	assert lib.dense_latent_prefill_ok(128, 64, 128) == 1 and lib.dense_latent_prefill_ok(192, 64, 256) == 1 and lib.dense_latent_prefill_ok(1024, 64, 128) == 0


def test_config_reads_every_constant_and_checks_shared_caches():
	c = BefalixConfig.from_dict(LM.ODD)
	assert (c.vocab_size, c.width, c.norm_eps, c.residual_mult, c.logit_scale) == (101, 72, 1e-5, 0.8, 1.7)
	assert [l.ff for l in c.layers] == [56, None, 90, 33] and [l.mixer.kv_from for l in c.layers] == [None, None, 0, 1]
	assert c.layers[1].mixer.rot_base == 300.0 and c.layers[0].mixer.scale == 0.5
	shapes = c.tensor_shapes()
	assert shapes['l0.mix.dkv'] == (52, 72) and 'l2.mix.dkv' not in shapes and 'l1.norm2' not in shapes and 'l1.mlp.up' not in shapes
	for bad in (2, 3, 1):          # a later layer, a layer that has no rows of its own, other sizes
		d = json.loads(json.dumps(LM.ODD))
		d['layers'][2 if bad != 3 else 3]['mixer']['kv_from'] = bad if bad != 3 else 2
		with pytest.raises(ValueError):
			BefalixConfig.from_dict(d)
	d = json.loads(json.dumps(LM.ODD))
	d['layers'][0]['type'] = 'something_else'
	with pytest.raises(ValueError):
		BefalixConfig.from_dict(d)


def test_packed_weights_hold_the_checkpoint():
	"""Padding and packing on the CPU: the packed matrices applied to padded rows give the checkpoint's projections."""
	cfg = BefalixConfig.from_dict(LM.ODD)
	T = LM.tensors(LM.ODD)
	model = BefalixForCausalLM(cfg, T, torch.float32, 'cpu')
	gen = torch.Generator().manual_seed(1)
	h = torch.randn((4, cfg.width), generator=gen)
	hp = torch.zeros((4, padded(cfg.width)))
	hp[:, :cfg.width] = h
	for i, layer in enumerate(cfg.layers):
		s, m = layer.mixer, model.layers[i].mixer
		y = hp @ m.w_in.T
		n_q = s.heads * (m.D + m.R)
		q = y[:, :n_q].view(4, s.heads, m.D + m.R)
		want = (h @ T[f'l{i}.mix.q'].float().T).view(4, s.heads, s.dim + s.rot_dim)
		assert torch.allclose(q[..., :s.dim], want[..., :s.dim], atol=1e-5) and torch.allclose(q[..., m.D:m.D + s.rot_dim], want[..., s.dim:], atol=1e-5)
		assert q[..., s.dim:m.D].abs().max() == 0 if m.D > s.dim else True
		g = y[:, -m.G:]
		assert torch.allclose(g[:, :s.heads], h @ T[f'l{i}.mix.g'].float().T, atol=1e-5)
		if s.kv_from is None:
			kv, want = y[:, n_q:n_q + s.row], h @ T[f'l{i}.mix.dkv'].float().T
			assert torch.allclose(kv[:, :s.kv_rank], want[:, :s.kv_rank], atol=1e-5) and torch.allclose(kv[:, m.C:m.C + s.rot_dim], want[:, s.kv_rank:], atol=1e-5)
		if layer.ff is not None:
			mlp = model.layers[i].mlp
			z = (hp @ mlp.gate_up.T).view(4, -1, 2, 8)
			a = torch.nn.functional.silu(z[:, :, 0]) * z[:, :, 1]
			out = (a.reshape(4, -1) @ mlp.down.T)[:, :cfg.width]
			ref = O.dense_ff(h, T[f'l{i}.mlp.gate'].float(), T[f'l{i}.mlp.up'].float(), T[f'l{i}.mlp.down'].float())
			assert torch.allclose(out, ref, atol=1e-4)
		norm = model.layers[i].mixer_norm
		assert torch.allclose(norm.gain[:cfg.width], cfg.residual_mult * T[f'l{i}.norm1'].float() * T[f'l{i}.ls1'].float(), rtol=1e-6)
		assert norm.gain[cfg.width:].abs().sum() == 0 and norm.shift[cfg.width:].abs().sum() == 0


def test_checkpoint_must_fit_the_configuration():
	cfg = BefalixConfig.from_dict(LM.PARTIAL)
	T = LM.tensors(LM.PARTIAL)
	with pytest.raises(ValueError, match='missing'):
		BefalixForCausalLM(cfg, {k: v for k, v in T.items() if k != 'l0.mix.g'}, torch.float32, 'cpu')
	with pytest.raises(ValueError, match='shape'):
		BefalixForCausalLM(cfg, {**T, 'l0.mix.o': torch.zeros(3, 3)}, torch.float32, 'cpu')
	with pytest.warns(UserWarning, match='does not use'):
		BefalixForCausalLM(cfg, {**T, 'extra': torch.zeros(1)}, torch.float32, 'cpu')
	with pytest.raises(ValueError):
		BefalixForCausalLM(cfg, T, torch.float16, 'cpu')


def test_registry_knows_models_by_their_config(tmp_path):
	def checkpoint(name, config, quant=False):
		d = tmp_path / name
		d.mkdir()
		(d / 'config.json').write_text(json.dumps(config))
		if quant:
			(d / 'quant_config.json').write_text('{"wbits": 4, "groupsize": 128}')
		return d
	assert registry.architecture_of(checkpoint('a', LM.ODD)).name == 'Befalix'
	assert registry.architecture_of(checkpoint('b', {'hidden_size': 512}, quant=True)).name == 'LlamaForCausalLM'
	assert registry.architecture_of(checkpoint('c', {'architectures': ['LlamaForCausalLM']})).name == 'LlamaForCausalLM'
	with pytest.raises(ValueError, match='not one of'):
		registry.architecture_of(checkpoint('d', {'architecture': 'Unknown'}))
	with pytest.raises(ValueError, match='runs in'):
		registry.load_model(tmp_path / 'a', 'cpu', torch.float16)


def test_cache_sharing():
	c = StaticCache([{'rows': (10, 4)}, {'rows': (10, 6)}, 0, 1, 0], batch=2, dtype=torch.float32, device='cpu')
	assert len(c) == 5 and c[2]['rows'] is c[0]['rows'] and c[4]['rows'] is c[0]['rows'] and c[3]['rows'] is c[1]['rows']
	assert c.nbytes() == 2 * 10 * (4 + 6) * 4
	for bad in ([0], [{'rows': (1, 1)}, 1], [{'rows': (1, 1)}, 0, 1]):
		with pytest.raises(ValueError):
			StaticCache(bad, 1, torch.float32, 'cpu')


class CountingEngine(StaticEngine):
	"""Logits that name what was fed: logits[v] is largest at v = (sum of all tokens so far) mod 7."""
	max_portion = 5

	def __init__(self, max_seq=40):
		super().__init__(None, 1, max_seq, 'cpu', use_graph=False)
		self.calls, self.sums = [], []

	def _one(self, tok, pos):
		assert pos == len(self.sums) or pos < len(self.sums)
		del self.sums[pos:]
		self.sums.append((self.sums[-1] if self.sums else 0) + int(tok))
		return torch.nn.functional.one_hot(torch.tensor(self.sums[-1] % 7), 7).float()

	def _portion(self, ids, start, want):
		self.calls.append((start, ids.shape[1]))
		rows = [self._one(t, start + i) for i, t in enumerate(ids[0].tolist())]
		return torch.stack([rows[w] for w in want])[None] if want else None

	def _step_body(self):
		self.calls.append((int(self.pos), 1))
		self.logits = self._one(self.tok, int(self.pos)).view(1, 1, -1)
		self.tok.copy_(self.logits.argmax(-1))
		self.pos.add_(1)


def test_feed_cuts_portions_and_orders_what_is_wanted():
	toks = torch.arange(1, 13)[None]
	e = CountingEngine()
	out = e.feed(toks, [11, 0, 6, 6, 4])
	assert e.calls == [(0, 5), (5, 5), (10, 2)] and e.next_pos == 12 and int(e.pos) == 12
	sums = torch.cumsum(toks[0], 0)
	assert out[0].argmax(-1).tolist() == [int(sums[i]) % 7 for i in (11, 0, 6, 6, 4)]
	assert int(e.tok) == int(sums[11]) % 7                          # the last place was wanted: the greedy token is ready
	assert e.feed(torch.tensor([[3, 4]]), []) is None and e.next_pos == 14
	one = e.feed(torch.tensor([[5]]), [0, 0])                       # a single token is a decode step
	assert one.shape == (1, 2, 7) and e.calls[-1] == (14, 1) and e.next_pos == 15
	with pytest.raises(RuntimeError, match='larger max_seq'):
		e.feed(torch.zeros((1, 26), dtype=torch.int64))
	e.reset()
	assert e.next_pos == 0 and int(e.feed(torch.tensor([[2, 2]]))[0, -1].argmax()) == 4
	with pytest.raises(ValueError):
		e.feed(torch.zeros((2, 1), dtype=torch.int64))


def test_generate_continues_the_prompt():
	e = CountingEngine()
	import gptq_triton_b200._lib as L
	L_status, L.kernel_status = L.kernel_status, lambda device=None: 0
	try:
		got = e.generate(torch.tensor([[3, 5]]), 4)[0].tolist()
	finally:
		L.kernel_status = L_status
	total, want = 8, []
	for _ in range(4):
		want.append(total % 7)
		total += want[-1]
	assert got == want


def test_replay_runs_requests_one_after_the_other():
	from gptq_triton_b200.trace import Replay
	r = Replay(CountingEngine())
	a = r.run({'step': 0, 'entries': [{'id': 'a', 'tokens': [1, 2, 3], 'want': [0, 2]}], 'end': []})
	assert a.argmax(-1).tolist() == [1, 6]
	with pytest.raises(RuntimeError, match='still holds'):
		r.run({'step': 1, 'entries': [{'id': 'b', 'tokens': [1], 'want': [0]}], 'end': []})
	r = Replay(CountingEngine())
	assert r.run({'step': 0, 'entries': [{'id': 'a', 'tokens': [1, 2, 3], 'want': []}], 'end': []}) is None
	assert r.run({'step': 1, 'entries': [{'id': 'a', 'tokens': [4], 'want': [0]}], 'end': ['a']}).argmax(-1).tolist() == [3]
	assert r.run({'step': 2, 'entries': [{'id': 'b', 'tokens': [2], 'want': [0]}], 'end': ['b']}).argmax(-1).tolist() == [2]      # position 0 again
	assert r.run({'step': 3, 'entries': [{'id': 'a', 'tokens': [5, 1], 'want': [1]}], 'end': ['a']}).argmax(-1).tolist() == [6]


def test_trace_run_refuses_a_number_format_at_the_start(tmp_path):
	from gptq_triton_b200 import trace
	(tmp_path / 'config.json').write_text('{"hidden_size": 512}')
	(tmp_path / 'quant_config.json').write_text('{"wbits": 4, "groupsize": 128}')
	assert trace.main(['--model', str(tmp_path), '--dtype', 'float32', '--out', str(tmp_path), '--max-tokens', '8']) == 3


def test_oracle_mechanisms():
	"""The oracle's own pieces against closed forms."""
	x = torch.tensor([[3.0, 4.0]], dtype=torch.float64)
	assert torch.allclose(O.rms_norm(x, torch.ones(2), 0.0), x / (12.5 ** 0.5))
	assert torch.allclose(O.layer_norm(x, torch.tensor([2.0, 2.0]), torch.tensor([1.0, 0.0]), 0.0), torch.tensor([[-1.0, 2.0]], dtype=torch.float64))
	v = torch.arange(6, dtype=torch.float64)[None].repeat(3, 1)
	r = O.rotate_interleaved(v, torch.tensor([0, 1, 2]), 10.0, 4)
	assert torch.equal(r[0], v[0]) and torch.equal(r[:, 4:], v[:, 4:])
	c, s = torch.cos(torch.tensor(2.0, dtype=torch.float64)), torch.sin(torch.tensor(2.0, dtype=torch.float64))
	assert torch.allclose(r[2, :2], torch.stack([0 * c - 1 * s, 1 * c + 0 * s]))
	f = 10.0 ** -0.5
	assert torch.allclose(r[1, 2], 2 * torch.cos(torch.tensor(f, dtype=torch.float64)) - 3 * torch.sin(torch.tensor(f, dtype=torch.float64)))
	a = O.causal_softmax_attention(torch.zeros((3, 3), dtype=torch.float64), torch.eye(3, dtype=torch.float64))
	assert torch.allclose(a, torch.tensor([[1, 0, 0], [0.5, 0.5, 0], [1 / 3, 1 / 3, 1 / 3]], dtype=torch.float64))
