"""Host side of the Lifinex models: configuration, layer order, weight layout, carried state, argument checks, oracle pieces."""
import ctypes
import json

import pytest
import torch

import lifinex_models as LM
from gptq_triton_b200 import _dense, registry
from gptq_triton_b200.cache import Carried, StaticCache
from gptq_triton_b200.dense import RMSNorm, padded
from gptq_triton_b200.engine import StaticEngine
from gptq_triton_b200.gqa_attention import GroupedAttentionSpec, diff_lambda
from gptq_triton_b200.lifinex import LifinexConfig, LifinexForCausalLM
from gptq_triton_b200.ssm import StateSpaceSpec
from oracle import lifinex_oracle as O


@pytest.fixture(scope='module')
def lib():
	from gptq_triton_b200 import build
	build.build(only=['dense'])
	return _dense.lib()


def edited(cfg, f):
	c = json.loads(json.dumps(cfg))
	f(c)
	return c


def test_config_reads_every_size_and_constant():
	c = LifinexConfig.from_dict(LM.ODD)
	assert (c.vocab_size, c.width, c.norm_eps, c.max_positions, c.side_dim) == (101, 88, 1e-5, 1300, 22)
	assert (c.loop.start, c.loop.stop, c.loop.times) == (1, 4, 2) and [l.ff for l in c.layers] == [56, 33, None, None, 90]
	assert c.layers[0].mixer == GroupedAttentionSpec(6, 2, 20, 24, 0.5, 7.0, 2, 0.55)
	assert c.layers[1].mixer == StateSpaceSpec(6, 20, 24, 3, 4, 5)
	s = c.tensor_shapes()
	assert s['l0.mix.q'] == (240, 88) and s['l0.mix.k'] == (80, 88) and s['l0.mix.v'] == (48, 88) and s['l0.mix.lq2'] == (20,)
	assert s['l1.mix.in'] == (2 * 120 + 2 * 72 + 6, 88) and s['l1.mix.conv'] == (264, 4) and s['l3.mix.norm'] == (126,)
	assert s['loop.in'] == (88, 176) and s['loop.step'] == (2, 88) and s['side.embed'] == (101, 110) and s['l4.side.proj'] == (88, 22)
	assert 'l2.norm2' not in s and 'l3.mlp.up' not in s
	p = LifinexConfig.from_dict(LM.PLAIN)
	assert p.loop is None and p.side_dim is None and 'loop.in' not in p.tensor_shapes() and 'l0.side.gate' not in p.tensor_shapes()


@pytest.mark.parametrize('edit', [
	lambda c: c['loop'].update(stop=6), lambda c: c['loop'].update(start=4), lambda c: c['loop'].update(times=0),
	lambda c: c['layers'][0].update(type='something_else'), lambda c: c['layers'][0]['mlp'].update(kind='sparse'),
	lambda c: c['layers'][0]['mixer'].update(kv_heads=4), lambda c: c['layers'][0]['mixer'].update(softcap=0.0), lambda c: c['layers'][0]['mixer'].update(dim=513),
	lambda c: c['layers'][1]['mixer'].update(groups=4), lambda c: c['layers'][1]['mixer'].update(norm_groups=7), lambda c: c['layers'][1]['mixer'].update(state=257),
	lambda c: c['layers'][1]['mixer'].update(conv=17)])
def test_what_does_not_fit_is_refused(edit):
	with pytest.raises(ValueError):
		LifinexConfig.from_dict(edited(LM.ODD, edit))


@pytest.mark.parametrize('loop', [None, (0, 1, 1), (0, 5, 2), (1, 4, 3), (4, 5, 2), (2, 3, 4)])
def test_order_of_layer_runs(loop):
	c = LM.config(LM.ODD['layers'], loop=loop)
	runs = LifinexConfig.from_dict(c).runs()
	assert runs == O.layer_runs(c)
	if loop == (1, 4, 3):
		assert [i for i, _ in runs] == [0, 1, 2, 3, 1, 2, 3, 1, 2, 3, 4] and [t for _, t in runs if t is not None] == [0, 1, 2]


@pytest.mark.parametrize('name', list(LM.CONFIGS))
def test_packed_weights_hold_the_checkpoint(name):
	"""The packed matrices applied to padded rows give the checkpoint's projections."""
	cfg = LifinexConfig.from_dict(LM.CONFIGS[name])
	T = {k: v.float() for k, v in LM.tensors(LM.CONFIGS[name]).items()}
	m = LifinexForCausalLM(cfg, T, torch.float32, 'cpu')
	h = torch.randn((3, cfg.width), generator=torch.Generator().manual_seed(1))
	hp = torch.nn.functional.pad(h, (0, padded(cfg.width) - cfg.width))
	close = lambda a, b: torch.allclose(a, b, atol=2e-5)
	zero_pads = lambda t, n: t[..., n:].numel() == 0 or float(t[..., n:].abs().max()) == 0
	for i, (layer, packed) in enumerate(zip(cfg.layers, m.layers)):
		s, mx, p = layer.mixer, packed.mixer, f'l{i}.'
		y = hp @ mx.w_in.T
		if isinstance(s, GroupedAttentionSpec):
			nq, nk = s.heads * 2 * mx.D, s.kv_heads * 2 * mx.D
			for part, key, n, d in ((y[:, :nq], 'q', s.heads * 2, s.dim), (y[:, nq:nq + nk], 'k', s.kv_heads * 2, s.dim), (y[:, nq + nk:], 'v', s.kv_heads, s.vdim)):
				part = part.view(3, n, -1)
				assert close(part[..., :d], (h @ T[f'{p}mix.{key}'].T).view(3, n, d)) and zero_pads(part, d)
			o = torch.randn((3, s.heads, s.vdim), generator=torch.Generator().manual_seed(2))
			op = torch.nn.functional.pad(o, (0, mx.V - s.vdim))
			assert close((op.flatten(1) @ mx.w_o.T)[:, :cfg.width], o.flatten(1) @ T[p + 'mix.o'].T)
			want = O.diff_lambda({k: T[f'{p}mix.{k}'].double() for k in ('lq1', 'lk1', 'lq2', 'lk2')}, {'diff': s.diff})
			assert abs(mx.lam - float(want)) < 1e-12
		else:
			want = (h @ T[p + 'mix.in'].T).split([s.inner, s.channels, s.heads], 1)
			for at, w in zip((0, mx.conv_at, mx.dt_at), want):
				assert close(y[:, at:at + w.shape[1]], w)
			assert torch.equal(mx.conv_w[:, :s.channels].T, T[p + 'mix.conv']) and torch.equal(mx.conv_b[:s.channels], T[p + 'mix.conv.b'])
			assert torch.allclose(mx.a, -T[p + 'mix.A_log'].exp()) and mx.norm.parts == s.norm_groups
		assert torch.equal(packed.mixer_norm.weight[:cfg.width], 1 + T[p + 'norm1']) and zero_pads(packed.mixer_norm.weight[None], padded(cfg.width))
		if layer.ff is not None:
			z = (hp @ packed.mlp.gate_up.T).view(3, -1, 2, 8)
			a = O.gelu_tanh(z[:, :, 0]) * z[:, :, 1]
			assert close((a.reshape(3, -1) @ packed.mlp.down.T)[:, :cfg.width], O.dense_ff(h, T[p + 'mlp.gate'], T[p + 'mlp.up'], T[p + 'mlp.down']))
		if cfg.side_dim is not None:
			d = cfg.side_dim
			assert torch.equal(m.side[:, packed.side.column:packed.side.column + d], T['side.embed'][:, i * d:(i + 1) * d])
			assert close((hp @ packed.side.gate.T)[:, :d], h @ T[p + 'side.gate'].T)
	if cfg.loop is not None:
		x0 = torch.randn((3, cfg.width), generator=torch.Generator().manual_seed(3))
		x0p = torch.nn.functional.pad(x0, (0, padded(cfg.width) - cfg.width))
		got = (hp @ m.loop_x.T + x0p @ m.loop_x0.T + m.loop_step[0])[:, :cfg.width]
		assert close(got, O.loop_entry(h, x0, T['loop.in'], T['loop.step'][0]))


def test_checkpoint_must_fit_the_configuration():
	cfg, T = LifinexConfig.from_dict(LM.PLAIN), LM.tensors(LM.PLAIN)
	with pytest.raises(ValueError, match='missing'):
		LifinexForCausalLM(cfg, {k: v for k, v in T.items() if k != 'l1.mix.lk2'}, torch.float32, 'cpu')
	with pytest.raises(ValueError, match='shape'):
		LifinexForCausalLM(cfg, {**T, 'l0.mix.in': torch.zeros(3, 3)}, torch.float32, 'cpu')
	with pytest.warns(UserWarning, match='does not use'):
		LifinexForCausalLM(cfg, {**T, 'extra': torch.zeros(1)}, torch.float32, 'cpu')
	with pytest.raises(ValueError):
		LifinexForCausalLM(cfg, T, torch.float16, 'cpu')


def test_registry_knows_the_design(tmp_path):
	(tmp_path / 'config.json').write_text(json.dumps(LM.LOOPED))
	arch = registry.architecture_of(tmp_path)
	assert arch.name == 'Lifinex' and arch.dtypes == (torch.bfloat16, torch.float32) and arch.libraries == ('dense',)
	with pytest.raises(ValueError, match='runs in'):
		registry.load_model(tmp_path, 'cpu', torch.float16)


def test_carried_state_has_its_own_type_and_place():
	s = StateSpaceSpec(3, 10, 6, 1, 4, 2)
	c = StaticCache([s.cache_layout(), {'k': (7, 4)}, s.cache_layout()], 2, torch.bfloat16, 'cpu')
	assert c[0]['s'].shape == (2, 3, 10, 6) and c[0]['ring'].shape == (2, 4, padded(30 + 12)) and c[0]['s'].dtype == torch.float32 and c[1]['k'].dtype == torch.bfloat16
	assert len(c.carried) == 4 and c.carried[0] is c[0]['ring'] and c[0]['s'] is not c[2]['s']
	assert isinstance(s.cache_layout()['s'], Carried)


def test_every_pass_has_a_cache_of_its_own():
	cfg = LifinexConfig.from_dict(LM.ODD)
	spec = [cfg.layers[i].mixer for i, _ in cfg.runs()]
	c = StaticCache([m.cache_layout(9) if isinstance(m, GroupedAttentionSpec) else m.cache_layout() for m in spec], 1, torch.float32, 'cpu')
	assert len(c) == 8 and len({t.data_ptr() for l in c.layers for t in l.values()}) == 16


def test_arguments_are_refused_on_the_host(lib):
	p = 0x1000
	a = _dense.Gqa()
	assert lib.dense_gqa_append(ctypes.byref(a), 0, None) == -1 and lib.dense_gqa_attend(None, 0, None) == -1 and lib.dense_gqa_merge(ctypes.byref(a), 0, None) == -1
	a.M, a.rows_per_seq, a.heads, a.kv_heads, a.maps, a.dim, a.vdim, a.dim_true, a.vdim_true, a.max_seq, a.splits = 1, 1, 2, 1, 2, 32, 32, 32, 32, 8, 1
	a.pos = a.raw = a.k_cache = a.v_cache = a.q_hi = a.status = p
	a.raw_ld = 100          # shorter than a row
	assert lib.dense_gqa_append(ctypes.byref(a), 0, None) == -4
	a.maps = 3
	assert lib.dense_gqa_append(ctypes.byref(a), 0, None) == -1
	s = _dense.Ssm()
	assert lib.dense_ssm_step(ctypes.byref(s), None) == -1 and lib.dense_ssm_conv(None, 0, None) == -1 and lib.dense_ssm_chunked(ctypes.byref(s), None) == -1 and lib.dense_ssm_scan(ctypes.byref(s), None) == -1
	r = _dense.Rows()
	r.x_in, r.width, r.ld, r.eps, r.status, r.fin_norm, r.fin_groups = p, 48, 48, 1e-5, p, _dense.NORM_RMS, 5
	assert lib.dense_prepare_rows(ctypes.byref(r), 1, ctypes.c_void_p(p), 48, 0, None) == -1          # 48 entries in 5 parts
	e = _dense.Epilogue()
	e.mode, e.out, e.ldo, e.tab, e.tab_token, e.tab_rows, e.tab_ld, e.tab_col = _dense.EPI_TABLE, p, 16, p, p, 4, 32, 24
	v = ctypes.c_void_p(p)
	assert lib.dense_matmul(v, 64, v, 64, 1, 64, 16, 0, None, ctypes.byref(e), None, v, None) == -4          # columns beyond the table's row
	e.mode, e.act = _dense.EPI_F32, 7
	assert lib.dense_matmul(v, 64, v, 64, 1, 64, 16, 0, None, ctypes.byref(e), None, v, None) == -1
	assert lib.dense_gqa_splits(1, 32, 8, 2, 4096, 0) > 1 and lib.dense_gqa_splits(4096, 32, 8, 2, 4096, 0) == 1
	with pytest.raises(ValueError):
		RMSNorm(torch.ones(12), parts=5)


class SummingEngine(StaticEngine):
	"""State that every step overwrites: the running sum of all tokens."""

	def __init__(self):
		super().__init__(None, 1, 20, 'cpu', use_graph=False)
		self.total = torch.zeros(1)

	def _carried(self):
		return [self.total]

	def _step_body(self):
		self.total += self.tok.float().view(-1)
		self.logits = torch.nn.functional.one_hot(self.total.long() % 7, 7).float().view(1, 1, -1)
		self.tok.copy_(self.logits.argmax(-1))
		self.pos.add_(1)


def test_engine_names_what_a_trial_run_overwrites():
	e = SummingEngine()
	assert e.feed(torch.tensor([[5]])).argmax() == 5 and e._carried()[0] is e.total and StaticEngine(None, 1, 4, 'cpu')._carried() == []


def test_oracle_mechanisms():
	"""The oracle's own pieces against closed forms."""
	d = torch.float64
	x = torch.tensor([[3.0, 4.0, 0.0, 1.0]], dtype=d)
	assert torch.allclose(O.rms_norm_parts(x, torch.ones(4, dtype=d), 2, 0.0), torch.tensor([[3 / 12.5 ** 0.5, 4 / 12.5 ** 0.5, 0, 2 ** 0.5]], dtype=d))
	assert torch.allclose(O.rms_norm_centred(x, torch.zeros(4, dtype=d), 0.0), x / 6.5 ** 0.5)
	z = torch.linspace(-4, 4, 9, dtype=d)
	assert torch.allclose(O.gelu_tanh(z), torch.nn.functional.gelu(z, approximate='tanh')) and torch.allclose(O.silu(z), torch.nn.functional.silu(z))
	assert torch.allclose(O.softplus(z), torch.nn.functional.softplus(z)) and torch.allclose(O.soft_cap(z, 2.0), 2 * torch.tanh(z / 2))
	u = torch.arange(1.0, 5.0, dtype=d)[:, None]
	assert O.causal_conv(u, torch.tensor([[100.0, 10.0, 1.0]], dtype=d), torch.tensor([0.5], dtype=d))[:, 0].tolist() == [1.5, 12.5, 123.5, 234.5]
	ones = torch.ones((3, 1, 1), dtype=d)
	y = O.state_space_scan(ones, 2 * ones, ones, torch.full((3, 1), 0.5, dtype=d), torch.zeros(1, dtype=d), torch.tensor([3.0], dtype=d), 1)
	f = float(torch.exp(torch.tensor(-0.5)))
	assert torch.allclose(y.flatten(), torch.tensor([4.0, 1 + f + 3, 1 + f + f * f + 3], dtype=d))
	q = torch.zeros((3, 2, 2, 1), dtype=d)
	v = torch.tensor([[[1.0]], [[2.0]], [[6.0]]], dtype=d)
	assert torch.allclose(O.attention_maps(q, q[:, :1], v, 1.0, 5.0)[:, 1, 1, 0], torch.tensor([1.0, 1.5, 3.0], dtype=d))
	a = torch.tensor([[[[3.0, 4.0], [1.0, 0.0]]]], dtype=d)
	assert torch.allclose(O.combine_maps(a, 2.0, 0.25, 0.0), torch.tensor([[1.0, 4.0]], dtype=d) / 8.5 ** 0.5 * 0.75)
	e = torch.zeros(4)
	assert diff_lambda(e, e, e, e, 0.3) == 0.3 and abs(diff_lambda(e + 0.5, e + 0.5, e, e, 0.3) - (2.718281828459045 - 1 + 0.3)) < 1e-12


def test_mistakes_that_the_comparisons_must_see():
	"""Each mechanism changed in the oracle moves the logits far beyond the limits of the GPU tests."""
	found = LM.planted_mistakes()
	assert all(v > 1.5 * LM.LIMIT[torch.bfloat16][0] for v in found.values()), found
