"""Host-side parts of the Salizen design that need no GPU: the configuration reader, the registry, synthetic weights under
the checkpoint's names, and properties of the float64 oracle itself (causality, window, sink, cap, rotation, pair hash,
streams, router, recurrences)."""
import math

import pytest
import torch

from oracle import salizen_ref as R
from test_salizen_engine_gpu import cfg_a, cfg_b, cfg_c, prompt

F64 = torch.float64


def test_configuration_reader_and_registry():
    from dli_b200 import models, salizen

    cfg = cfg_a()
    assert models.family(cfg) == "salizen" and models.supports_float32(cfg)
    spec = models.spec_from_config(cfg)
    assert [L.mixer.kind for L in spec.layers] == ["linear_attention", "side_by_side", "linear_attention", "linear_attention", "side_by_side",
                                                   "linear_attention"]
    assert spec.streams == 3 and spec.bigram == (53, 13, 5) and spec.embed_scale == 3.0 and spec.norm_groups == 1 and spec.taps == 1
    assert all(L.pre_norm and L.ff_fn == "gelu_tanh" and not (L.token_shift or L.layer_scale or L.depth_avg) for L in spec.layers)
    m = spec.layers[0].mixer
    assert (m.heads, m.dim, m.vdim, m.qkv_silu, m.norm_heads_together, m.gate_fn, m.rot_dims, m.q_scale, m.k_scale) == \
           (3, 6, 10, True, True, "sigmoid", 0, 1.0, 1.0) and len(m.decay) == 3 and not m.tau
    m = spec.layers[2].mixer
    assert (m.qkv_silu, m.norm_heads_together, m.gate_fn, m.rot_dims, m.rot_halves) == (False, False, "silu", 6, True)
    assert abs(m.k_scale - 8 ** -0.5) < 1e-12 and m.q_scale == 1.0
    a, b = spec.layers[1].mixer.parts
    assert (a.window, a.chunk, a.softcap, a.zero_sink, a.sink, a.out_gate, a.head_gate, a.keys_as_values, a.rot_halves, a.out_scale) == \
           (9, 0, 5.0, True, False, True, False, True, True, 0.7) and a.rot_scaling["original"] == 64
    assert (b.tau, b.decay, b.out_scale, b.gate_fn) == (3.0, None, 0.4, "silu") and abs(b.q_scale - 6 ** -0.5) < 1e-12
    assert spec.layers[1].mixer.out_width == 4 * 8 + 2 * 4 and spec.layers[1].mixer.cached is a and spec.layers[0].mixer.cached is None
    assert spec.layers[4].mixer.parts[0].rot_scaling is None
    e = spec.layers[3].moe
    assert (e.experts, e.identity, e.top, e.ff, e.act, e.router_bias, e.gated, e.renorm, e.shared_ff) == (5, 0, 3, 20, "silu", True, True, True, 0)
    assert spec.layers[2].moe is None and spec.layers[2].ff == 0 and spec.layers[4].ff == 24
    for make in (cfg_a, cfg_b, cfg_c):
        s = salizen.spec_from_config(make())
        assert salizen.spec_from_config(salizen.config_from_spec(s)) == s


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][0].update(type="convolution"), lambda c: c["layers"][0]["mixer"]["decay"].pop(),
    lambda c: c["layers"][2]["mixer"].update(decay=[0.5, 1.5]), lambda c: c["layers"][1]["mixer"]["left"].update(vdim=4),
    lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=3), lambda c: c["layers"][0]["mlp"].update(kind="maxout"),
    lambda c: c["layers"][1]["mlp"]["router"].update(top=7), lambda c: c.update(architecture="Salis")])
def test_configurations_that_cannot_be_served_are_refused(change):
    from dli_b200 import salizen

    cfg = cfg_a()
    change(cfg)
    with pytest.raises(ValueError):
        salizen.spec_from_config(cfg)


def test_synthetic_weights_have_the_checkpoint_names_and_shapes():
    from dli_b200 import salizen

    cfg = cfg_a()
    spec = salizen.spec_from_config(cfg)
    sd = salizen.random_state_dict(spec, seed=3, rank=5)
    assert sd["embed"].shape == (97, 48) and sd["bigram"].shape == (54, 48) and sd["final.norm"].shape == (48,)
    assert sd["l0.mix.q"].shape == (18, 48) and sd["l0.mix.v"].shape == (30, 48) and sd["l0.mix.norm"].shape == (30,)
    assert sd["l1.mix.left.k"].shape == (16, 48) and sd["l1.mix.left.g"].shape == (32, 48) and sd["l1.mix.left.o"].shape == (48, 32)
    assert sd["l1.mix.right.a1"].shape == (5, 48) and sd["l1.mix.right.a2"].shape == (12, 5) and sd["l1.mix.right.a2.b"].shape == (12,)
    assert sd["l1.mix.right.norm"].shape == (4,) and "l1.mix.left.v" not in sd and "l2.mix.norm" not in sd and "l2.norm2" not in sd
    assert sd["l0.hc1.mix"].shape == (3, 3) and sd["l0.hc2.in"].shape == (3,) and "l2.hc2.in" not in sd
    assert sd["l1.mlp.router"].shape == (6, 48) and sd["l1.mlp.router.b"].shape == (6,) and sd["l1.mlp.e5.down"].shape == (48, 12)
    t = salizen.model_tensors(spec, sd)
    assert sorted(t["layers"]) == list(range(6)) and len(t["layers"][1]["parts"]) == 2 and len(t["layers"][1]["experts"]) == 6
    R.forward(cfg, sd, prompt(5, cfg["vocab"], 0))   # the oracle finds every tensor it needs


def test_state_slots_hold_an_integer_beside_the_states():
    from dli_b200.state_cache import StateSlots

    s = StateSlots(3, "cpu")
    s.add(("last",), dtype=torch.int32)
    s.add(("S", 0), 2, 4, 5)
    assert s[("last",)].dtype == torch.int32 and s[("last",)].shape == (3,) and s[("S", 0)].shape == (3, 2, 4, 5)
    assert s.bytes() == 3 * 4 + 3 * 40 * 4


def test_oracle_window_sink_and_cap():
    vis = R.window_visible(7, 3)
    assert vis[5].nonzero().flatten().tolist() == [3, 4, 5] and vis[1].nonzero().flatten().tolist() == [0, 1]
    assert R.window_visible(5, 0).tolist() == torch.ones(5, 5).tril().bool().tolist()
    q, k, v = torch.zeros(4, 2, 3, dtype=F64), torch.ones(4, 1, 3, dtype=F64), torch.ones(4, 1, 3, dtype=F64)
    o = R.capped_attention(q, k, v, 1.0, 5.0, 0)
    assert torch.allclose(o[:, 0, 0], torch.tensor([(t + 1) / (t + 2) for t in range(4)], dtype=F64))
    assert abs(float(R.softcap(torch.tensor(1e6, dtype=F64), 4.0)) - 4.0) < 1e-9
    assert abs(float(R.softcap(torch.tensor(0.01, dtype=F64), 4.0)) - 4.0 * math.tanh(0.0025)) < 1e-15
    assert float(R.softcap(torch.tensor(7.0, dtype=F64), 0.0)) == 7.0


def test_oracle_rotation_and_pairs():
    x = torch.zeros(2, 1, 6, dtype=F64)
    x[:, 0, 0], x[:, 0, 5] = 1.0, 9.0
    f = R.frequencies(100.0, 4, None)
    assert f == [1.0, 100.0 ** -0.5]
    y = R.rotate_halves(x, f, first_pos=3)
    assert torch.allclose(y[0, 0], torch.tensor([math.cos(3), 0.0, math.sin(3), 0.0, 0.0, 9.0], dtype=F64))
    assert R.bigram_rows([4, 6, 1], {"buckets": 10, "mul_prev": 7, "mul_cur": 3}) == [10, (28 + 18) % 10, (42 + 3) % 10]


def test_oracle_streams_and_router():
    xs = [torch.tensor([[1.0]], dtype=F64), torch.tensor([[10.0]], dtype=F64)]
    new = R.streams_write(xs, torch.tensor([[1.0, 2.0], [3.0, 4.0]]), torch.tensor([0.5, 0.25]), torch.tensor([[100.0]], dtype=F64))
    assert [float(t) for t in new] == [1.0 + 30.0 + 50.0, 2.0 + 40.0 + 25.0]
    assert float(R.streams_read(xs, torch.tensor([2.0, 0.5]))) == 7.0
    idx, wt = R.route(torch.eye(3, dtype=F64)[:1], torch.tensor([[1.0, 0, 0], [0.5, 0, 0], [-9.0, 0, 0]]).double(), torch.tensor([0.0, 0.0, 9.75]), 2)
    assert idx[0].tolist() == [0, 2] and torch.allclose(wt[0], torch.softmax(torch.tensor([1.0, 0.75], dtype=F64), 0))


def test_oracle_recurrence_closed_form():
    """With a constant decay the state is the weighted sum of the writes; carried on from a state it continues it."""
    torch.manual_seed(0)
    q, k, v = (torch.randn(9, 2, n, dtype=F64) for n in (4, 4, 3))
    w = R.fixed_decay([0.5, 0.9], 9, 4)
    o, S = R.matrix_recurrence(q, k, v, w)
    for h, d in enumerate((0.5, 0.9)):
        ref = sum(d ** (8 - s) * float(q[8, h] @ k[s, h]) * v[s, h] for s in range(9))
        assert torch.allclose(o[8, h], ref)
    _, S1 = R.matrix_recurrence(q[:4], k[:4], v[:4], w[:4])
    o2, S2 = R.matrix_recurrence(q[4:], k[4:], v[4:], w[4:], S=S1)
    assert torch.allclose(o2, o[4:]) and torch.allclose(S2, S)


def test_oracle_is_causal():
    from dli_b200 import salizen

    for make in (cfg_a, cfg_b, cfg_c):
        cfg = make()
        sd = salizen.random_state_dict(salizen.spec_from_config(cfg), seed=1, std=0.15, rank=5)
        toks = prompt(21, cfg["vocab"], 7)
        layers = []
        full = R.forward(cfg, sd, toks, layers)
        assert torch.allclose(full[:13], R.forward(cfg, sd, toks[:13]), atol=1e-10)
        assert len(layers) == len(cfg["layers"]) and layers[0].shape == (21, cfg["width"])
