"""Host-side parts of the Finezen design that need no GPU: the configuration reader, the registry, synthetic weights under
the checkpoint's names, the rotation table's frequencies, and properties of the float64 oracle itself (maps, window, sink,
gates, rotation, router, weighted inputs, loop, causality)."""
import math

import pytest
import torch

from oracle import finezen_ref as R
from test_finezen_engine_gpu import SCALING, cfg_a, cfg_b, cfg_c, prompt

F64 = torch.float64


def test_configuration_reader_and_registry():
    from dli_b200 import finezen, models

    cfg = cfg_a()
    assert models.family(cfg) == "finezen" and models.supports_float32(cfg)
    spec = models.spec_from_config(cfg)
    assert [L.ckpt for L in spec.layers] == [0, 1, 2, 1, 2, 1, 2, 3]
    assert [L.weights_of for L in spec.layers] == [None, None, None, 1, 2, 1, 2, None]
    assert [L.add_embedding for L in spec.layers] == [False, False, False, True, False, True, False, False]
    assert spec.norm_fn == "tanh" and spec.residual_mult == 0.8 and spec.embed_scale == 2.5 and spec.norm_groups == 1 and spec.taps == 1
    assert all(L.pre_norm and not (L.token_shift or L.layer_scale or L.depth_avg or L.ff) for L in spec.layers)
    m = spec.layers[0].mixer
    assert (m.kind, m.heads, m.kv_heads, m.dim, m.vdim, m.scale, m.window, m.chunk, m.keep_first) == ("attention", 4, 2, 8, 6, 0.4, 9, 0, 0)
    assert (m.rot_dims, m.rot_base, m.rot_halves, m.rot_scaling) == (8, 300.0, True, SCALING)
    assert m.qk_norm and m.qk_norm_whole and m.sink and m.head_gate and not m.out_gate
    m = spec.layers[1].mixer
    assert (m.kind, m.heads, m.dim, m.vdim, m.kv_rank, m.q_rank, m.rot_dims, m.window, m.sink, m.head_gate) == \
           ("latent_attention", 3, 6, 10, 12, 20, 0, 14, False, True)
    assert spec.layers[1].moe is None and spec.layers[2].mixer.rot_scaling is None
    e = spec.layers[2].moe
    assert (e.experts, e.top, e.ff, e.shared_ff, e.act, e.score, e.renorm, e.weight_in, e.shared_gate, e.groups, e.route_scale) == \
           (5, 3, 20, 8, "silu", "sigmoid", False, True, True, 1, 1.0)
    b = finezen.spec_from_config(cfg_b())
    assert [L.mixer.window for L in b.layers] == [1, 0, 0, 1] and not b.layers[0].moe.shared_gate and b.layers[0].moe.shared_ff == 0
    assert not any(L.add_embedding for L in b.layers) and b.layers[1].mixer.rot_dims == 0
    for make in (cfg_a, cfg_c):
        s = finezen.spec_from_config(make())
        assert finezen.spec_from_config(finezen.config_from_spec(s)) == s


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][0].update(type="convolution"), lambda c: c["layers"][0]["mixer"].update(kv_heads=3),
    lambda c: c["layers"][0]["mixer"]["rot"].update(dims=10), lambda c: c["layers"][0]["mixer"]["rot"].update(dims=5),
    lambda c: c["layers"][0]["mlp"].update(kind="maxout"), lambda c: c["layers"][0]["mlp"]["router"].update(top=7),
    lambda c: c["loop"].update(stop=5), lambda c: c["loop"].update(times=0), lambda c: c.update(architecture="Finer")])
def test_configurations_that_cannot_be_served_are_refused(change):
    from dli_b200 import finezen

    cfg = cfg_a()
    change(cfg)
    with pytest.raises(ValueError):
        finezen.spec_from_config(cfg)


def test_synthetic_weights_have_the_checkpoint_names_and_shapes():
    from dli_b200 import finezen

    cfg = cfg_a()
    spec = finezen.spec_from_config(cfg)
    sd = finezen.random_state_dict(spec, seed=3)
    assert sd["embed"].shape == sd["head"].shape == (97, 48) and sd["final.norm"].shape == sd["final.norm.b"].shape == (48,)
    assert sd["final.norm.alpha"].shape == () and sd["l1.norm1b.alpha"].shape == () and "l1.norm2" not in sd and "l4.norm1" not in sd
    assert sd["l0.mix.q.norm"].shape == (32,) and sd["l0.mix.k.norm"].shape == (16,) and sd["l0.mix.sink"].shape == (4,)
    assert sd["l0.mix.v"].shape == (12, 48) and sd["l0.mix.g"].shape == (4, 48) and sd["l0.mix.o"].shape == (48, 24)
    assert sd["l1.mix.dkv"].shape == (12, 48) and sd["l1.mix.uk"].shape == (18, 12) and sd["l1.mix.uv"].shape == (30, 12)
    assert sd["l1.mix.uq"].shape == (18, 20) and sd["l0.mlp.shared.sg"].shape == (1, 48) and sd["l2.mlp.e4.down"].shape == (48, 20)
    t = finezen.model_tensors(spec, sd)
    assert sorted(t["layers"]) == [0, 1, 2, 7] and len(t["layers"][0]["experts"]) == 6 and t["layers"][0]["shared_g"].shape == (1, 48)
    assert t["final_norm_a"].shape == () and {"norm1b", "norm1b_b", "norm1b_a"} <= set(t["layers"][1]) and "router" not in t["layers"][1]
    for make in (cfg_a, cfg_b, cfg_c):
        c = make()
        R.forward(c, finezen.random_state_dict(finezen.spec_from_config(c)), prompt(5, c["vocab"], 0))   # the oracle finds every tensor


@pytest.mark.parametrize("base,dims,sc", [
    (300.0, 8, SCALING), (10000.0, 32, {"factor": 8.0, "original": 512, "fast": 16.0, "slow": 2.0}),
    (500.0, 6, {"factor": 2.0, "original": 16, "fast": 1.0, "slow": 1.0}),          # both ends on one pair
    (50.0, 4, {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}),        # the ends beyond the last pair
    (50.0, 4, {"factor": 4.0, "original": 8, "fast": 64.0, "slow": 2.0})])          # the ends below the first
def test_rotation_frequencies_with_scaling_by_pair_number(base, dims, sc):
    from dli_b200.ragged_engine import rot_frequencies, rot_gain

    f, gain = R.rotation({"base": base, "dims": dims, "scaling": sc})
    assert torch.allclose(rot_frequencies(base, dims, sc), torch.tensor(f, dtype=F64), rtol=1e-13)
    assert abs(rot_gain(sc) - gain) < 1e-15 and gain == 1.0 + 0.1 * math.log(sc["factor"])
    plain, one = R.rotation({"base": base, "dims": dims})
    assert one == 1.0 and rot_gain(None) == 1.0 and torch.allclose(rot_frequencies(base, dims, None), torch.tensor(plain, dtype=F64))
    assert rot_gain({"factor": 3.0, "low": 1.0, "high": 4.0, "original": 64}) == 1.0
    if sc is SCALING:
        kinds = ["kept" if b == a else ("slowed" if abs(b - a / 3) < 1e-12 else "between") for a, b in zip(plain, f)]
        assert kinds == ["kept", "between", "slowed", "slowed"]


def test_oracle_maps_and_rotation():
    x = torch.tensor([[0.5, -2.0]], dtype=F64)
    y = R.dyn_tanh(x, 0.7, torch.tensor([2.0, 3.0]), torch.tensor([0.25, -1.0]))
    assert torch.allclose(y, torch.tensor([[2 * math.tanh(0.35) + 0.25, 3 * math.tanh(-1.4) - 1.0]], dtype=F64))
    x = torch.zeros(4, 1, 6, dtype=F64)
    x[:, 0, 0], x[:, 0, 5] = 1.0, 9.0
    y = R.rotate_halves(x, [1.0, 0.1], gain=2.0)
    assert torch.allclose(y[3, 0], torch.tensor([2 * math.cos(3), 0.0, 2 * math.sin(3), 0.0, 0.0, 9.0], dtype=F64))


def test_oracle_window_and_sink():
    vis = R.window_visible(7, 3)
    assert vis[5].nonzero().flatten().tolist() == [3, 4, 5] and vis[1].nonzero().flatten().tolist() == [0, 1]
    assert R.window_visible(5, 0).tolist() == torch.ones(5, 5).tril().bool().tolist()
    q, k, v = torch.zeros(4, 2, 3, dtype=F64), torch.ones(4, 1, 3, dtype=F64), torch.ones(4, 1, 3, dtype=F64)
    sink = torch.tensor([0.0, math.log(3.0)])
    o = R.windowed_attention(q, k, v, 5.0, 2, sink)
    n = torch.tensor([1.0, 2.0, 2.0, 2.0], dtype=F64)
    assert torch.allclose(o[:, 0, 0], n / (n + 1)) and torch.allclose(o[:, 1, 0], n / (n + 3), atol=1e-6)
    assert torch.allclose(R.windowed_attention(q, k, v, 5.0, 2), torch.ones(4, 2, 3, dtype=F64))


def test_oracle_router_and_weighted_inputs():
    """The weight goes through the experts' nonlinearity: with one expert of one channel the output is silu(w g) (w u)."""
    h = torch.eye(2, dtype=F64)[:1]
    idx, wt = R.route(h, torch.tensor([[0.5, 0.0], [-3.0, 0.0], [2.0, 0.0]]), 2)
    assert idx[0].tolist() == [2, 0] and torch.allclose(wt[0], torch.sigmoid(torch.tensor([2.0, 0.5], dtype=F64)))
    sd = {"router": torch.tensor([[0.5, 0.0]]), "e0.gate": torch.tensor([[2.0, 0.0]]), "e0.up": torch.tensor([[4.0, 0.0]]),
          "e0.down": torch.tensor([[1.0], [0.0]]), "shared.gate": torch.tensor([[1.0, 0.0]]), "shared.up": torch.tensor([[1.0, 0.0]]),
          "shared.down": torch.tensor([[0.0], [1.0]]), "shared.sg": torch.tensor([[-1.0, 0.0]])}
    w = 1.0 / (1.0 + math.exp(-0.5))
    y = R.moe_ff(h, sd, "", {"router": {"top": 1}, "shared": {"ff": 1}})
    sig = lambda z: 1.0 / (1.0 + math.exp(-z))  # noqa: E731
    assert abs(float(y[0, 0]) - 2 * w * sig(2 * w) * 4 * w) < 1e-12 and abs(float(y[0, 1]) - sig(-1.0) * sig(1.0)) < 1e-12


def test_oracle_loop_order():
    assert R.layer_order({"layers": [0] * 4, "loop": {"start": 1, "stop": 3, "times": 3}}) == \
           [(0, False), (1, False), (2, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    assert R.layer_order({"layers": [0] * 2, "loop": {"start": 1, "stop": 2, "times": 2}}) == [(0, False), (1, False), (1, True)]
    assert R.layer_order({"layers": [0] * 2}) == [(0, False), (1, False)]


def test_oracle_is_causal():
    from dli_b200 import finezen

    for make in (cfg_a, cfg_b, cfg_c):
        cfg = make()
        sd = finezen.random_state_dict(finezen.spec_from_config(cfg), seed=1, std=0.15)
        toks = prompt(21, cfg["vocab"], 7)
        layers = []
        full = R.forward(cfg, sd, toks, layers)
        assert torch.allclose(full[:13], R.forward(cfg, sd, toks[:13]), atol=1e-10)
        assert len(layers) == len(R.layer_order(cfg)) and layers[0].shape == (21, cfg["width"])
