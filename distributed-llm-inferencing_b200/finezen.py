"""The Finezen design: a decoder whose norms are dynamic tanh maps, tanh(alpha z) * w + b per channel, one before and one
after every sublayer (x += residual_mult * map'(sublayer(map(x)))).  A layer's mixer is `attention` (sliding window,
grouped key/value heads, one RMS norm over the whole query and key projections, YaRN-scaled half-split rotation of part of a
head, a sink per head) or `latent_attention` (queries and keys / values through latents, no positions, sliding window); both
multiply every head's output by a sigmoid made from the mixer's input.  The feed-forward is a mixture of gated SiLU experts with
sigmoid scores that are not renormalised and scale the experts' inputs, beside a shared expert with a sigmoid gate per token.  A
range of layers may run several times in a row with the same weights: every pass has caches of its own, and passes after the
first add the embedding output to the residual stream.  This module is the model definition only — the configuration reader, the
checkpoint's tensor names and synthetic weights; the step function, caches and kernels are ragged_engine.RaggedEngine's.

config.json keys read here: architecture, vocab, width, embedding.scale, norm.eps, residual_mult, loop {start, stop, times},
layers[] with type, mixer and mlp (null or {kind: moe, expert {ff}, router {experts, top}, shared {ff}}).  mixer: attention
{heads, kv_heads, dim, vdim, scale, mask {size}, rot {base, dims, scaling {factor, original, fast, slow}}}; latent_attention
{heads, dim, vdim, kv_rank, q_rank, scale, mask {size}}.
Tensor names: embed, head; every map <name> has <name> [width], <name>.b [width], <name>.alpha []: final.norm, l<i>.norm1,
l<i>.norm1b, l<i>.norm2, l<i>.norm2b; attention l<i>.mix.{q, k, v, q.norm, k.norm, sink, g, o}; latent attention
l<i>.mix.{dq, dq.norm, uq, dkv, dkv.norm, uk, uv, g, o}; experts l<i>.mlp.{router, e<k>.{gate, up, down}, shared.{gate, up, down,
sg}}.
"""
from __future__ import annotations

from typing import Dict, List

import torch

from .ragged_engine import HybridSpec, LayerSpec, MixerSpec, MoESpec

ARCHITECTURE = "Finezen"


def _window(m: dict) -> int:
    return int((m.get("mask") or {}).get("size") or 0)


def _mixer(i: int, L: dict) -> MixerSpec:
    m, kind = L["mixer"], L.get("type")
    H = int(m["heads"])
    if kind == "attention":
        G, rot = int(m.get("kv_heads", H)), m.get("rot") or {}
        if H % G:
            raise ValueError(f"layer {i}: {H} query heads over {G} key/value heads")
        if int(rot.get("dims", 0)) > int(m["dim"]) or int(rot.get("dims", 0)) % 2:
            raise ValueError(f"layer {i}: {rot['dims']} rotated dimensions in heads of {m['dim']}")
        return MixerSpec(kind="attention", heads=H, kv_heads=G, dim=int(m["dim"]), vdim=int(m["vdim"]), scale=float(m["scale"]),
                         rot_dims=int(rot.get("dims", 0)), rot_base=float(rot.get("base", 10000.0)), rot_halves=True,
                         rot_scaling=dict(rot["scaling"]) if rot.get("scaling") else None, window=_window(m), qk_norm=True,
                         qk_norm_whole=True, sink=True, head_gate=True)
    if kind == "latent_attention":
        return MixerSpec(kind="latent_attention", heads=H, kv_heads=1, dim=int(m["dim"]), vdim=int(m["vdim"]), scale=float(m["scale"]),
                         kv_rank=int(m["kv_rank"]), q_rank=int(m["q_rank"]), window=_window(m), head_gate=True)
    raise ValueError(f"layer {i}: unknown mixer type {kind!r}")


def _moe(i: int, mlp):
    if mlp is None:
        return None
    if mlp.get("kind", "moe") != "moe":
        raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
    r, sh = mlp["router"], mlp.get("shared")
    n, top = int(r["experts"]), int(r["top"])
    if not 1 <= top <= n:
        raise ValueError(f"layer {i}: {top} of {n} experts per token")
    return MoESpec(experts=n, identity=0, top=top, ff=int(mlp["expert"]["ff"]), limit=0.0, act="silu", score="sigmoid", renorm=False,
                   weight_in=True, shared_ff=int(sh["ff"]) if sh else 0, shared_gate=bool(sh))


def spec_from_config(cfg: dict) -> HybridSpec:
    """The layer RUNS in order: a looped range appears once per pass, later passes naming the first pass's run as the
    owner of their weights (`weights_of`) and `ckpt` the checkpoint's layer; `add_embedding` marks the first run of a pass
    after the first."""
    if cfg.get("architecture") != ARCHITECTURE:
        raise ValueError(f"not a {ARCHITECTURE} config")
    n, lp = len(cfg["layers"]), cfg.get("loop")
    a, b, times = (int(lp["start"]), int(lp["stop"]), int(lp["times"])) if lp else (0, 0, 0)
    if lp and not (0 <= a < b <= n and times >= 1):
        raise ValueError(f"loop {lp} does not fit {n} layers")
    order = [(i, 0) for i in range(a)] + [(i, t) for t in range(times) for i in range(a, b)] + [(i, 0) for i in range(b, n)]
    first_run: Dict[int, int] = {}
    layers: List[LayerSpec] = []
    for run, (i, t) in enumerate(order):
        L = cfg["layers"][i]
        layers.append(LayerSpec(mixer=_mixer(i, L), moe=_moe(i, L.get("mlp")), pre_norm=True, ckpt=i, weights_of=first_run.get(i),
                                add_embedding=t > 0 and i == a))
        first_run.setdefault(i, run)
    return HybridSpec(arch="finezen", vocab=int(cfg["vocab"]), width=int(cfg["width"]), eps=float(cfg["norm"]["eps"]), taps=1,
                      layers=layers, embed_scale=float((cfg.get("embedding") or {}).get("scale", 1.0)), norm_groups=1, norm_fn="tanh",
                      residual_mult=float(cfg.get("residual_mult", 1.0)))


def _map_tensors(sd: Dict[str, torch.Tensor], name: str, key: str) -> dict:
    return {key: sd[name], key + "_b": sd[name + ".b"], key + "_a": sd[name + ".alpha"]}


def layer_tensors(spec: HybridSpec, sd: Dict[str, torch.Tensor], run: int) -> dict:
    """The checkpoint's tensors of layer run `run` under the names the engine uses."""
    L = spec.layers[run]
    p = f"l{L.ckpt}."
    out = {}
    for k in ("norm1", "norm1b") + (("norm2", "norm2b") if L.moe is not None else ()):
        out.update(_map_tensors(sd, p + k, k))
    for k in ("q", "k", "v", "sink", "g", "o") if L.mixer.kind == "attention" else ("dq", "uq", "dkv", "uk", "uv", "g", "o"):
        out[k] = sd[p + "mix." + k]
    for k in ("q", "k") if L.mixer.kind == "attention" else ("dq", "dkv"):
        out[k + "_norm"] = sd[p + f"mix.{k}.norm"]
    if L.moe is not None:
        q = p + "mlp."
        out.update(router=sd[q + "router"], experts=[tuple(sd[f"{q}e{k}.{n}"] for n in ("gate", "up", "down")) for k in range(L.moe.experts)])
        if L.moe.shared_ff:
            out.update(shared=tuple(sd[f"{q}shared.{n}"] for n in ("gate", "up", "down")), shared_g=sd[q + "shared.sg"])
    return out


def model_tensors(spec: HybridSpec, sd: Dict[str, torch.Tensor]) -> dict:
    out = {"embed": sd["embed"], "head": sd["head"],
           "layers": {i: layer_tensors(spec, sd, i) for i, L in enumerate(spec.layers) if L.weights_of is None}}
    out.update(_map_tensors(sd, "final.norm", "final_norm"))
    return out


def random_state_dict(spec: HybridSpec, seed: int = 0, std: float = 0.05, device="cpu") -> Dict[str, torch.Tensor]:
    """Synthetic weights under the checkpoint's names (benchmarks and tests; there are no checkpoints offline)."""
    g = torch.Generator(device="cpu").manual_seed(seed)
    W = spec.width

    def n(*shape, s=std, mean=0.0):
        return (mean + s * torch.randn(tuple(shape), generator=g)).to(torch.bfloat16).to(device)

    sd = {"embed": n(spec.vocab, W, s=1.0 / max(spec.embed_scale, 1e-6)), "head": n(spec.vocab, W)}

    def tanh_map(name: str, alpha: float) -> None:
        sd[name], sd[name + ".b"] = n(W, mean=1.0, s=0.1), n(W, s=0.05)
        sd[name + ".alpha"] = torch.tensor(alpha * (1.0 + 0.2 * float(torch.randn((), generator=g)))).to(torch.bfloat16).to(device)

    tanh_map("final.norm", 0.5)
    for L in spec.layers:
        if L.weights_of is not None:
            continue
        m, p = L.mixer, f"l{L.ckpt}."
        H, D, V = m.heads, m.dim, m.vdim
        tanh_map(p + "norm1", 0.6)
        tanh_map(p + "norm1b", 1.0)
        if m.kind == "attention":
            G = m.kv_heads
            sd[p + "mix.q"], sd[p + "mix.k"], sd[p + "mix.v"] = n(H * D, W), n(G * D, W), n(G * V, W)
            sd[p + "mix.q.norm"], sd[p + "mix.k.norm"] = n(H * D, mean=1.0, s=0.2), n(G * D, mean=1.0, s=0.2)
            sd[p + "mix.sink"] = n(H, s=1.0)
        else:
            K, Q = m.kv_rank, m.q_rank
            sd[p + "mix.dq"], sd[p + "mix.dq.norm"] = n(Q, W), n(Q, mean=1.0, s=0.1)
            sd[p + "mix.uq"] = n(H * D, Q, s=1.0 / Q ** 0.5)
            sd[p + "mix.dkv"], sd[p + "mix.dkv.norm"] = n(K, W), n(K, mean=1.0, s=0.1)
            sd[p + "mix.uk"], sd[p + "mix.uv"] = n(H * D, K, s=1.0 / K ** 0.5), n(H * V, K, s=1.0 / K ** 0.5)
        sd[p + "mix.g"], sd[p + "mix.o"] = n(H, W, s=4 * std), n(W, H * V)
        if L.moe is not None:
            e, q = L.moe, p + "mlp."
            tanh_map(p + "norm2", 0.6)
            tanh_map(p + "norm2b", 1.0)
            sd[q + "router"] = n(e.experts, W, s=0.3)
            for k in range(e.experts):
                sd[f"{q}e{k}.gate"], sd[f"{q}e{k}.up"], sd[f"{q}e{k}.down"] = n(e.ff, W), n(e.ff, W), n(W, e.ff)
            if e.shared_ff:
                sd[q + "shared.gate"], sd[q + "shared.up"] = n(e.shared_ff, W), n(e.shared_ff, W)
                sd[q + "shared.down"], sd[q + "shared.sg"] = n(W, e.shared_ff), n(1, W, s=4 * std)
    return sd


def config_from_spec(spec: HybridSpec) -> dict:
    """The config.json of a spec (tests and benchmarks write model directories with it)."""
    runs = [L.ckpt for L in spec.layers]
    own = [L for L in spec.layers if L.weights_of is None]
    layers = []
    for L in own:
        m, e = L.mixer, L.moe
        mx = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale}
        if m.window:
            mx["mask"] = {"size": m.window}
        if m.kind == "attention":
            mx["kv_heads"] = m.kv_heads
            if m.rot_dims:
                mx["rot"] = {"base": m.rot_base, "dims": m.rot_dims}
                if m.rot_scaling:
                    mx["rot"]["scaling"] = dict(m.rot_scaling)
        else:
            mx.update(kv_rank=m.kv_rank, q_rank=m.q_rank)
        mlp = None
        if e is not None:
            mlp = {"kind": "moe", "expert": {"ff": e.ff}, "router": {"experts": e.experts, "top": e.top}}
            if e.shared_ff:
                mlp["shared"] = {"ff": e.shared_ff}
        layers.append({"type": m.kind, "mixer": mx, "mlp": mlp})
    cfg = {"architecture": ARCHITECTURE, "vocab": spec.vocab, "width": spec.width, "embedding": {"scale": spec.embed_scale},
           "norm": {"eps": spec.eps}, "residual_mult": spec.residual_mult, "layers": layers}
    looped = sorted({i for i in runs if runs.count(i) > 1})
    if looped:
        cfg["loop"] = {"start": looped[0], "stop": looped[-1] + 1, "times": runs.count(looped[0])}
    return cfg
