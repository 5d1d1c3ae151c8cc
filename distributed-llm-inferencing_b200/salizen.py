"""The Salizen design: a pre-norm decoder with several residual streams (hyper-connections).  The embedding output is
the token's row times a constant plus a row of a table of hashed token pairs; it starts every stream.  Each sublayer
reads a weighted sum of the streams and all streams are then mixed and given a share of its result.  A layer's mixer
is `lightning` or `retention` (linear attention with a fixed decay per head: SiLU on q / k / v and one norm over all
heads, or rotation and a norm per head) or `parallel`: windowed softmax attention whose values are its unrotated keys,
with soft-capped scores, a sink and an output gate per channel, side by side with linear attention whose decay is made
per key channel from the input.  The feed-forward is gated (GELU, tanh form) or a mixture of gated SiLU experts whose
weights are the softmax over the chosen logits.  This module is the model definition only — the configuration reader,
the checkpoint's tensor names and synthetic weights; the step function, caches and kernels are
ragged_engine.RaggedEngine's.

config.json keys read here: architecture, vocab, width, streams, norm.eps, embedding {scale, bigram {buckets, mul_prev,
mul_cur}}, layers[] with type, mixer and mlp (null, {kind: dense, ff} or {kind: moe, expert {ff}, router {experts, top}}).
mixer: lightning {heads, dim, vdim, decay}; retention {heads, dim, vdim, decay, rot {base, dims, scaling}};
parallel {left_scale, right_scale, left {heads, kv_heads, dim, vdim, scale, softcap, mask {size}, rot {base, dims,
scaling {factor, low, high, original}}}, right {heads, dim, vdim, tau}}.
Tensor names: embed, bigram, head, final.norm; l<i>.norm1 / norm2 [width], l<i>.hc1 / hc2.{in, mix, out};
l<i>.mix.{q, k, v, g, o} (lightning: .norm [heads*vdim]); parallel: l<i>.mix.left.{q, k, g, o},
l<i>.mix.right.{q, k, v, g, o, norm, a1, a2, a2.b}; dense l<i>.mlp.{gate, up, down}; experts l<i>.mlp.e<k>.{gate, up,
down}, l<i>.mlp.router, l<i>.mlp.router.b.
"""
from __future__ import annotations

from typing import Dict, List

import torch

from .ragged_engine import HybridSpec, LayerSpec, MixerSpec, MoESpec

ARCHITECTURE = "Salizen"


def _rot(m: dict) -> dict:
    rot = m.get("rot")
    if not rot:
        return {}
    return {"rot_dims": int(rot["dims"]), "rot_base": float(rot["base"]), "rot_halves": True,
            "rot_scaling": dict(rot["scaling"]) if rot.get("scaling") else None}


def _heads(m: dict) -> dict:
    return {"heads": int(m["heads"]), "kv_heads": int(m.get("kv_heads", m["heads"])), "dim": int(m["dim"]), "vdim": int(m["vdim"])}


def _fixed_decay(i: int, m: dict) -> tuple:
    decay = tuple(float(d) for d in m["decay"])
    if len(decay) != int(m["heads"]) or not all(0.0 <= d <= 1.0 for d in decay):
        raise ValueError(f"layer {i}: {len(decay)} decays for {m['heads']} heads (each between 0 and 1)")
    return decay


def _mixer(i: int, L: dict) -> MixerSpec:
    m, kind = L["mixer"], L.get("type")
    if kind == "lightning":
        return MixerSpec(kind="linear_attention", **_heads(m), decay=_fixed_decay(i, m), qkv_silu=True, norm_heads_together=True,
                         gate_fn="sigmoid")
    if kind == "retention":
        return MixerSpec(kind="linear_attention", **_heads(m), **_rot(m), decay=_fixed_decay(i, m), k_scale=int(m["dim"]) ** -0.5,
                         gate_fn="silu")
    if kind == "parallel":
        a, b = m["left"], m["right"]
        if int(a["heads"]) % int(a.get("kv_heads", a["heads"])):
            raise ValueError(f"layer {i}: {a['heads']} query heads over {a['kv_heads']} key/value heads")
        if int(a["vdim"]) != int(a["dim"]):
            raise ValueError(f"layer {i}: the values are the keys, but their sizes are {a['vdim']} and {a['dim']}")
        left = MixerSpec(kind="attention", **_heads(a), **_rot(a), scale=float(a["scale"]), softcap=float(a.get("softcap") or 0.0),
                         window=int((a.get("mask") or {}).get("size", 0)), zero_sink=True, out_gate=True, keys_as_values=True,
                         out_scale=float(m["left_scale"]))
        right = MixerSpec(kind="linear_attention", **_heads(b), tau=float(b["tau"]), q_scale=int(b["dim"]) ** -0.5, gate_fn="silu",
                          out_scale=float(m["right_scale"]))
        return MixerSpec(kind="side_by_side", heads=left.heads, kv_heads=left.kv_heads, dim=left.dim, vdim=left.vdim,
                         parts=(left, right))
    raise ValueError(f"layer {i}: unknown mixer type {kind!r}")


def _moe(i: int, mlp: dict) -> MoESpec:
    r = mlp["router"]
    n, top = int(r["experts"]), int(r["top"])
    if not 1 <= top <= n:
        raise ValueError(f"layer {i}: {top} of {n} experts per token")
    return MoESpec(experts=n, identity=0, top=top, ff=int(mlp["expert"]["ff"]), limit=0.0, act="silu", router_bias=True)


def spec_from_config(cfg: dict) -> HybridSpec:
    if cfg.get("architecture") != ARCHITECTURE:
        raise ValueError(f"not a {ARCHITECTURE} config")
    layers: List[LayerSpec] = []
    for i, L in enumerate(cfg["layers"]):
        mlp = L.get("mlp")
        kind = None if mlp is None else mlp.get("kind", "dense")
        if kind not in (None, "dense", "moe"):
            raise ValueError(f"layer {i}: unknown feed-forward kind {kind!r}")
        layers.append(LayerSpec(mixer=_mixer(i, L), ff=int(mlp["ff"]) if kind == "dense" else 0,
                                moe=_moe(i, mlp) if kind == "moe" else None, pre_norm=True, ff_fn="gelu_tanh"))
    e = cfg.get("embedding") or {}
    bg = e.get("bigram")
    return HybridSpec(arch="salizen", vocab=int(cfg["vocab"]), width=int(cfg["width"]), eps=float(cfg["norm"]["eps"]), taps=1,
                      layers=layers, embed_scale=float(e.get("scale", 1.0)), norm_groups=1, streams=int(cfg.get("streams", 1)),
                      bigram=(int(bg["buckets"]), int(bg["mul_prev"]), int(bg["mul_cur"])) if bg else None)


def layer_tensors(spec: HybridSpec, sd: Dict[str, torch.Tensor], i: int) -> dict:
    """The checkpoint's tensors of layer i under the names the engine uses."""
    L = spec.layers[i]
    p = f"l{i}."

    def linear(q: str, m: MixerSpec) -> dict:
        d = {k: sd[q + k] for k in ("q", "k", "v", "g", "o")}
        if q + "norm" in sd:
            d["out_norm"] = sd[q + "norm"]
        if m.tau:
            d.update(a1=sd[q + "a1"], a2=sd[q + "a2"], a2_b=sd[q + "a2.b"])
        return d

    out = {"norm1": sd[p + "norm1"]}
    if L.mixer.kind == "side_by_side":
        left = {k: sd[p + "mix.left." + k] for k in ("q", "k", "g", "o")}
        out["parts"] = [left, linear(p + "mix.right.", L.mixer.parts[1])]
    else:
        out.update(linear(p + "mix.", L.mixer))
    for n in ("hc1", "hc2") if (L.ff or L.moe is not None) else ("hc1",):
        for k in ("in", "mix", "out"):
            out[f"{n}_{k}"] = sd[f"{p}{n}.{k}"]
    if L.ff:
        out.update(norm2=sd[p + "norm2"], gate=sd[p + "mlp.gate"], up=sd[p + "mlp.up"], down=sd[p + "mlp.down"])
    if L.moe is not None:
        out.update(norm2=sd[p + "norm2"], router=sd[p + "mlp.router"], router_b=sd[p + "mlp.router.b"],
                   experts=[tuple(sd[p + f"mlp.e{k}.{n}"] for n in ("gate", "up", "down")) for k in range(L.moe.experts)])
    return out


def model_tensors(spec: HybridSpec, sd: Dict[str, torch.Tensor]) -> dict:
    out = {"embed": sd["embed"], "head": sd["head"], "final_norm": sd["final.norm"],
           "layers": {i: layer_tensors(spec, sd, i) for i in range(spec.n_layers)}}
    if spec.bigram:
        out["bigram"] = sd["bigram"]
    return out


def random_state_dict(spec: HybridSpec, seed: int = 0, std: float = 0.05, device="cpu", rank: int = 16) -> Dict[str, torch.Tensor]:
    """Synthetic weights under the checkpoint's names (benchmarks and tests; there are no checkpoints offline).  rank: size
    of the decay projection."""
    g = torch.Generator(device="cpu").manual_seed(seed)
    W, S = spec.width, spec.streams

    def n(*shape, s=std, mean=0.0):
        return (mean + s * torch.randn(tuple(shape), generator=g)).to(torch.bfloat16).to(device)

    sd = {"embed": n(spec.vocab, W, s=1.0 / max(spec.embed_scale, 1e-6)), "head": n(spec.vocab, W), "final.norm": n(W, mean=1.0, s=0.1)}
    if spec.bigram:
        sd["bigram"] = n(spec.bigram[0] + 1, W, s=0.7)

    def linear(q: str, m: MixerSpec) -> None:
        H, D, V = m.heads, m.dim, m.vdim
        sd[q + "q"], sd[q + "k"] = n(H * D, W), n(H * D, W)
        sd[q + "v"], sd[q + "g"], sd[q + "o"] = n(H * V, W), n(H * V, W), n(W, H * V)
        if m.norm_heads_together:
            sd[q + "norm"] = n(H * V, mean=1.0, s=0.2)
        if m.tau:
            sd[q + "norm"] = n(V, mean=1.0, s=0.2)
            sd[q + "a1"], sd[q + "a2"], sd[q + "a2.b"] = n(rank, W), n(H * D, rank, s=0.5), n(H * D, mean=1.0, s=1.0)

    for i, L in enumerate(spec.layers):
        m, p = L.mixer, f"l{i}."
        sd[p + "norm1"] = n(W, mean=1.0, s=0.1)
        if m.kind == "side_by_side":
            a = m.parts[0]
            sd[p + "mix.left.q"], sd[p + "mix.left.k"] = n(a.heads * a.dim, W), n(a.kv_heads * a.dim, W)
            sd[p + "mix.left.g"], sd[p + "mix.left.o"] = n(a.heads * a.vdim, W), n(W, a.heads * a.vdim)
            linear(p + "mix.right.", m.parts[1])
        else:
            linear(p + "mix.", m)
        has_ff = bool(L.ff) or L.moe is not None
        for q in ("hc1", "hc2") if has_ff else ("hc1",):
            sd[f"{p}{q}.in"] = n(S, mean=1.0 / S, s=0.3)
            sd[f"{p}{q}.out"] = n(S, mean=1.0, s=0.3)
            sd[f"{p}{q}.mix"] = (0.8 * torch.eye(S) + 0.2 / S + 0.1 * torch.randn(S, S, generator=g)).to(torch.bfloat16).to(device)
        if has_ff:
            sd[p + "norm2"] = n(W, mean=1.0, s=0.1)
        if L.ff:
            sd[p + "mlp.gate"], sd[p + "mlp.up"], sd[p + "mlp.down"] = n(L.ff, W), n(L.ff, W), n(W, L.ff)
        if L.moe is not None:
            e = L.moe
            for k in range(e.experts):
                q = p + f"mlp.e{k}."
                sd[q + "gate"], sd[q + "up"], sd[q + "down"] = n(e.ff, W), n(e.ff, W), n(W, e.ff)
            sd[p + "mlp.router"], sd[p + "mlp.router.b"] = n(e.experts, W, s=0.3), n(e.experts, s=0.5)
    return sd


def config_from_spec(spec: HybridSpec) -> dict:
    """The config.json of a spec (tests and benchmarks write model directories with it)."""
    def sizes(m: MixerSpec) -> dict:
        return {"heads": m.heads, "dim": m.dim, "vdim": m.vdim}

    def rot(m: MixerSpec) -> dict:
        if not m.rot_dims:
            return {}
        r = {"base": m.rot_base, "dims": m.rot_dims}
        if m.rot_scaling:
            r["scaling"] = dict(m.rot_scaling)
        return {"rot": r}

    layers = []
    for L in spec.layers:
        m = L.mixer
        if m.kind == "side_by_side":
            a, b = m.parts
            kind = "parallel"
            mx = {"left_scale": a.out_scale, "right_scale": b.out_scale, "right": dict(sizes(b), tau=b.tau),
                  "left": dict(sizes(a), kv_heads=a.kv_heads, scale=a.scale, softcap=a.softcap, mask={"size": a.window}, **rot(a))}
        else:
            kind = "lightning" if m.qkv_silu else "retention"
            mx = dict(sizes(m), decay=list(m.decay), **rot(m))
        if L.moe is not None:
            mlp = {"kind": "moe", "expert": {"ff": L.moe.ff}, "router": {"experts": L.moe.experts, "top": L.moe.top}}
        else:
            mlp = {"kind": "dense", "ff": L.ff} if L.ff else None
        layers.append({"type": kind, "mixer": mx, "mlp": mlp})
    emb = {"scale": spec.embed_scale}
    if spec.bigram:
        emb["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), spec.bigram))
    return {"architecture": ARCHITECTURE, "vocab": spec.vocab, "width": spec.width, "streams": spec.streams, "embedding": emb,
            "norm": {"eps": spec.eps}, "layers": layers}
