"""Plain restatement of the Finezen design in float64: whole sequences, one function per mechanism.

It is the oracle of the tests and imports nothing of the product.  A model is (cfg, sd): the dictionary of
config.json and the tensors under the checkpoint's names.  Notation: T tokens, W width, positions are 0-based per
sequence.  Every function takes and returns float64 tensors.

The design: e_t = embed[token_t] * scale.  A sublayer f is wrapped as x <- x + m D'(f(D(x))) with two elementwise
"dynamic tanh" maps D(z) = tanh(alpha z) * w + b in place of norms.  Mixers: windowed softmax attention with a sink,
rotation with interpolated frequencies on part of every head and a norm over the whole query / key projection, and windowed
latent attention without positions; both gate every head's output.  The feed-forward is a mixture of experts whose weights
scale the experts' INPUTS, beside a gated shared expert.  A range of layers may run several times; passes after the first
add the embedding output.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional, Tuple

import torch

F64 = torch.float64


def lin(h: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    return h @ w.to(F64).T


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * torch.sigmoid(x)


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w.to(F64)


def dyn_tanh(x: torch.Tensor, alpha: float, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    return torch.tanh(alpha * x) * w.to(F64) + b.to(F64)


def dt_named(x: torch.Tensor, sd: Dict[str, torch.Tensor], name: str) -> torch.Tensor:
    return dyn_tanh(x, float(sd[name + ".alpha"]), sd[name], sd[name + ".b"])


# ---------------------------------------------------------------------------------------------------- rotation
def rotation(rot: dict) -> Tuple[List[float], float]:
    """Angle per position of every pair and the factor on sine and cosine.  With scaling: pair i keeps its frequency while
    it turns more than `fast` times over `original` positions, is slowed by `factor` below `slow` turns, and between the
    two (in pair numbers, rounded outwards) is blended linearly."""
    base, dims, sc = float(rot["base"]), int(rot["dims"]), rot.get("scaling")
    freqs = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not sc:
        return freqs, 1.0

    def pair_with_turns(t: float) -> float:
        return dims * math.log(float(sc["original"]) / (2.0 * math.pi * t)) / (2.0 * math.log(base))

    first = max(math.floor(pair_with_turns(float(sc["fast"]))), 0)
    last = min(math.ceil(pair_with_turns(float(sc["slow"]))), dims - 1)
    out = []
    for i, f in enumerate(freqs):
        slowed = min(max((i - first) / max(last - first, 0.001), 0.0), 1.0)
        out.append(slowed * f / float(sc["factor"]) + (1.0 - slowed) * f)
    return out, 1.0 + 0.1 * math.log(float(sc["factor"]))


def rotate_halves(x: torch.Tensor, freqs: List[float], gain: float = 1.0) -> torch.Tensor:
    """x [T, heads, D]: dimensions i and i + n (n = len(freqs)) of every head are turned by position * freqs[i] and
    stretched by gain; the dimensions from 2n on stay."""
    n = len(freqs)
    out = x.clone()
    for t in range(x.shape[0]):
        for i in range(n):
            c, s = gain * math.cos(t * freqs[i]), gain * math.sin(t * freqs[i])
            u, v = x[t, :, i], x[t, :, i + n]
            out[t, :, i] = u * c - v * s
            out[t, :, i + n] = v * c + u * s
    return out


def rotate(x: torch.Tensor, rot: Optional[dict]) -> torch.Tensor:
    return x if not rot else rotate_halves(x, *rotation(rot))


# ---------------------------------------------------------------------------------------------------- attention
def window_visible(T: int, size: int) -> torch.Tensor:
    """bool [T, T]: query i sees key j when 0 <= i - j < size (size 0: every earlier key and itself)."""
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    ok = j <= i
    return ok & (i - j < size) if size > 0 else ok


def windowed_attention(q, k, v, scale: float, size: int, sink: Optional[torch.Tensor] = None) -> torch.Tensor:
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H, V]: softmax over the visible scores, for head h with exp(sink[h])
    more in the denominator; head h reads key/value head h // (H / G)."""
    T, H, _ = q.shape
    G = k.shape[1]
    vis = window_visible(T, size)
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for h in range(H):
        g = h // (H // G)
        s = ((q[:, h] @ k[:, g].T) * scale).masked_fill(~vis, -math.inf)
        if sink is not None:
            s = torch.cat((s, sink[h].to(F64).expand(T, 1)), dim=1)
        out[:, h] = torch.softmax(s, dim=-1)[:, :T] @ v[:, g]
    return out


def _size(m: dict) -> int:
    return int((m.get("mask") or {}).get("size", 0))


def head_gate(o: torch.Tensor, h: torch.Tensor, w_g: torch.Tensor) -> torch.Tensor:
    """o [T, H, V] times one sigmoid per head, made from the mixer's input; heads concatenated."""
    return (o * torch.sigmoid(lin(h, w_g))[:, :, None]).reshape(o.shape[0], -1)


def attention(h: torch.Tensor, sd: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, D, V = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = rms_norm(lin(h, sd[p + "q"]), sd[p + "q.norm"], eps).reshape(T, H, D)
    k = rms_norm(lin(h, sd[p + "k"]), sd[p + "k.norm"], eps).reshape(T, G, D)
    v = lin(h, sd[p + "v"]).reshape(T, G, V)
    o = windowed_attention(rotate(q, m.get("rot")), rotate(k, m.get("rot")), v, float(m["scale"]), _size(m), sd[p + "sink"])
    return lin(head_gate(o, h, sd[p + "g"]), sd[p + "o"])


def latent_attention(h: torch.Tensor, sd: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, D, V = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = lin(rms_norm(lin(h, sd[p + "dq"]), sd[p + "dq.norm"], eps), sd[p + "uq"]).reshape(T, H, D)
    c = rms_norm(lin(h, sd[p + "dkv"]), sd[p + "dkv.norm"], eps)
    k, v = lin(c, sd[p + "uk"]).reshape(T, H, D), lin(c, sd[p + "uv"]).reshape(T, H, V)
    o = windowed_attention(q, k, v, float(m["scale"]), _size(m))
    return lin(head_gate(o, h, sd[p + "g"]), sd[p + "o"])


def mixer(h: torch.Tensor, sd: Dict[str, torch.Tensor], p: str, L: dict, eps: float) -> torch.Tensor:
    return {"attention": attention, "latent_attention": latent_attention}[L["type"]](h, sd, p, L["mixer"], eps)


# ---------------------------------------------------------------------------------------------------- feed-forward
def gated(h: torch.Tensor, sd: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return lin(silu(lin(h, sd[p + "gate"])) * lin(h, sd[p + "up"]), sd[p + "down"])


def route(h: torch.Tensor, w_router: torch.Tensor, top: int):
    """Per row the experts with the largest sigmoid scores and those scores: (idx [T, top], weight [T, top])."""
    s = torch.sigmoid(lin(h, w_router))
    idx = torch.zeros(h.shape[0], top, dtype=torch.long)
    wt = torch.zeros(h.shape[0], top, dtype=F64)
    for t in range(h.shape[0]):
        order = sorted(range(s.shape[1]), key=lambda e: (-float(s[t, e]), e))[:top]
        idx[t], wt[t] = torch.tensor(order), s[t, order]
    return idx, wt


def moe_ff(h: torch.Tensor, sd: Dict[str, torch.Tensor], p: str, mlp: dict) -> torch.Tensor:
    idx, wt = route(h, sd[p + "router"], int(mlp["router"]["top"]))
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(idx[t].tolist(), wt[t].tolist()):
            out[t] = out[t] + gated(w * h[t:t + 1], sd, p + f"e{e}.")[0]
    if mlp.get("shared"):
        out = out + torch.sigmoid(lin(h, sd[p + "shared.sg"])) * gated(h, sd, p + "shared.")
    return out


# ---------------------------------------------------------------------------------------------------- model
def layer_order(cfg: dict) -> List[Tuple[int, bool]]:
    """(layer, is it the first of a pass after the first) for every layer run."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, False) for i in range(n)]
    a, b = int(lp["start"]), int(lp["stop"])
    runs = [(i, False) for i in range(a)]
    for t in range(int(lp["times"])):
        runs += [(i, t > 0 and i == a) for i in range(a, b)]
    return runs + [(i, False) for i in range(b, n)]


def forward(cfg: dict, sd: Dict[str, torch.Tensor], tokens: List[int], trace: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one whole sequence; trace (a list) collects the residual stream after every layer run."""
    eps, m = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    x0 = sd["embed"].to(F64)[torch.tensor(tokens, dtype=torch.long)] * float(cfg["embedding"]["scale"])
    x = x0
    for i, again in layer_order(cfg):
        L, p = cfg["layers"][i], f"l{i}."
        if again:
            x = x + x0
        y = mixer(dt_named(x, sd, p + "norm1"), sd, p + "mix.", L, eps)
        x = x + m * dt_named(y, sd, p + "norm1b")
        if L.get("mlp") is not None:
            y = moe_ff(dt_named(x, sd, p + "norm2"), sd, p + "mlp.", L["mlp"])
            x = x + m * dt_named(y, sd, p + "norm2b")
        if trace is not None:
            trace.append(x)
    return lin(dt_named(x, sd, "final.norm"), sd["head"])


def greedy(cfg: dict, sd: Dict[str, torch.Tensor], prompt: List[int], n_new: int) -> List[int]:
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(forward(cfg, sd, toks)[-1].argmax()))
    return toks
