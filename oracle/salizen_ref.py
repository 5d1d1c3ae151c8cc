"""Plain restatement of the Salizen design in float64: whole sequences, one function per mechanism.

It is the oracle of the tests and imports nothing of the product.  A model is (cfg, sd): the dictionary of
config.json and the tensors under the checkpoint's names.  Notation: T tokens, W width, positions are 0-based per
sequence.  Every function takes and returns float64 tensors.

The design: e_t = embed[token_t] * scale + bigram[row(token_(t-1), token_t)] starts every one of `streams` residual
streams.  A sublayer q of a layer reads u = sum_s a_s x_s, computes y = sublayer(rmsnorm(u) * w) and replaces the
streams by x_t <- sum_s M[s, t] x_s + b_t y.  The mixers are linear attention with a matrix state per head (fixed decay
per head with or without rotation, or a decay per key channel made from the input), and softmax attention side by side
with such a layer; the feed-forward is gated (GELU, tanh form) or a mixture of gated SiLU experts.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64


def rms_norm(x: torch.Tensor, w: Optional[torch.Tensor], eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis, times w when there is one."""
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w.to(F64)


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * torch.sigmoid(x)


def gelu_tanh(x: torch.Tensor) -> torch.Tensor:
    return 0.5 * x * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (x + 0.044715 * x ** 3)))


def lin(h: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    return h @ w.to(F64).T


# ---------------------------------------------------------------------------------------------------- embedding
def bigram_rows(tokens: List[int], bg: dict) -> List[int]:
    """Row of the pair table for every position; the first position has a row of its own behind the hashed ones."""
    n = int(bg["buckets"])
    rows = []
    for t, tok in enumerate(tokens):
        rows.append(n if t == 0 else (tokens[t - 1] * int(bg["mul_prev"]) + tok * int(bg["mul_cur"])) % n)
    return rows


def embed(cfg: dict, sd: Dict[str, torch.Tensor], tokens: List[int]) -> torch.Tensor:
    e = cfg["embedding"]
    x = sd["embed"].to(F64)[torch.tensor(tokens, dtype=torch.long)] * float(e.get("scale", 1.0))
    if e.get("bigram"):
        x = x + sd["bigram"].to(F64)[torch.tensor(bigram_rows(tokens, e["bigram"]), dtype=torch.long)]
    return x


# ---------------------------------------------------------------------------------------------------- streams
def streams_read(xs: List[torch.Tensor], a: torch.Tensor) -> torch.Tensor:
    u = torch.zeros_like(xs[0])
    for s in range(len(xs)):
        u = u + float(a[s]) * xs[s]
    return u


def streams_write(xs: List[torch.Tensor], mix: torch.Tensor, out: torch.Tensor, y: torch.Tensor) -> List[torch.Tensor]:
    """New streams from the old ones: mix is indexed [from, to]."""
    new = []
    for t in range(len(xs)):
        v = float(out[t]) * y
        for s in range(len(xs)):
            v = v + float(mix[s, t]) * xs[s]
        new.append(v)
    return new


# ---------------------------------------------------------------------------------------------------- rotation
def frequencies(base: float, dims: int, scaling: Optional[dict]) -> List[float]:
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling:
            wl = 2.0 * math.pi / f
            orig, lo, hi, fac = (float(scaling[k]) for k in ("original", "low", "high", "factor"))
            if wl > orig / lo:
                f = f / fac
            elif wl >= orig / hi:
                s = (orig / wl - lo) / (hi - lo)
                f = (1.0 - s) * f / fac + s * f
        out.append(f)
    return out


def rotate_halves(x: torch.Tensor, freqs: List[float], first_pos: int = 0) -> torch.Tensor:
    """x [T, heads, D]: dimensions i and i + n (n = len(freqs)) of every head are turned by position * freqs[i]."""
    n = len(freqs)
    out = x.clone()
    for t in range(x.shape[0]):
        for i in range(n):
            a = (first_pos + t) * freqs[i]
            u, v = x[t, :, i], x[t, :, i + n]
            out[t, :, i] = u * math.cos(a) - v * math.sin(a)
            out[t, :, i + n] = v * math.cos(a) + u * math.sin(a)
    return out


def rotate(x: torch.Tensor, rot: Optional[dict]) -> torch.Tensor:
    if not rot:
        return x
    return rotate_halves(x, frequencies(float(rot["base"]), int(rot["dims"]), rot.get("scaling")))


# ---------------------------------------------------------------------------------------------------- softmax attention
def window_visible(T: int, size: int) -> torch.Tensor:
    """bool [T, T]: query i sees key j when 0 <= i - j < size (size 0: every earlier key and itself)."""
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    ok = j <= i
    return ok & (i - j < size) if size > 0 else ok


def softcap(s: torch.Tensor, cap: float) -> torch.Tensor:
    return cap * torch.tanh(s / cap) if cap > 0 else s


def capped_attention(q, k, v, scale, cap, size):
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H, V]: softmax over the visible capped scores with 1 added to the
    denominator; head h reads key/value head h // (H / G)."""
    T, H, _ = q.shape
    G = k.shape[1]
    vis = window_visible(T, size)
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for h in range(H):
        g = h // (H // G)
        p = torch.exp(softcap((q[:, h] @ k[:, g].T) * scale, cap)) * vis
        out[:, h] = (p @ v[:, g]) / (1.0 + p.sum(-1, keepdim=True))
    return out


def attention(h: torch.Tensor, sd: Dict[str, torch.Tensor], p: str, m: dict) -> torch.Tensor:
    T = h.shape[0]
    H, G, D = int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    q = lin(h, sd[p + "q"]).reshape(T, H, D)
    k = lin(h, sd[p + "k"]).reshape(T, G, D)
    size = int((m.get("mask") or {}).get("size", 0))
    o = capped_attention(rotate(q, m.get("rot")), rotate(k, m.get("rot")), k, float(m["scale"]), float(m.get("softcap") or 0.0), size)
    return lin(o.reshape(T, H * D) * torch.sigmoid(lin(h, sd[p + "g"])), sd[p + "o"])


# ---------------------------------------------------------------------------------------------------- linear attention
def matrix_recurrence(q, k, v, decay, S=None):
    """q, k [T, H, D], v [T, H, V], decay [T, H, D] (factor of every state row at every position): S <- decay S + k v^T,
    o = S^T q, position by position.  Returns (o [T, H, V], S [H, D, V])."""
    T, H, D = q.shape
    V = v.shape[2]
    S = torch.zeros(H, D, V, dtype=F64) if S is None else S.clone()
    o = torch.zeros(T, H, V, dtype=F64)
    for t in range(T):
        S = decay[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return o, S


def fixed_decay(decay: List[float], T: int, D: int) -> torch.Tensor:
    return torch.tensor(decay, dtype=F64)[None, :, None].expand(T, len(decay), D)


def channel_decay(h: torch.Tensor, sd: Dict[str, torch.Tensor], p: str, H: int, D: int, tau: float) -> torch.Tensor:
    z = lin(lin(h, sd[p + "a1"]), sd[p + "a2"]) + sd[p + "a2.b"].to(F64)
    return (torch.sigmoid(z) ** (1.0 / tau)).reshape(h.shape[0], H, D)


def gated_linear_attention(h: torch.Tensor, sd: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, D, V = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = lin(h, sd[p + "q"]).reshape(T, H, D) / math.sqrt(D)
    k, v = lin(h, sd[p + "k"]).reshape(T, H, D), lin(h, sd[p + "v"]).reshape(T, H, V)
    o, _ = matrix_recurrence(q, k, v, channel_decay(h, sd, p, H, D, float(m["tau"])))
    o = rms_norm(o, sd[p + "norm"], eps).reshape(T, H * V)
    return lin(o * silu(lin(h, sd[p + "g"])), sd[p + "o"])


def retention(h: torch.Tensor, sd: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, D, V = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = rotate(lin(h, sd[p + "q"]).reshape(T, H, D), m.get("rot"))
    k = rotate(lin(h, sd[p + "k"]).reshape(T, H, D), m.get("rot")) / math.sqrt(D)
    v = lin(h, sd[p + "v"]).reshape(T, H, V)
    o, _ = matrix_recurrence(q, k, v, fixed_decay(m["decay"], T, D))
    o = rms_norm(o, None, eps).reshape(T, H * V)
    return lin(o * silu(lin(h, sd[p + "g"])), sd[p + "o"])


def lightning(h: torch.Tensor, sd: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, D, V = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q, k = silu(lin(h, sd[p + "q"])).reshape(T, H, D), silu(lin(h, sd[p + "k"])).reshape(T, H, D)
    v = silu(lin(h, sd[p + "v"])).reshape(T, H, V)
    o, _ = matrix_recurrence(q, k, v, fixed_decay(m["decay"], T, D))
    o = rms_norm(o.reshape(T, H * V), sd[p + "norm"], eps)
    return lin(o * torch.sigmoid(lin(h, sd[p + "g"])), sd[p + "o"])


def mixer(h: torch.Tensor, sd: Dict[str, torch.Tensor], p: str, L: dict, eps: float) -> torch.Tensor:
    m = L["mixer"]
    if L["type"] == "parallel":
        return float(m["left_scale"]) * attention(h, sd, p + "left.", m["left"]) + \
            float(m["right_scale"]) * gated_linear_attention(h, sd, p + "right.", m["right"], eps)
    return {"retention": retention, "lightning": lightning}[L["type"]](h, sd, p, m, eps)


# ---------------------------------------------------------------------------------------------------- feed-forward
def dense_ff(h: torch.Tensor, sd: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return lin(gelu_tanh(lin(h, sd[p + "gate"])) * lin(h, sd[p + "up"]), sd[p + "down"])


def route(h: torch.Tensor, w_router: torch.Tensor, bias: torch.Tensor, top: int):
    """Per row the experts with the largest logits and the softmax over just those: (idx [T, top], weight [T, top])."""
    z = lin(h, w_router) + bias.to(F64)
    idx = torch.zeros(h.shape[0], top, dtype=torch.long)
    wt = torch.zeros(h.shape[0], top, dtype=F64)
    for t in range(h.shape[0]):
        order = sorted(range(z.shape[1]), key=lambda e: (-float(z[t, e]), e))[:top]
        idx[t] = torch.tensor(order)
        wt[t] = torch.softmax(z[t, order], dim=0)
    return idx, wt


def moe_ff(h: torch.Tensor, sd: Dict[str, torch.Tensor], p: str, mlp: dict) -> torch.Tensor:
    r = mlp["router"]
    idx, wt = route(h, sd[p + "router"], sd[p + "router.b"], int(r["top"]))
    out = torch.zeros_like(h)
    for e in range(int(r["experts"])):
        y = lin(silu(lin(h, sd[p + f"e{e}.gate"])) * lin(h, sd[p + f"e{e}.up"]), sd[p + f"e{e}.down"])
        out = out + (wt * (idx == e)).sum(-1, keepdim=True) * y
    return out


# ---------------------------------------------------------------------------------------------------- model
def forward(cfg: dict, sd: Dict[str, torch.Tensor], tokens: List[int], trace: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one whole sequence; trace (a list) collects the sum of the streams after every layer."""
    eps = float(cfg["norm"]["eps"])
    x0 = embed(cfg, sd, tokens)
    xs = [x0.clone() for _ in range(int(cfg.get("streams", 1)))]
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = mixer(rms_norm(streams_read(xs, sd[p + "hc1.in"]), sd[p + "norm1"], eps), sd, p + "mix.", L, eps)
        xs = streams_write(xs, sd[p + "hc1.mix"], sd[p + "hc1.out"], y)
        mlp = L.get("mlp")
        if mlp is not None:
            h = rms_norm(streams_read(xs, sd[p + "hc2.in"]), sd[p + "norm2"], eps)
            y = dense_ff(h, sd, p + "mlp.") if mlp.get("kind", "dense") == "dense" else moe_ff(h, sd, p + "mlp.", mlp)
            xs = streams_write(xs, sd[p + "hc2.mix"], sd[p + "hc2.out"], y)
        if trace is not None:
            trace.append(sum(xs))
    return lin(rms_norm(sum(xs), sd["final.norm"], eps), sd["head"])


def greedy(cfg: dict, sd: Dict[str, torch.Tensor], prompt: List[int], n_new: int) -> List[int]:
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(forward(cfg, sd, toks)[-1].argmax()))
    return toks
