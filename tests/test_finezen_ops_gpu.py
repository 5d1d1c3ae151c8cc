"""Each mechanism of the Finezen design alone: kernels against float64 restatements (oracle/finezen_ref.py), on inputs made so
that a fault shows — maps whose offset and slope differ per channel, rows in every position of a router's row group, logits
where fp32's sigmoid is already 1, weights far from 1 in front of the experts' activation, keys planted at a window's edges,
scratch full of garbage."""
import math

import pytest
import torch

pytestmark = pytest.mark.gpu

from oracle import finezen_ref as R  # noqa: E402

DEV = "cuda:0"
F64 = torch.float64


def close(got, ref, tol):
    g = got.double().cpu()
    assert torch.isfinite(g).all()
    err = (g - ref).abs().max() / max(float(ref.abs().max()), 1e-9)
    assert err < tol, f"relative error {err:.2e} (bound {tol:.0e})"


def meta(entries):
    """entries [(slot, n, start)] -> row_ent, ent, tiles as a step builds them."""
    row_ent, ent, tiles, r = [], [], [], 0
    for i, (slot, n, start) in enumerate(entries):
        ent += [slot, r, n, start]
        row_ent += [i] * n
        tiles += [x for q0 in range(0, n, 64) for x in (i, q0)]
        r += n
    return tuple(torch.tensor(v, dtype=torch.int32, device=DEV) for v in (row_ent, ent, tiles))


def rand_map(d, alpha):
    return torch.randn(d) * 0.5 + 1.0, torch.randn(d) * 0.3, alpha


def on_dev(m):
    return m[0].to(DEV), m[1].to(DEV), m[2]


def route_buffers(rows, n, top, sg=True):
    """Outputs of the router, full of garbage."""
    f = lambda *s: torch.full(s, 77.0, device=DEV)  # noqa: E731
    return dict(wts=f(rows, n), idw=f(rows), sel_idx=torch.full((rows, top), -5, dtype=torch.int32, device=DEV), sel_w=f(rows, top),
                n_real=n, top=top, renorm=False, score="sigmoid", **(dict(sg=f(rows)) if sg else {}))


# ---------------------------------------------------------------------------------------------------- maps and residual
@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows,d", [(1, 48), (5, 45), (3, 4100), (64, 256), (65, 256), (130, 1028), (203, 33)])
@pytest.mark.parametrize("opts", ["open", "close", "close_add", "close_next", "close_add_next", "add_next"])
def test_close_against_reference(dt, rows, d, opts):
    from dli_b200 import ops

    torch.manual_seed(rows + d)
    x, y, add = torch.randn(rows, d), (2 * torch.randn(rows, d)).to(dt), torch.randn(rows, d)
    post, nxt = rand_map(d, 0.8), rand_map(d, 0.45)
    has_y, has_add, has_n = "close" in opts, "add" in opts, opts == "open" or "next" in opts
    xd = x.to(DEV)
    out_f = torch.full((rows, d), 9.0, device=DEV)
    out_e = torch.full((rows, d), 9.0, dtype=dt, device=DEV)
    ops.dyn_tanh_close(xd, y.to(DEV) if has_y else None, on_dev(post) if has_y else None, 0.3, add.to(DEV) if has_add else None,
                       nxt=on_dev(nxt) if has_n else None, out_f=out_f if has_n else None, out_e=out_e if has_n else None)
    ref = x.double()
    if has_y:
        ref = ref + 0.3 * R.dyn_tanh(y.double(), 0.8, post[0], post[1])
    if has_add:
        ref = ref + add.double()
    close(xd, ref, 1e-6)
    if has_n:
        h = R.dyn_tanh(ref, 0.45, nxt[0], nxt[1])
        close(out_f, h, 1e-6)
        close(out_e, h, 1e-6 if dt == torch.float32 else 0.004)
    else:
        assert torch.all(out_f == 9.0) and torch.all(out_e == 9.0)


@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows,d,n,top,sg", [(1, 48, 6, 2, True), (9, 45, 5, 5, False), (64, 128, 17, 3, True), (66, 128, 16, 1, True), (129, 30, 1, 1, True),
                                             (131, 256, 40, 4, True), (70, 64, 33, 2, False), (67, 6400, 9, 2, True)])
def test_close_with_the_router_against_reference(dt, rows, d, n, top, sg):
    """One row per CTA (few rows, or rows too long for four), or four with a ragged last group; the shared expert's gate is one
    more row of the router."""
    from dli_b200 import ops

    torch.manual_seed(n)
    x, y, post, nxt = torch.randn(rows, d), torch.randn(rows, d).to(dt), rand_map(d, 0.8), rand_map(d, 0.6)
    w, sw = torch.randn(n, d) * (2.0 / d ** 0.5), torch.randn(d) * (2.0 / d ** 0.5)
    ref = x.double() + 1.3 * R.dyn_tanh(y.double(), 0.8, post[0], post[1])
    h = R.dyn_tanh(ref, 0.6, nxt[0], nxt[1])
    idx, wt = R.route(h, w, top)
    z = R.lin(h, w).sort(-1, descending=True).values
    sure = (z[:, top - 1] - z[:, top] > 1e-4) if top < n else torch.ones(rows, dtype=torch.bool)   # not a close call
    dense = torch.zeros(rows, n, dtype=F64).scatter_(1, idx, wt)
    outs = []
    for alone in (False, True):
        xd, he = x.to(DEV), torch.empty(rows, d, dtype=dt, device=DEV)
        r = dict(route_buffers(rows, n, top, sg), w_router=w.to(DEV), correction=None, **(dict(sg_w=sw.to(DEV)) if sg else {}))
        if alone:      # the router by itself on the rows of the closing kernel
            hf = torch.empty(rows, d, device=DEV)
            ops.dyn_tanh_close(xd, y.to(DEV), on_dev(post), 1.3, nxt=on_dev(nxt), out_f=hf, out_e=he)
            ops.moe_route(hf, **r)
        else:
            ops.dyn_tanh_close(xd, y.to(DEV), on_dev(post), 1.3, nxt=on_dev(nxt), out_e=he, route=r)
        close(xd, ref, 1e-6)
        close(he, h, 1e-6 if dt == torch.float32 else 0.004)
        assert sure.double().mean() > 0.9
        close(r["wts"][sure.to(DEV)], dense[sure], 1e-5)
        got = torch.zeros(rows, n, dtype=F64).scatter_(1, r["sel_idx"].cpu().long(), r["sel_w"].double().cpu())
        close(got[sure], dense[sure], 1e-5)
        assert torch.all(r["idw"] == 0)
        if sg:
            close(r["sg"], torch.sigmoid(R.lin(h, sw[None]))[:, 0], 1e-5)
        outs.append(r)
    assert torch.equal(outs[0]["sel_idx"].cpu()[sure], outs[1]["sel_idx"].cpu()[sure])


@pytest.mark.parametrize("rows", [3, 80])
def test_router_orders_by_logit_where_sigmoids_are_equal_in_fp32(rows):
    """Logits of 30, 40 and 35: all three scores round to 1; the largest logits are still the ones chosen.  With a correction the
    choice follows score + correction."""
    from dli_b200 import ops

    h = torch.zeros(rows, 4, device=DEV)
    h[:, 0] = 1.0
    w = torch.zeros(4, 4, device=DEV)
    w[:, 0] = torch.tensor([30.0, 40.0, -2.0, 35.0])
    r = route_buffers(rows, 4, 2, sg=False)
    ops.moe_route(h, w, None, **r)
    assert torch.all(r["sel_idx"] == torch.tensor([1, 3], dtype=torch.int32, device=DEV)) and torch.all(r["sel_w"] == 1.0)
    r = route_buffers(rows, 4, 2, sg=False)
    ops.moe_route(h, w, torch.tensor([0.0, 0.5, 2.0, 0.25], device=DEV), **r)
    assert torch.all(r["sel_idx"] == torch.tensor([2, 1], dtype=torch.int32, device=DEV))
    close(r["sel_w"][:, 0], torch.full((rows,), 1 / (1 + math.exp(2.0)), dtype=F64), 1e-5)


def test_router_groups_and_scale_with_sigmoid_scores():
    """Options of the router that another design may combine: groups of outputs, renormalisation and a factor."""
    from dli_b200 import ops

    torch.manual_seed(2)
    h, w = torch.randn(20, 16), torch.randn(6, 16)
    r = route_buffers(20, 6, 2, sg=False)
    r.update(renorm=True, groups=3, keep=1, wscale=2.5)
    ops.moe_route(h.to(DEV), w.to(DEV), None, **r)
    s = torch.sigmoid(h.double() @ w.double().T)
    for t in range(20):
        g = int(torch.stack([s[t, :2].max(), s[t, 2:4].max(), s[t, 4:].max()]).argmax())
        order = sorted((2 * g, 2 * g + 1), key=lambda e: -float(s[t, e]))
        assert r["sel_idx"][t].tolist() == order
        close(r["sel_w"][t], 2.5 * s[t, order] / s[t, order].sum(), 1e-5)


# ---------------------------------------------------------------------------------------------------- experts
def experts_case(n, ff, ff_s, d, dt, std=0.2):
    torch.manual_seed(n * ff)
    mk = lambda *s: (std * torch.randn(*s)).to(dt)  # noqa: E731
    gate, up, down = [mk(ff, d) for _ in range(n)], [mk(ff, d) for _ in range(n)], [mk(d, ff) for _ in range(n)]
    sh = (mk(ff_s, d), mk(ff_s, d), mk(d, ff_s)) if ff_s else None
    blocks = [x for g, u in zip(gate, up) for x in (g, u)] + ([sh[0], sh[1]] if ff_s else [])
    return gate, up, down, sh, torch.cat(blocks).contiguous().to(DEV), torch.cat(down + ([sh[2]] if ff_s else []), dim=1).contiguous().to(DEV)


@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows,d,n,top,ff,ff_s", [(1, 64, 6, 2, 16, 24), (7, 48, 3, 3, 12, 20), (90, 64, 8, 1, 32, 0), (70, 64, 5, 2, 9, 11)])
def test_experts_with_weighted_inputs_and_a_gated_shared_expert(dt, rows, d, n, top, ff, ff_s):
    """All experts' projections at once and (bf16) the chosen experts only; weights of 0.05 to 0.95 go through the activation."""
    from dli_b200 import ops

    gate, up, down, sh, w_gu, w_down = experts_case(n, ff, ff_s, d, dt)
    h = torch.randn(rows, d).to(dt)
    idx = torch.stack([torch.randperm(n)[:top] for _ in range(rows)])
    wt = 0.05 + 0.9 * torch.rand(rows, top)
    sg = torch.rand(rows)
    dense = torch.zeros(rows, n).scatter_(1, idx, wt)
    ref = torch.zeros(rows, d, dtype=F64)
    one = lambda v, g, u, dn: R.lin(R.silu(R.lin(v, g)) * R.lin(v, u), dn)  # noqa: E731
    for t in range(rows):
        for e, w in zip(idx[t].tolist(), wt[t].tolist()):
            ref[t] += one(w * h[t:t + 1].double(), gate[e], up[e], down[e])[0]
        if ff_s:
            ref[t] += float(sg[t]) * one(h[t:t + 1].double(), *sh)[0]
    tol = 1e-5 if dt == torch.float32 else 0.03
    hd, sgd = h.to(DEV), sg.to(DEV) if ff_s else None
    gu = torch.empty(rows, w_gu.shape[0], dtype=dt, device=DEV)
    ops.linear_any(hd, w_gu, gu)
    act = torch.full((rows, n * ff + ff_s), 5.0, dtype=dt, device=DEV)
    ops.moe_act(gu, dense.to(DEV), act, n, ff, 0.0, ff_s, silu=True, weight_in=True, sg=sgd)
    y = torch.empty(rows, d, dtype=dt, device=DEV)
    ops.linear_any(act, w_down, y)
    close(y, ref, tol)
    if dt == torch.bfloat16 and rows < 10 and ops.moe_sel_supported(d, ff, ff_s, top):
        act = torch.full((rows, top * ff + ff_s), 5.0, dtype=dt, device=DEV)
        y2 = torch.empty_like(y)
        ops.moe_sel(hd, w_gu, w_down, idx.to(torch.int32).to(DEV), wt.to(DEV), act, y2, n, top, ff, 0.0, ff_s, silu=True, weight_in=True, sg=sgd)
        close(y2, ref, tol)


@pytest.mark.parametrize("form", ["clamped", "relu2"])
@pytest.mark.parametrize("ff,ff_s", [(8, 16), (9, 5)])
def test_weighted_inputs_of_the_other_expert_activations(form, ff, ff_s):
    from dli_b200 import ops

    torch.manual_seed(3)
    rows, n = 11, 4
    gated = form == "clamped"
    gu = 3 * torch.randn(rows, (2 if gated else 1) * (n * ff + ff_s))
    wts, sg = torch.rand(rows, n) * (torch.rand(rows, n) > 0.5), torch.rand(rows)
    ref = torch.zeros(rows, n * ff + ff_s, dtype=F64)
    for e in range(n + 1):
        f, at = (ff, e * ff) if e < n else (ff_s, n * ff)
        w = wts[:, e:e + 1].double() if e < n else torch.ones(rows, 1, dtype=F64)
        wo = 1.0 if e < n else sg[:, None].double()
        if gated:
            g, u = gu[:, 2 * at:2 * at + f].double() * w, gu[:, 2 * at + f:2 * at + 2 * f].double() * w
            g, u = g.clamp(max=2.0), u.clamp(-2.0, 2.0)
            v = g * torch.sigmoid(1.702 * g) * (u + 1.0) * (w != 0)
        else:
            v = (gu[:, at:at + f].double() * w).clamp(min=0) ** 2
        ref[:, at:at + f] = v * wo
    act = torch.full((rows, n * ff + ff_s), 5.0, device=DEV)
    ops.moe_act(gu.to(DEV), wts.to(DEV), act, n, ff, 2.0, ff_s, 2.0, gated=gated, weight_in=True, sg=sg.to(DEV))
    close(act, ref, 1e-5)


# ---------------------------------------------------------------------------------------------------- attention
def attention_case(T, H, G, D, V, size, rot, dt, cuts, scale=None, page=4, plant=None, kernel="auto", sink=None, norm=True):
    """One sequence through prep and attention in portions `cuts`, its pages in reverse order in a pool full of garbage; returns
    (got [T, H*V], ref, heads' outputs before the gate)."""
    from dli_b200 import ops
    from dli_b200.ragged_engine import rot_frequencies, rot_gain

    torch.manual_seed(7)
    scale = scale or D ** -0.5
    q, k, v, g = torch.randn(T, H, D) * torch.linspace(0.2, 3.0, H)[None, :, None], torch.randn(T, G, D), torch.randn(T, G, V), torch.randn(T, H)
    qn, kn = torch.rand(H * D) + 0.5, torch.rand(G * D) + 0.5
    sink = torch.randn(H) if sink is None else sink
    if plant:
        plant(q, k, v)
    proj = torch.cat((q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1), g), dim=1).to(dt).contiguous()
    qo, ko, vo, go = 0, H * D, (H + G) * D, (H + G) * D + G * V
    rd, sc = (int(rot["dims"]), rot.get("scaling")) if rot else (0, None)
    cos_t = sin_t = None
    if rd:
        ang = torch.arange(T, dtype=F64)[:, None] * rot_frequencies(float(rot["base"]), rd, sc)[None, :]
        cos_t, sin_t = ((rot_gain(sc) * f).float().to(DEV) for f in (ang.cos(), ang.sin()))
    pages = (T + page - 1) // page
    kc = torch.full((pages + 3, G, page, D), 99.0, dtype=dt, device=DEV)
    vc = torch.full((pages + 3, G, page, V), -99.0, dtype=dt, device=DEV)
    pt = torch.zeros(3, pages, dtype=torch.int32)
    pt[1] = torch.arange(pages - 1, -1, -1)
    pt = pt.to(DEV)
    out = torch.empty(T, H * V, dtype=dt, device=DEV)
    at = 0
    for n in cuts:
        row_ent, ent, tiles = meta([(1, n, at)])
        pr = proj[at:at + n].contiguous().to(DEV)
        qbuf = torch.full((n, H * D), 1e4, device=DEV)
        ops.attn_prep_append(pr, qbuf, kc, vc, row_ent, ent, pt, H, G, D, V, rd, qo, ko, vo, qn.to(DEV) if norm else None, kn.to(DEV) if norm else None,
                             1e-5, cos_t, sin_t, None, None, halves=True, whole_norm=norm)
        kw = dict(window=size, sink=sink.to(DEV), g_off=go)
        o = torch.empty(n, H * V, dtype=dt, device=DEV)
        if kernel == "tc" or (kernel == "auto" and n >= 16 and ops.attn_ragged_tc_supported(D, V, dt)):
            ops.attn_ragged_tc(qbuf, kc, vc, pr, o, ent, tiles, pt, H, G, D, V, scale, **kw)
        else:
            splits = 3 if n <= 2 else 1
            part = torch.empty(n * H * splits * (V + 2), device=DEV) if splits > 1 else None
            ops.attn_ragged(qbuf, kc, vc, pr, o, row_ent, ent, pt, H, G, D, V, scale, splits=splits, part=part, **kw)
        out[at:at + n] = o
        at += n
    p = proj.double()
    qr, kr = p[:, :ko], p[:, ko:vo]
    if norm:
        qr, kr = R.rms_norm(qr, qn, 1e-5), R.rms_norm(kr, kn, 1e-5)
    heads = R.windowed_attention(R.rotate(qr.reshape(T, H, D), rot), R.rotate(kr.reshape(T, G, D), rot), p[:, vo:go].reshape(T, G, V), scale, size, sink)
    return out, (heads * torch.sigmoid(p[:, go:])[:, :, None]).reshape(T, H * V), heads


SC = {"factor": 6.0, "original": 96, "fast": 6.0, "slow": 1.5}


@pytest.mark.parametrize("T,H,G,D,V,size,rd,sc,dt,cuts", [
    (60, 4, 2, 8, 6, 9, 4, SC, torch.float32, [60]), (60, 4, 2, 8, 6, 9, 8, SC, torch.float32, [7, 2, 1, 1, 1, 30, 18]),
    (40, 3, 1, 10, 4, 1, 2, None, torch.float32, [20, 1, 19]), (40, 2, 2, 6, 14, 0, 6, None, torch.float32, [1] * 3 + [37]),
    (40, 5, 5, 6, 2, 33, 0, None, torch.bfloat16, [30, 2, 8]), (200, 4, 2, 64, 64, 70, 32, SC, torch.bfloat16, [200]),
    (200, 6, 2, 128, 64, 33, 20, SC, torch.bfloat16, [66, 1, 1, 64, 3, 65]), (130, 2, 1, 64, 128, 0, 64, None, torch.bfloat16, [130]),
    (150, 2, 2, 40, 32, 64, 16, SC, torch.bfloat16, [17, 133]), (150, 3, 1, 72, 136, 50, 24, SC, torch.bfloat16, [17, 1, 132]),
    (150, 2, 1, 48, 120, 20, 48, None, torch.bfloat16, [150]), (150, 2, 2, 104, 88, 0, 8, SC, torch.bfloat16, [70, 80]),
    (90, 4, 1, 32, 256, 65, 32, None, torch.bfloat16, [90])])
def test_attention_with_norms_over_whole_projections(T, H, G, D, V, size, rd, sc, dt, cuts):
    """Heads of very different size: a norm per head would change the scores' proportions.  bf16 portions run on the
    tensor-core tiles, also where the head sizes lie between the tiles'."""
    rot = {"base": 700.0, "dims": rd, "scaling": sc} if rd else None
    out, ref, _ = attention_case(T, H, G, D, V, size, rot, dt, cuts)
    close(out, ref, 1e-5 if dt == torch.float32 else 0.02)


@pytest.mark.parametrize("H,G,D,n", [(3, 1, 10, 1), (8, 2, 64, 1), (8, 8, 64, 3), (4, 2, 128, 70), (5, 5, 6, 9)])
@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
def test_norm_over_the_whole_projection_alone(H, G, D, n, dt):
    """Queries and cached keys as they leave the prep kernel; with biases; queries only; columns that start anywhere."""
    from dli_b200 import ops

    torch.manual_seed(D)
    V, pad = 4, 6
    cols = pad + (H + G) * D + G * V
    proj = torch.randn(n, cols).to(dt)
    qn, kn, bias = torch.rand(H * D) + 0.5, torch.rand(G * D) + 0.5, torch.randn(cols)
    row_ent, ent, _ = meta([(0, n, 0)])
    pt = torch.arange((n + 3) // 4, dtype=torch.int32, device=DEV)[None].contiguous()
    for with_bias in (False, True):
        for q_only in (False, True):
            kc, vc = torch.zeros(pt.numel(), G, 4, D, dtype=dt, device=DEV), torch.zeros(pt.numel(), G, 4, V, dtype=dt, device=DEV)
            qbuf = torch.zeros(n, H * D, device=DEV)
            ops.attn_prep_append(proj.to(DEV), qbuf, kc, vc, row_ent, ent, pt, H, G, D, V, 0, pad, pad + H * D, pad + (H + G) * D, qn.to(DEV),
                                 kn.to(DEV), 1e-5, None, None, None, None, bias=bias.to(DEV) if with_bias else None, q_only=q_only, whole_norm=True)
            p = proj.double() + (bias.double() if with_bias else 0.0)
            close(qbuf, R.rms_norm(p[:, pad:pad + H * D], qn, 1e-5), 1e-6)
            got = kc.permute(0, 2, 1, 3).reshape(-1, G * D)[:n]
            if q_only:
                assert torch.all(got == 0)
            else:
                close(got, R.rms_norm(p[:, pad + H * D:pad + (H + G) * D], kn, 1e-5), 1e-6 if dt == torch.float32 else 0.004)


@pytest.mark.parametrize("dt,D,V", [(torch.float32, 8, 6), (torch.bfloat16, 64, 64), (torch.bfloat16, 56, 40)])
@pytest.mark.parametrize("at,size", [(10, 21), (63, 65), (64, 64), (15, 1), (3, 80)])
def test_a_planted_key_counts_exactly_inside_the_window(dt, D, V, at, size):
    """Every query scores 8 on the key at `at` and 0 elsewhere: up to position at + size - 1 the output is mostly that value, and
    from at + size on it is gone."""
    T = 150

    def plant(q, k, v):
        q.zero_()
        k[..., -1] = 0.0
        q[..., -1] = 8.0                        # a dimension that is not rotated
        k[at, :, -1] = 1.0
        v[..., 0] = 0.0
        v[at, :, 0] = 50.0

    for kernel in ("auto", "rows"):
        for cuts in ([T], [at + size - 1, 2, T - at - size - 1], [at + size, 1, T - at - size - 1]):
            out, ref, heads = attention_case(T, 2, 2, D, V, size, {"base": 700.0, "dims": 2}, dt, cuts, scale=1.0, plant=plant, kernel=kernel,
                                             sink=torch.zeros(2), norm=False)
            close(out, ref, 1e-5 if dt == torch.float32 else 0.02)
    last = at + size - 1
    assert heads[at:last + 1, :, 0].min() > 45.0 and heads[last + 1:, :, 0].abs().max() < 1e-9


@pytest.mark.parametrize("dt,D,V", [(torch.float32, 8, 6), (torch.bfloat16, 64, 64), (torch.bfloat16, 40, 56)])
def test_the_sink_takes_its_share_and_is_not_scaled(dt, D, V):
    """Equal scores of 0 and sinks of ln 2 and -1: position t averages its keys over their number plus exp(sink)."""
    sink = torch.tensor([math.log(2.0), -1.0])

    def plant(q, k, v):
        q.zero_()
        v[:] = 1.0

    for cuts in ([40], [1] * 5 + [35]):
        out, ref, heads = attention_case(40, 2, 1, D, V, 17, None, dt, cuts, scale=0.125, plant=plant, sink=sink, norm=False)
        n = torch.tensor([min(t + 1, 17) for t in range(40)], dtype=F64)
        assert torch.allclose(heads[:, 0, 0], n / (n + 2), atol=1e-6) and torch.allclose(heads[:, 1, 0], n / (n + math.exp(-1.0)), atol=1e-6)
        close(out, ref, 1e-5 if dt == torch.float32 else 0.01)


# ---------------------------------------------------------------------------------------------------- latent attention
@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,K", [(4, 16), (2, 32), (3, 32), (4, 40), (6, 128), (4, 512)])
@pytest.mark.parametrize("T,size,sp", [(70, 9, 3), (150, 64, 1), (150, 1, 2), (300, 200, 7), (40, 0, 5), (300, 129, 1)])
def test_windowed_attention_over_one_shared_key_value_row(dt, H, K, T, size, sp):
    """The cached latents as keys and values of all heads (two or four heads per CTA, or one where the head count or the size
    allows no more), with and without key splits; the last position scores one key just inside its window highest."""
    from dli_b200 import ops

    torch.manual_seed(K + T)
    page = 8
    pages = (T + page - 1) // page
    c = torch.randn(T, K).to(dt)
    q = torch.randn(3, H, K) * K ** -0.5
    ins = max(T - size, 0) if size else 0                       # oldest visible key of the last position
    q[2] = c[ins].float() * (8.0 / float(c[ins].float().pow(2).sum()))
    pool = torch.full((pages + 1, 1, page, K), 60.0, dtype=dt)
    flat = pool[torch.arange(pages - 1, -1, -1)].reshape(-1, K)
    flat[:T] = c
    pool[torch.arange(pages - 1, -1, -1)] = flat.reshape(pages, 1, page, K)
    pt = torch.zeros(2, pages, dtype=torch.int32)
    pt[1] = torch.arange(pages - 1, -1, -1)
    row_ent, ent, _ = meta([(1, 3, T - 3)])
    out = torch.empty(3, H * K, dtype=dt, device=DEV)
    part = torch.full((3 * H * sp * (K + 2),), 1e9, device=DEV)
    p = pool.to(DEV)
    ops.attn_ragged(q.reshape(3, H * K).to(DEV), p, p, None, out, row_ent, ent, pt.to(DEV), H, 1, K, K, 1.0, ldv=K, splits=sp,
                    part=part if sp > 1 else None, window=size)
    qf = torch.zeros(T, H, K, dtype=F64)
    qf[T - 3:] = q.double()
    ref = R.windowed_attention(qf, c.double()[:, None], c.double()[:, None], 1.0, size)[T - 3:].reshape(3, H * K)
    close(out, ref, 1e-5 if dt == torch.float32 else 0.01)


@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows,H,V,K", [(1, 3, 10, 12), (9, 4, 64, 128), (20, 2, 6, 520), (70, 5, 24, 64)])
@pytest.mark.parametrize("per_head", [True, False])
def test_value_up_projection_with_a_gate_per_head_or_channel(dt, rows, H, V, K, per_head):
    from dli_b200 import ops

    torch.manual_seed(rows)
    o, uv, n_g = torch.randn(rows, H * K).to(dt), (torch.randn(H * V, K) * K ** -0.5).to(dt), H if per_head else H * V
    proj = torch.randn(rows, n_g + 8).to(dt)
    out = torch.empty(rows, H * V, dtype=dt, device=DEV)
    ops.latent_v_up(o.to(DEV), uv.to(DEV), proj.to(DEV), out, H, V, K, g_off=5, g_head=per_head)
    u = torch.einsum("rhk,hvk->rhv", o.double().reshape(rows, H, K), uv.double().reshape(H, V, K))
    z = torch.sigmoid(proj.double()[:, 5:5 + n_g])
    ref = u * (z[:, :, None] if per_head else z.reshape(rows, H, V))
    close(out, ref.reshape(rows, H * V), 1e-5 if dt == torch.float32 else 0.006)
