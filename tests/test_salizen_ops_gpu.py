"""The mechanisms of the Salizen design one at a time, kernels against the plain float64 oracle (oracle/salizen_ref.py):
the embedding with hashed token pairs, the closing kernel of layers with several residual streams (with the router),
linear attention in its three forms (row by row, blocks in order, tiles in parallel; CUDA cores and tensor cores) with
fixed and input-made decays, the norm and gate of its outputs, attention with keys as values, half-split rotation, a
soft cap, a sink and a gate per channel, the router with a bias, gated SiLU experts and the GELU gate.  Slots and caches
hold garbage before use."""
import math

import pytest
import torch

pytestmark = pytest.mark.gpu

from oracle import salizen_ref as R  # noqa: E402

DEV = "cuda:0"
F64 = torch.float64
DTS = [torch.float32, torch.bfloat16]


def meta(entries):
    """entries [(slot, rows, first position)] -> row_ent, ent, 64-row tiles on the device."""
    row_ent, ent, tiles, at = [], [], [], 0
    for i, (slot, n, pos) in enumerate(entries):
        row_ent += [i] * n
        ent += [slot, at, n, pos]
        for q0 in range(0, n, 64):
            tiles += [i, q0]
        at += n
    return tuple(torch.tensor(t, dtype=torch.int32, device=DEV) for t in (row_ent, ent, tiles))


def close(got, ref, tol):
    ref = ref.double()
    err = (got.double().cpu() - ref).abs().max()
    assert err < tol * max(1e-6, float(ref.abs().max())), float(err)


# ---------------------------------------------------------------------------------------------------- embedding
@pytest.mark.parametrize("width", [48, 30, 7])
@pytest.mark.parametrize("dt", DTS)
@pytest.mark.parametrize("hash_", [(11, 31, 7), (1, 5, 3), (1009, 4000000007, 2147483647)])
def test_embedding_with_token_pairs(width, dt, hash_):
    """A sequence's start, a portion in the middle and a single token (previous token from the slot), 3 streams; the slots'
    last tokens move on, the others' stay."""
    from dli_b200 import ops

    torch.manual_seed(0)
    n, mp, mc = hash_
    sd = {"embed": torch.randn(50, width).to(dt), "bigram": torch.randn(n + 1, width).to(dt)}
    cfg = {"embedding": {"scale": 2.5, "bigram": {"buckets": n, "mul_prev": mp, "mul_cur": mc}}}
    seqs = {2: torch.randint(0, 50, (4,)).tolist(), 0: torch.randint(0, 50, (9,)).tolist(), 3: torch.randint(0, 50, (6,)).tolist()}
    last = torch.full((5,), 10 ** 6, dtype=torch.int32, device=DEV)
    last[0], last[3] = seqs[0][3], seqs[3][4]
    entries, parts = [(2, 4, 0), (0, 5, 4), (3, 1, 5)], [seqs[2], seqs[0][4:], seqs[3][5:]]
    row_ent, ent, _ = meta(entries)
    ids = torch.tensor(sum(parts, []), dtype=torch.int32, device=DEV)
    x = torch.full((3, 12, width), 7.0, device=DEV)
    ops.embedding_f32(ids, sd["embed"].to(DEV), x, 2.5, row_ent=row_ent, ent=ent, bigram=sd["bigram"].to(DEV), mul_prev=mp, mul_cur=mc, last=last)
    ref = torch.cat([R.embed(cfg, sd, seqs[2]), R.embed(cfg, sd, seqs[0])[4:], R.embed(cfg, sd, seqs[3])[5:]])
    for s in range(3):
        close(x[s, :10], ref, 1e-6)
    assert torch.all(x[:, 10:] == 7.0)
    assert last.tolist() == [seqs[0][8], 10 ** 6, seqs[2][3], seqs[3][5], 10 ** 6]


# ---------------------------------------------------------------------------------------------------- several streams
@pytest.mark.parametrize("dt", DTS)
@pytest.mark.parametrize("S,rows,width", [(1, 5, 48), (2, 70, 40), (3, 4, 33), (4, 3, 2048), (8, 2, 24)])
def test_streams_close_against_reference(dt, S, rows, width):
    from dli_b200 import ops

    torch.manual_seed(1)
    cap = rows + 3
    x, y = torch.randn(S, cap, width), torch.randn(rows, width).to(dt)
    mix, out, inn, w = torch.randn(S, S), torch.randn(S), torch.randn(S), torch.rand(width) + 0.5
    xd = x.clone().to(DEV)
    of, oe = torch.empty(rows, width, device=DEV), torch.empty(rows, width, dtype=dt, device=DEV)
    g = lambda t: t.to(DEV)  # noqa: E731
    ops.streams_close(xd, rows, g(y), g(mix), g(out), g(inn), g(w), out_f=of, out_e=oe, eps=1e-5)
    xs = [x[s, :rows].double() for s in range(S)]
    new = R.streams_write(xs, mix, out, y.double())
    for s in range(S):
        close(xd[s, :rows], new[s], 2e-6)
    assert torch.equal(xd[:, rows:].cpu(), x[:, rows:])          # rows behind the step's are left alone
    h = R.rms_norm(R.streams_read(new, inn), w, 1e-5)
    close(of, h, 2e-5)
    close(oe, h, 2e-5 if dt == torch.float32 else 1e-2)
    # the sum of the streams for a model's last norm; reading only (no result) leaves the streams alone
    before = xd.clone()
    ops.streams_close(xd, rows, w_next=g(w), out_f=of, eps=1e-5)
    assert torch.equal(before, xd)
    close(of, R.rms_norm(sum(new), w, 1e-5), 2e-5)
    # writing only
    ops.streams_close(xd, rows, g(y), g(mix), g(out))
    close(xd[S - 1, :rows], R.streams_write(new, mix, out, y.double())[S - 1], 4e-6)


def test_the_mix_is_indexed_from_to():
    from dli_b200 import ops

    x = torch.zeros(2, 1, 4, device=DEV)
    x[0] = 1.0
    y = torch.zeros(1, 4, device=DEV)
    ops.streams_close(x, 1, y, torch.tensor([[0.0, 5.0], [9.0, 0.0]], device=DEV), torch.zeros(2, device=DEV))
    assert x[0].abs().max() == 0 and torch.all(x[1] == 5.0)


# ---------------------------------------------------------------------------------------------------- router, experts, gate
@pytest.mark.parametrize("rows,width,n,top", [(5, 48, 6, 2), (70, 40, 13, 4), (3, 33, 4, 4), (2, 64, 1, 1), (9, 24, 40, 7)])
def test_router_with_bias_weights_are_the_softmax_over_the_chosen(rows, width, n, top):
    """Through the closing kernel and through the router alone; the bias decides some choices (and counts in the weights)."""
    from dli_b200 import ops

    torch.manual_seed(2)
    S = 2
    x, w = torch.randn(S, rows, width), torch.rand(width) + 0.5
    wr, b = torch.randn(n, width) * 0.3, torch.randn(n) * 2
    y, mix, out, inn = torch.randn(rows, width), torch.randn(S, S), torch.randn(S), torch.rand(S)
    new = R.streams_write([x[s].double() for s in range(S)], mix, out, y.double())
    h = R.rms_norm(R.streams_read(new, inn), w, 1e-5)
    idx, wt = R.route(h, wr, b, top)
    g = lambda t: t.to(DEV)  # noqa: E731

    def outputs():
        return dict(wts=torch.full((rows, n), 9.0, device=DEV), idw=torch.empty(rows, device=DEV),
                    sel_idx=torch.empty(rows, top, dtype=torch.int32, device=DEV), sel_w=torch.empty(rows, top, device=DEV))

    args = dict(w_router=g(wr), correction=None, logit_bias=g(b), n_real=n, top=top)
    a = dict(args, **outputs())
    ops.streams_close(g(x), rows, g(y), g(mix), g(out), g(inn), g(w), out_e=torch.empty(rows, width, device=DEV), eps=1e-5, route=a)
    c = dict(args, **outputs())
    ops.moe_route(h.float().to(DEV), **c)
    dense = torch.zeros(rows, n, dtype=F64)
    dense.scatter_(1, idx, wt)
    for r in (a, c):
        assert r["sel_idx"].cpu().tolist() == idx.tolist()
        close(r["sel_w"], wt, 2e-5)
        close(r["wts"], dense, 2e-5)


@pytest.mark.parametrize("dt", DTS)
@pytest.mark.parametrize("rows,width,n,top,ff", [(5, 48, 6, 2, 12), (2, 64, 5, 3, 16), (70, 64, 4, 1, 24), (3, 40, 3, 3, 7)])
def test_gated_silu_experts(dt, rows, width, n, top, ff):
    from dli_b200 import ops

    torch.manual_seed(3)
    h = torch.randn(rows, width).to(dt)
    sd = {"router": torch.randn(n, width), "router.b": torch.randn(n)}
    for k in range(n):
        sd[f"e{k}.gate"], sd[f"e{k}.up"] = (torch.randn(ff, width) * 0.3).to(dt), (torch.randn(ff, width) * 0.3).to(dt)
        sd[f"e{k}.down"] = (torch.randn(width, ff) * 0.3).to(dt)
    ref = R.moe_ff(h.double(), sd, "", {"router": {"experts": n, "top": top}})
    idx, wt = R.route(h.double(), sd["router"], sd["router.b"], top)
    dense = torch.zeros(rows, n, dtype=F64)
    dense.scatter_(1, idx, wt)
    w_gu = torch.cat([sd[f"e{k}.{p}"] for k in range(n) for p in ("gate", "up")]).to(DEV)
    w_dn = torch.cat([sd[f"e{k}.down"] for k in range(n)], dim=1).contiguous().to(DEV)
    gu = torch.empty(rows, w_gu.shape[0], dtype=dt, device=DEV)
    act = torch.empty(rows, n * ff, dtype=dt, device=DEV)
    y = torch.empty(rows, width, dtype=dt, device=DEV)
    ops.linear_any(h.to(DEV), w_gu, gu)
    ops.moe_act(gu, dense.float().to(DEV), act, n, ff, 0.0, silu=True)
    ops.linear_any(act, w_dn, y)
    close(y, ref, 1e-5 if dt == torch.float32 else 0.02)
    if dt == torch.bfloat16 and ops.moe_sel_supported(width, ff, 0, top):
        y2 = torch.empty_like(y)
        ops.moe_sel(h.to(DEV), w_gu, w_dn, idx.to(torch.int32).to(DEV), wt.float().to(DEV), torch.empty(rows, top * ff, dtype=dt, device=DEV), y2,
                    n, top, ff, 0.0, silu=True)
        close(y2, ref, 0.02)


@pytest.mark.parametrize("rows", [1, 2, 7, 64, 200])
def test_gelu_gate_as_the_projections_epilogue_and_alone(rows):
    from dli_b200 import ops

    torch.manual_seed(4)
    K, F = 128, 256
    x, wg, wu = torch.randn(rows, K), torch.randn(F, K) * 0.2, torch.randn(F, K) * 0.2
    bx, bg, bu = (t.to(torch.bfloat16) for t in (x, wg, wu))
    ref = R.gelu_tanh(R.lin(bx.double(), bg)) * R.lin(bx.double(), bu)
    scr = torch.zeros(ops.gemm_splitk_scratch_bytes(128, 2 * F), dtype=torch.uint8, device=DEV) if 2 < rows <= 128 else None
    got = ops.linear_gated_act(bx.to(DEV), ops.pack_gate_up(bg, bu).to(DEV), torch.zeros(2, device=DEV), scr)
    close(got, ref, 0.015)
    for dt, tol in ((torch.float32, 2e-6), (torch.bfloat16, 0.01)):
        for n in (24, 7):
            gu = (torch.randn(rows, 2 * n) * 3).to(dt)
            out = torch.empty(rows, n, dtype=dt, device=DEV)
            ops.silu_mul(gu.to(DEV), out, gelu=True)
            close(out, R.gelu_tanh(gu[:, :n].double()) * gu[:, n:].double(), tol)


# ---------------------------------------------------------------------------------------------------- linear attention
ENTRIES = [(2, 130, 0), (0, 1, 5), (3, 64, 70), (1, 17, 3)]     # a whole prompt, a decoded token, a full tile, a short portion
FORMS = ["rows", "blocks", "tiles"]


def linear_case(H, D, V, gated, silu, rd, dt, tau=2.0, strong=1.0, decay=None, rank=5, entries=ENTRIES):
    """Inputs, and a function that runs one form of the kernel -> (o, S)."""
    from dli_b200 import ops

    torch.manual_seed(5)
    rows = sum(n for _, n, _ in entries)
    cols = 2 * H * D + H * V + rank
    proj = torch.randn(rows, (cols + 15) // 16 * 16).to(dt)
    S0 = torch.randn(4, H, D, V)
    decay = decay or [0.02 + 0.97 * k / max(H - 1, 1) for k in range(H)]
    a2, a2b = torch.randn(H * D, rank) * strong, torch.randn(H * D)
    freqs = R.frequencies(100.0, rd, None)
    ang = torch.arange(256, dtype=F64)[:, None] * torch.tensor(freqs, dtype=F64)[None, :] if rd else None
    row_ent, ent, tiles = meta(entries)
    kw = dict(silu=silu, q_scale=0.3, k_scale=0.7, rd=rd)
    if rd:
        kw.update(cos_t=ang.cos().float().to(DEV), sin_t=ang.sin().float().to(DEV))
    if gated:
        kw.update(a_off=2 * H * D + H * V, a2=a2.to(DEV), a2_b=a2b.to(DEV), inv_tau=1.0 / tau)
    else:
        kw.update(log_decay=torch.tensor([math.log(d) if d > 0 else -1e4 for d in decay], dtype=F64).float().to(DEV))

    def run(form):
        S, o = S0.clone().to(DEV), torch.full((rows, H * V), 7.0, device=DEV)
        k = dict(kw)
        if form != "rows":
            k.update(blocked=True, lg=torch.full((rows * H * (2 * D + V),), float("nan"), device=DEV))
        if form == "tiles":
            k.update(tiles=tiles, scratch=torch.full((ops.linattn_scratch_floats(tiles.numel() // 2, H, D, V),), float("nan"), device=DEV))
        ops.linattn_ragged(proj.to(DEV), S, o, ent, H, D, V, 0, H * D, 2 * H * D, **k)
        return o, S

    p = proj.double()
    f = R.silu if silu else (lambda t: t)
    q, k, v = (f(p[:, a:b]).reshape(rows, H, -1) for a, b in ((0, H * D), (H * D, 2 * H * D), (2 * H * D, 2 * H * D + H * V)))
    w = R.fixed_decay(decay, rows, D)
    if gated:
        z = R.lin(p[:, 2 * H * D + H * V:cols], a2) + a2b.double()
        w = (torch.sigmoid(z) ** (1.0 / tau)).reshape(rows, H, D)
    o_ref, S_ref, at = [], S0.double().clone(), 0
    for slot, n, pos in entries:
        sl = slice(at, at + n)
        qq, kk = (R.rotate_halves(t[sl], freqs, pos) if rd else t[sl] for t in (q, k))
        oo, S_ref[slot] = R.matrix_recurrence(0.3 * qq, 0.7 * kk, v[sl], w[sl], S=S_ref[slot] if pos > 0 else None)
        o_ref.append(oo.reshape(n, H * V))
        at += n
    return run, torch.cat(o_ref), S_ref


@pytest.mark.parametrize("dt", DTS)
@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("H,D,V,silu,rd", [(3, 32, 64, True, 0), (2, 64, 32, False, 64), (2, 48, 72, False, 20), (1, 128, 128, True, 0),
                                           (2, 16, 8, False, 0), (1, 7, 5, True, 2), (2, 30, 6, False, 30), (1, 144, 200, False, 32)])
def test_linear_attention_fixed_decay(dt, form, H, D, V, silu, rd):
    run, o_ref, S_ref = linear_case(H, D, V, False, silu, rd, dt)
    o, S = run(form)
    tol = 3e-5 if dt == torch.bfloat16 and form == "tiles" else 4e-6      # two bf16 numbers per operand: 2^-17
    close(o, o_ref, tol)
    close(S, S_ref, tol)


@pytest.mark.parametrize("dt", DTS)
@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("H,D,V,tau,strong", [(2, 48, 64, 16.0, 1.0), (1, 128, 128, 3.0, 1.0), (2, 16, 200, 2.0, 1.0), (2, 80, 24, 1.0, 4.0),
                                              (2, 64, 16, 0.25, 8.0), (1, 20, 6, 2.0, 1.0), (1, 300, 40, 2.0, 1.0)])
def test_linear_attention_decay_per_channel(dt, form, H, D, V, tau, strong):
    """Decays from nearly 1 to far below fp32's range inside one block of 16 rows (tau 0.25, large pre-activations)."""
    run, o_ref, S_ref = linear_case(H, D, V, True, False, 0, dt, tau=tau, strong=strong)
    o, S = run(form)
    assert torch.isfinite(o).all() and torch.isfinite(S).all()
    tol = 3e-5 if dt == torch.bfloat16 and form == "tiles" else 1e-5
    close(o, o_ref, tol)
    close(S, S_ref, tol)


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("decay", [[0.0, 1.0], [1.0, 0.5], [1e-30, 0.9999]])
def test_linear_attention_decays_at_the_ends_of_their_range(form, decay):
    run, o_ref, S_ref = linear_case(2, 32, 24, False, False, 0, torch.bfloat16, decay=decay)
    o, S = run(form)
    close(o, o_ref, 3e-5)
    close(S, S_ref, 3e-5)


@pytest.mark.parametrize("dt", DTS)
def test_decay_projection_of_larger_ranks(dt):
    for rank in (1, 16, 33):
        run, o_ref, S_ref = linear_case(2, 24, 8, True, False, 0, dt, rank=rank, strong=0.5)
        for form in FORMS:
            o, S = run(form)
            close(o, o_ref, 3e-5)


@pytest.mark.parametrize("gated", [False, True])
def test_one_key_far_back_stands_out_across_tiles(gated):
    """All keys but one are zero: the row of 200 earlier positions is what every later output reads, in every form, with the
    weight of its distance."""
    from dli_b200 import ops

    H, D, V, T = 1, 16, 8, 300
    proj = torch.zeros(T, 48)
    proj[:, :D] = 1.0
    proj[37, D:2 * D] = 3.0
    proj[:, 2 * D:2 * D + V] = torch.randn(T, V)
    proj = proj.to(torch.bfloat16)
    _, ent, tiles = meta([(0, T, 0)])
    w = 0.995
    z = math.log(w / (1 - w))
    kw = dict(a_off=2 * D + V, a2=torch.zeros(D, 4, device=DEV), a2_b=torch.full((D,), z, device=DEV)) if gated else \
        dict(log_decay=torch.tensor([math.log(w)], device=DEV))
    for form in FORMS:
        S, o = torch.full((1, H, D, V), 1e4, device=DEV), torch.empty(T, V, device=DEV)
        k = dict(kw)
        if form != "rows":
            k.update(blocked=True, lg=torch.empty(T * (2 * D + V), device=DEV))
        if form == "tiles":
            k.update(tiles=tiles, scratch=torch.empty(ops.linattn_scratch_floats(tiles.numel() // 2, H, D, V), device=DEV))
        ops.linattn_ragged(proj.to(DEV), S, o, ent, H, D, V, 0, D, 2 * D, **k)
        v = proj[37, 2 * D:2 * D + V].double()
        for t in (0, 36, 37, 38, 63, 64, 127, 128, 191, 256, 299):
            ref = torch.zeros(V, dtype=F64) if t < 37 else 3.0 * D * w ** (t - 37) * v
            assert (o[t].double().cpu() - ref).abs().max() < 2e-4 * 3.0 * D, (form, t)


@pytest.mark.parametrize("dt", DTS)
@pytest.mark.parametrize("rows,H,V,together,gate,weight", [(5, 3, 10, False, 1, False), (70, 2, 64, False, 1, True), (4, 2, 8, True, 2, True),
                                                           (3, 16, 128, True, 2, True), (2, 33, 128, True, 2, True), (3, 1, 5, False, 1, True)])
def test_norm_of_the_outputs_and_gate(dt, rows, H, V, together, gate, weight):
    """Per head (with a shared weight or none) with a SiLU gate, over all heads with a sigmoid gate; into a column range of
    wider rows."""
    from dli_b200 import ops

    torch.manual_seed(6)
    n = H * V
    o, proj = torch.randn(rows, n), torch.randn(rows, n + 24).to(dt)
    h_, v_ = (1, n) if together else (H, V)
    w = torch.rand(v_) + 0.5 if weight else None
    buf = torch.full((rows, n + 8), 7.0, dtype=dt, device=DEV)
    ops.head_rmsnorm_gate(o.to(DEV), proj.to(DEV), w.to(DEV) if weight else None, buf[:, 4:4 + n], h_, v_, 1e-5, gate=gate, g_off=12)
    z = proj[:, 12:12 + n].double()
    ref = R.rms_norm(o.double().reshape(rows, h_, v_), w, 1e-5).reshape(rows, n) * (R.silu(z) if gate == 1 else torch.sigmoid(z))
    close(buf[:, 4:4 + n], ref, 1e-5 if dt == torch.float32 else 0.01)
    assert torch.all(buf[:, :4] == 7.0) and torch.all(buf[:, 4 + n:] == 7.0)


# ---------------------------------------------------------------------------------------------------- softmax attention
def attention_case(T, H, G, D, size, cap, rd, dt, cuts, scale=None, page=4, plant=None, scaling=None, kernel="auto", out_scale=0.6):
    """One sequence through prep and attention in portions `cuts`, its pages in reverse order in a pool full of garbage, beside a
    second sequence; returns (got [T, H*D], ref, heads' outputs before the gate)."""
    from dli_b200 import ops

    torch.manual_seed(7)
    scale = scale or D ** -0.5
    q, k, g = torch.randn(T, H, D), torch.randn(T, G, D), torch.randn(T, H * D)
    if plant:
        plant(q, k)
    proj = torch.cat((q.reshape(T, -1), k.reshape(T, -1), g), dim=1).to(dt).contiguous()
    freqs = R.frequencies(700.0, rd, scaling)
    ang = torch.arange(T, dtype=F64)[:, None] * torch.tensor(freqs, dtype=F64)[None, :]
    cos_t, sin_t = ang.cos().float().to(DEV), ang.sin().float().to(DEV)
    pages = (T + page - 1) // page
    kc = torch.full((pages + 3, G, page, D), 99.0, dtype=dt, device=DEV)
    vc = torch.full_like(kc, -99.0)
    pt = torch.zeros(3, pages, dtype=torch.int32)
    pt[1] = torch.arange(pages - 1, -1, -1)
    pt = pt.to(DEV)
    sink = torch.zeros(H, device=DEV)
    out = torch.empty(T, H * D, dtype=dt, device=DEV)
    at = 0
    for n in cuts:
        row_ent, ent, tiles = meta([(1, n, at)])
        pr = proj[at:at + n].contiguous().to(DEV)
        qbuf = torch.empty(n, H * D, device=DEV)
        ops.attn_prep_append(pr, qbuf, kc, vc, row_ent, ent, pt, H, G, D, D, rd, 0, H * D, H * D, None, None, 1e-5, cos_t, sin_t, None, None,
                             halves=True)
        wide = torch.full((n, H * D + 6), 7.0, dtype=dt, device=DEV)
        kw = dict(window=size, sink=sink, g_off=(H + G) * D, cap=cap, g_chan=True, out_scale=out_scale)
        if kernel == "tc" or (kernel == "auto" and n >= 16 and ops.attn_ragged_tc_supported(D, D, dt)):
            ops.attn_ragged_tc(qbuf, kc, vc, pr, wide[:, 2:2 + H * D], ent, tiles, pt, H, G, D, D, scale, **kw)
        else:
            splits = 3 if n <= 2 else 1
            part = torch.empty(n * H * splits * (D + 2), device=DEV) if splits > 1 else None
            ops.attn_ragged(qbuf, kc, vc, pr, wide[:, 2:2 + H * D], row_ent, ent, pt, H, G, D, D, scale, splits=splits, part=part, **kw)
        out[at:at + n] = wide[:, 2:2 + H * D]
        assert torch.all(wide[:, :2] == 7.0) and torch.all(wide[:, 2 + H * D:] == 7.0)
        at += n
    p = proj.double()
    qr, kr = p[:, :H * D].reshape(T, H, D), p[:, H * D:(H + G) * D].reshape(T, G, D)
    heads = R.capped_attention(R.rotate_halves(qr, freqs), R.rotate_halves(kr, freqs), kr, scale, cap, size).reshape(T, H * D)
    return out, out_scale * heads * torch.sigmoid(p[:, (H + G) * D:]), heads


@pytest.mark.parametrize("T,H,G,D,size,cap,rd,dt,cuts", [
    (60, 4, 2, 8, 9, 3.0, 4, torch.float32, [60]), (60, 4, 2, 8, 9, 3.0, 8, torch.float32, [7, 2, 1, 1, 1, 30, 18]),
    (40, 3, 1, 10, 1, 0.5, 2, torch.float32, [20, 1, 19]), (40, 2, 2, 6, 0, 0.0, 6, torch.float32, [1] * 3 + [37]),
    (40, 2, 2, 6, 64, 20.0, 0, torch.bfloat16, [30, 2, 8]), (200, 4, 2, 64, 70, 4.0, 32, torch.bfloat16, [200]),
    (200, 6, 2, 128, 33, 15.0, 20, torch.bfloat16, [66, 1, 1, 64, 3, 65]), (130, 2, 1, 64, 0, 1.0, 64, torch.bfloat16, [130]),
    (150, 2, 2, 128, 64, 0.0, 128, torch.bfloat16, [17, 133])])
def test_attention_with_keys_as_values(T, H, G, D, size, cap, rd, dt, cuts):
    out, ref, _ = attention_case(T, H, G, D, size, cap, rd, dt, cuts)
    close(out, ref, 1e-5 if dt == torch.float32 else 0.02)


def test_frequency_scaling_in_all_three_ranges():
    sc = {"factor": 5.0, "low": 1.0, "high": 4.0, "original": 40}
    f, g = R.frequencies(700.0, 8, None), R.frequencies(700.0, 8, sc)
    kinds = {"kept" if b == a else ("divided" if abs(b - a / 5) < 1e-12 else "between") for a, b in zip(f, g)}
    assert kinds == {"kept", "divided", "between"}
    out, ref, _ = attention_case(60, 2, 1, 8, 0, 2.0, 8, torch.float32, [33, 1, 26], scaling=sc)
    close(out, ref, 1e-5)
    from dli_b200.ragged_engine import rot_frequencies
    assert torch.allclose(rot_frequencies(700.0, 8, sc), torch.tensor(g, dtype=F64), rtol=1e-12)


@pytest.mark.parametrize("dt,D", [(torch.float32, 8), (torch.bfloat16, 64)])
@pytest.mark.parametrize("at,size", [(10, 21), (63, 65), (64, 64), (15, 1), (3, 80)])
def test_a_planted_key_counts_exactly_inside_the_window(dt, D, at, size):
    """Every query scores the cap on the key at `at` and next to nothing elsewhere: up to position at + size - 1 the output is
    that value times e^cap / (1 + e^cap + ...), and from at + size on the value is gone."""
    T, cap = 150, 8.0

    def plant(q, k):
        q.zero_()
        k[..., -1] = 0.0
        q[..., -1] = 60.0                       # a dimension that is not rotated
        k[at, :, -1] = 60.0

    for kernel in ("auto", "rows"):
        for cuts in ([T], [at + size - 1, 2, T - at - size - 1], [at + size, 1, T - at - size - 1]):
            out, ref, heads = attention_case(T, 2, 2, D, size, cap, 2, dt, cuts, scale=0.01, plant=plant, kernel=kernel)
            close(out, ref, 1e-5 if dt == torch.float32 else 0.02)
    last = at + size - 1
    assert heads[last, D - 1] > 50.0 and heads[at:last + 1, D - 1].min() > 50.0 and heads[last + 1:, D - 1].abs().max() < 1e-9


@pytest.mark.parametrize("dt,D", [(torch.float32, 8), (torch.bfloat16, 64)])
def test_the_sink_takes_its_share_at_the_first_positions(dt, D):
    """Equal scores of 0: position t averages its t + 1 values over t + 2 terms.  Left out, the sink would double position 0."""
    def plant(q, k):
        q.zero_()
        k[:] = 1.0

    for cuts in ([40], [1] * 5 + [35]):
        out, ref, heads = attention_case(40, 2, 1, D, 0, 5.0, 0, dt, cuts, plant=plant)
        assert torch.allclose(heads[:, 0], torch.tensor([(t + 1) / (t + 2) for t in range(40)], dtype=F64))
        close(out, ref, 1e-5 if dt == torch.float32 else 0.01)


@pytest.mark.parametrize("dt,D", [(torch.float32, 8), (torch.bfloat16, 64)])
def test_large_scores_stop_at_the_cap(dt, D):
    """Scores of thousands: the weights are those of the cap (no overflow, and two keys past the cap count alike)."""
    def plant(q, k):
        q.zero_()
        k[..., -1] = 0.0
        q[..., -1] = 100.0
        k[3, :, -1], k[7, :, -1], k[11, :, -1] = 100.0, 200.0, -100.0

    for cap in (1.5, 30.0):
        for kernel in ("auto", "rows"):
            out, ref, heads = attention_case(60, 1, 1, D, 0, cap, 0, dt, [60], scale=1.0, plant=plant, kernel=kernel)
            assert torch.isfinite(out).all()
            close(out, ref, 2e-5 if dt == torch.float32 else 0.02)
