"""The Finezen design on the ragged engine against the plain float64 oracle (oracle/finezen_ref.py).

Small made-up configurations with random weights.  The float32 engine must agree with the oracle to ~1e-4 of the
logits' spread at EVERY position — a key one position off at a window's edge, a sink left out, a pass of the loop that reads
another pass's cache, an embedding added once too often or a routing weight on the wrong side of the activation changes
logits by orders of magnitude more — whatever the schedule: whole prompts, token-by-token decoding, portions down to two
tokens, mixed batches, small page pools and reused slots.  The bfloat16 engine is held to a bf16-sized bound and to
agreement between schedules.
"""
import pytest
import torch

pytestmark = pytest.mark.gpu

from oracle import finezen_ref as R  # noqa: E402

SCALING = {"factor": 3.0, "original": 64, "fast": 8.0, "slow": 1.0}   # pairs 0 / 1 / 2 of 8 dims: kept / between / slowed


def attn(heads=4, kv_heads=2, dim=8, vdim=6, size=9, scale=0.4, rot=4, base=300.0, scaling=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if size:
        m["mask"] = {"size": size}
    if rot:
        m["rot"] = {"base": base, "dims": rot}
        if scaling:
            m["rot"]["scaling"] = scaling
    return "attention", m


def latent(heads=3, dim=6, vdim=10, kv_rank=12, q_rank=20, size=14, scale=0.35):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale}
    if size:
        m["mask"] = {"size": size}
    return "latent_attention", m


def moe(experts=6, top=2, ff=12, shared=20):
    d = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        d["shared"] = {"ff": shared}
    return d


def config(layers, width=48, vocab=97, eps=1e-5, scale=2.5, mult=0.8, loop=None):
    c = {"architecture": "Finezen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
         "residual_mult": mult, "layers": [{"type": t, "mixer": m, "mlp": mlp} for (t, m), mlp in layers]}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


def cfg_a():
    """Every mechanism: both mixers with unequal windows, scaled rotation, layers with and without experts, two of the four
    layers running three times."""
    return config([(attn(scaling=SCALING, rot=8), moe()), (latent(), None), (attn(heads=3, kv_heads=1, dim=10, vdim=4, size=16, rot=6), moe(5, 3, 20, 8)),
                   (latent(heads=2, dim=4, vdim=6, kv_rank=16, q_rank=8, size=5), moe(3, 1, 8, 12))], loop=(1, 3, 3))


def cfg_b():
    """Values that often coincide taken apart, and extremes: a window of one position and none at all, every expert chosen, a
    single expert, no shared expert, one head, a key/value head per query head, the whole head rotated and none of it, a
    latent larger than the width, a loop that runs once, a residual factor of 1."""
    return config([(attn(heads=2, kv_heads=2, dim=6, vdim=8, size=1, rot=6), moe(3, 3, 8, 0)), (attn(heads=1, kv_heads=1, dim=4, vdim=12, size=0, rot=0), None),
                   (latent(heads=1, dim=8, vdim=2, kv_rank=56, q_rank=4, size=0), moe(1, 1, 16, 4)),
                   (latent(heads=5, dim=2, vdim=4, kv_rank=8, q_rank=44, size=1), None)],
                  width=40, vocab=53, scale=1.0, mult=1.0, eps=1e-3, loop=(0, 2, 1))


def cfg_c():
    """The whole stack twice, the last layer without experts."""
    return config([(latent(heads=4, dim=8, vdim=8, kv_rank=16, q_rank=12, size=7), moe(9, 2, 8, 16)), (attn(size=6, kv_heads=4), None)], width=32,
                  mult=0.5, loop=(0, 2, 2))


def build(cfg, dtype, seed=0, max_batch=4, max_seq_len=256, pool=None, page_size=4, std=0.15, sd=None):
    from dli_b200 import finezen
    from dli_b200.ragged_engine import RaggedEngine

    spec = finezen.spec_from_config(cfg)
    if sd is None:
        sd = finezen.random_state_dict(spec, seed=seed, std=std)
    eng = RaggedEngine(spec, max_batch=max_batch, max_seq_len=max_seq_len, page_size=page_size, kv_pool_tokens=pool, dtype=dtype)
    eng.load_tensors(finezen.model_tensors(spec, sd))
    return eng, sd


def prompt(n, vocab, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()


def rel_err(got, ref):
    """Per position: RMS of the logit difference (mean removed) over the RMS spread of the reference logits."""
    d = got.double().cpu() - ref
    d = d - d.mean(-1, keepdim=True)
    spread = (ref - ref.mean(-1, keepdim=True)).pow(2).mean().sqrt()
    return d.pow(2).mean(-1).sqrt() / spread


def run_schedule(eng, toks, cuts):
    """One sequence alone, cut into portions of the given sizes (the rest token by token); logits at every position."""
    slot = eng.open_sequence()
    out, at = [], 0
    sizes = list(cuts)
    while at < len(toks):
        n = min(sizes.pop(0) if sizes else 1, len(toks) - at)
        out.append(eng.step([(slot, toks[at:at + n])], [list(range(n))]).float().cpu())
        at += n
    eng.close_sequence(slot)
    return torch.cat(out)


TOL32, TOL16 = 2e-4, 0.08


def close16(err, flips=0):
    """bfloat16: nearly every position within the bf16-sized bound and none far from it.  flips: that many positions are
    left out of the second condition — where two experts' scores lie within a few thousandths of each other, bf16 rounding
    upstream decides the router's choice, and the logits of that one position move by the spread itself."""
    rest = err.flatten().sort().values[:err.numel() - flips] if flips else err
    return bool((err < TOL16).double().mean() >= 0.9 and rest.max() < 0.3)


ALL = [cfg_a, cfg_b, cfg_c]


@pytest.mark.parametrize("make", ALL)
def test_whole_prompt_float32_matches_oracle_at_every_position(make):
    cfg = make()
    eng, sd = build(cfg, torch.float32)
    toks = prompt(75, cfg["vocab"], 12)
    assert rel_err(run_schedule(eng, toks, [75]), R.forward(cfg, sd, toks)).max() < TOL32


@pytest.mark.parametrize("make", ALL)
def test_residual_stream_after_every_layer_run(make):
    """The stream as each run leaves it, before a next pass adds the embedding output; the logits of the traced steps (which
    take those two steps apart) equal the untraced ones."""
    cfg = make()
    eng, sd = build(cfg, torch.float32)
    toks = prompt(19, cfg["vocab"], 2)
    layers = []
    R.forward(cfg, sd, toks, layers)
    n = len(eng.spec.layers)
    assert n == len(layers) == len(R.layer_order(cfg))
    for cuts in ([19], []):
        plain = run_schedule(eng, toks, cuts)
        eng.layer_trace = []
        traced = run_schedule(eng, toks, cuts)
        trace, eng.layer_trace = eng.layer_trace, None
        assert rel_err(traced, plain.double()).max() < 1e-5
        assert len(trace) == n * (1 if cuts else 19)
        got = trace if cuts else [torch.cat(trace[i::n]) for i in range(n)]
        for g, ref in zip(got, layers):
            assert (g.double().cpu() - ref).abs().max() < 1e-4 * ref.abs().max()


@pytest.mark.parametrize("make", ALL)
@pytest.mark.parametrize("cuts", [[], [1, 1, 2], [2, 2, 3, 5, 7, 11], [17, 2, 16, 3], [30]])
def test_portions_and_decoding_float32(make, cuts):
    """Token by token from the first token; portions of 2..; a prompt then decoding over page borders and over the edges of
    windows of 1, 5, 6, 7, 9, 14 and 16 positions."""
    cfg = make()
    eng, sd = build(cfg, torch.float32)
    toks = prompt(52, cfg["vocab"], 3)
    assert rel_err(run_schedule(eng, toks, cuts), R.forward(cfg, sd, toks)).max() < TOL32


@pytest.mark.parametrize("make", [cfg_a, cfg_b])
def test_bfloat16_engine_is_close_and_schedules_agree(make):
    cfg = make()
    eng, sd = build(cfg, torch.bfloat16)
    toks = prompt(40, cfg["vocab"], 4)
    ref = R.forward(cfg, sd, toks)
    whole = run_schedule(eng, toks, [40])
    parts = run_schedule(eng, toks, [7, 2, 9, 3])
    assert close16(rel_err(whole, ref), flips=1)
    assert close16(rel_err(parts, ref), flips=1)
    assert close16(rel_err(parts, whole.double()), flips=1)


def cfg_tc():
    """Sizes of the tensor-core kernels (attention tiles of exact and of smaller head sizes, 64 / 128-wide projections) with
    widths in multiples of 64, windows inside one 64-position tile and across tiles."""
    return config([(attn(heads=4, kv_heads=2, dim=64, vdim=64, size=70, scale=0.125, rot=32, scaling=SCALING), moe(10, 2, 64, 128)),
                   (latent(heads=4, dim=64, vdim=72, kv_rank=64, q_rank=96, size=100, scale=0.12), moe(12, 2, 128, 64)),
                   (attn(heads=2, kv_heads=1, dim=128, vdim=128, size=20, scale=0.09, rot=64), None),
                   (latent(heads=2, dim=40, vdim=128, kv_rank=128, q_rank=64, size=33, scale=0.15), moe(8, 1, 64, 0)),
                   (attn(heads=2, kv_heads=2, dim=48, vdim=160, size=0, scale=0.14, rot=48), moe(6, 3, 64, 64))],
                  width=128, vocab=200, loop=(1, 3, 2))


def test_bfloat16_sizes_of_the_tensor_core_kernels():
    """Projections on the tensor-core GEMMs and the split-K weight stream, attention over portions of 16 rows and more on the
    tensor cores, latents expanded for the pages in view only, the chosen-experts kernels for decode rows and the all-experts
    form for portions, the row-wise kernels for the other steps; all against the oracle and against each other."""
    cfg = cfg_tc()
    eng, sd = build(cfg, torch.bfloat16, max_seq_len=256, page_size=16, pool=512, std=0.08)
    from dli_b200 import ops
    eng.moe_sel_min_bytes = 0                     # the engine keeps the chosen-experts kernels for large mixtures; here they run
    assert eng._moe_sel_ok(eng.spec.layers[0].moe, 1) and not eng._moe_sel_ok(eng.spec.layers[0].moe, 5)
    for i, L in enumerate(eng.spec.layers):
        assert ops.attn_ragged_tc_supported(L.mixer.dim, L.mixer.vdim, torch.bfloat16)
        assert L.mixer.kind == "attention" or "w_ukv" in eng.layers[eng.spec.source(i)]
    toks = prompt(230, cfg["vocab"], 6)
    ref = R.forward(cfg, sd, toks)
    whole = run_schedule(eng, toks, [230])
    hold = eng.open_sequence()                 # another sequence holds the first pages of the pool meanwhile
    eng.step([(hold, prompt(40, cfg["vocab"], 7))])
    parts = run_schedule(eng, toks, [70, 3, 64, 20, 50])
    slot = eng.open_sequence()
    eng.step([(slot, toks[:200])])
    eng.step([(slot, toks[200:])])             # 30 rows from position 200: a window of 33 needs pages from position 128 on
    pages = eng.kv.owned[slot]
    assert eng._pages_in_view(33) == (min(pages[8:]), max(pages[8:])) and eng._pages_in_view(0) == (min(pages), max(pages))
    eng.close_sequence(slot)
    eng.close_sequence(hold)
    eng.tc_min_rows = 10 ** 9
    eng.moe_sel_max_rows = 0
    rowwise = run_schedule(eng, toks, [230])
    for got in (whole, parts, rowwise):
        assert close16(rel_err(got, ref), flips=3)
    assert close16(rel_err(whole, rowwise.double()), flips=3)
    # a long portion beside a decoding sequence and a short portion in one step
    eng.tc_min_rows, eng.moe_sel_max_rows = 16, 8
    a, b, c = (eng.open_sequence() for _ in range(3))
    eng.step([(a, toks[:150]), (c, toks[:5])])
    both = eng.step([(a, [toks[150]]), (b, toks[:90]), (c, toks[5:8])], [[0], list(range(90)), [0, 1, 2]]).float().cpu()
    assert rel_err(both[:1], ref[150:151]).max() < 0.3 and close16(rel_err(both[1:91], ref[:90]), flips=2)
    assert rel_err(both[91:], ref[5:8]).max() < 0.3


def test_mixed_batches_of_unequal_requests_match_each_alone():
    """Four requests of different lengths move through shared steps in portions of different sizes, some decoding while
    others are in their prompt, some skipping steps; each position equals the oracle's for that request alone."""
    cfg = cfg_a()
    eng, sd = build(cfg, torch.float32, pool=192, max_seq_len=192)
    lens = [37, 9, 90, 1]
    reqs = [prompt(n, cfg["vocab"], 10 + i) for i, n in enumerate(lens)]
    refs = [R.forward(cfg, sd, t) for t in reqs]
    slots = [eng.open_sequence() for _ in reqs]
    at, got = [0] * len(reqs), [[] for _ in reqs]
    pattern = [[5, 2, 9, 1], [1, 0, 16, 0], [3, 1, 1, 0], [0, 3, 2, 0], [8, 1, 7, 0], [1, 1, 1, 0], [19, 1, 33, 0]]
    k = 0
    while any(a < n for a, n in zip(at, lens)):
        sizes = pattern[k % len(pattern)]
        k += 1
        batch, want, who = [], [], []
        for i, n in enumerate(sizes):
            n = min(n, lens[i] - at[i])
            if n > 0:
                batch.append((slots[i], reqs[i][at[i]:at[i] + n]))
                want.append(list(range(n)))
                who.append((i, n))
        if not batch:
            continue
        lg = eng.step(batch, want).float().cpu()
        o = 0
        for i, n in who:
            got[i].append(lg[o:o + n])
            o += n
            at[i] += n
    for i in range(len(reqs)):
        assert rel_err(torch.cat(got[i]), refs[i]).max() < TOL32, f"request {i}"


def test_pages_and_slots_are_used_again():
    """A pool that holds two sequences at most and two slots: six sequences pass through in turn, each against the oracle; a
    sequence's pages (every pass of the loop has its own pool) must not leak into the next sequence."""
    cfg = cfg_a()
    eng, sd = build(cfg, torch.float32, max_batch=2, pool=64, max_seq_len=64, page_size=4)
    assert len(eng.kv.k) == len(eng.spec.layers) == 8 and not eng.slots.tensors   # a cache per run, no other state
    for t in eng.kv.k + eng.kv.v:
        t.fill_(10000)                          # whatever a page held before
    for r in range(3):
        ta, tb = prompt(29 + r, cfg["vocab"], 20 + r), prompt(11 + 2 * r, cfg["vocab"], 30 + r)
        ra, rb = R.forward(cfg, sd, ta), R.forward(cfg, sd, tb)
        sa, sb = eng.open_sequence(), eng.open_sequence()
        la = [eng.step([(sa, ta[:13])], [list(range(13))])]
        both = eng.step([(sa, ta[13:]), (sb, tb)], [list(range(len(ta) - 13)), list(range(len(tb)))])
        la.append(both[:len(ta) - 13])
        assert rel_err(torch.cat(la), ra).max() < TOL32
        assert rel_err(both[len(ta) - 13:], rb).max() < TOL32
        eng.close_sequence(sb if r % 2 else sa)   # give the slots back in changing order
        eng.close_sequence(sa if r % 2 else sb)
    assert len(eng.kv.free) == eng.kv.num_pages and len(eng.slots.free) == 2


def mark_token(sd, token, name="l0.norm1"):
    """Embedding rows with two channels of their own, which the map in front of the mixer leaves apart: channel 0 is large for
    `token` and 0 for the others, channel 1 is the same for all, so that one projection row can be a mark of that token and
    another a constant query."""
    sd["embed"][:, 0], sd["embed"][:, 1] = 0.0, 1.0
    sd["embed"][token, 0] = 3.0
    sd[name][:2], sd[name + ".b"][:2] = 1.0, 0.0


def planted(kind, dim, size, score=9.0, seed=1):
    """One mixer layer in which every query scores `score` on token 5's key and 0 on every other, with that token's norm."""
    if kind == "attention":
        cfg = config([(attn(heads=2, kv_heads=2, dim=dim, vdim=dim, size=size, scale=score / dim, rot=2), None)], width=64, vocab=60, scale=1.0)
    else:
        cfg = config([(latent(heads=2, dim=dim, vdim=dim, kv_rank=2 * dim, q_rank=dim, size=size, scale=score / dim), None)], width=64, vocab=60, scale=1.0)
    from dli_b200 import finezen
    sd = finezen.random_state_dict(finezen.spec_from_config(cfg), seed=seed, std=0.15)
    mark_token(sd, 5)
    p = "l0.mix."
    if kind == "attention":
        sd[p + "q"].zero_(), sd[p + "q.norm"].fill_(1.0), sd[p + "k.norm"].fill_(1.0), sd[p + "sink"].fill_(0.0)
        for h in range(2):
            sd[p + "q"][h * dim + 3, 1] = 20.0      # dimension 3 is not rotated; the norm makes it sqrt(dim)
            sd[p + "k"][h * dim + 3].zero_()
            sd[p + "k"][h * dim + 3, 0] = 200.0     # token 5's key has all its norm there: sqrt(dim)
    else:
        K = 2 * dim
        sd[p + "dq"].zero_(), sd[p + "dq.norm"].fill_(1.0), sd[p + "dkv.norm"].fill_(1.0)
        sd[p + "dq"][0, 1] = 20.0                   # the query latent is sqrt(dim) at entry 0
        sd[p + "uq"].zero_()
        sd[p + "dkv"][0].zero_()
        sd[p + "dkv"][0, 0] = 20.0                  # token 5's latent has most of its norm, sqrt(K), at entry 0 ...
        for h in range(2):
            sd[p + "uq"][h * dim + 3, 0] = 1.0
            sd[p + "uk"][h * dim + 3].zero_()
            sd[p + "uk"][h * dim + 3, 0] = (dim / K) ** 0.5
    sd[p + "g"].zero_()                             # half of every head's output, so that no position hides the key
    sd[p + "o"] *= 6.0
    return cfg, sd


@pytest.mark.parametrize("kind", ["attention", "latent_attention"])
@pytest.mark.parametrize("dtype,dim", [(torch.float32, 8), (torch.bfloat16, 64), (torch.bfloat16, 40)])
@pytest.mark.parametrize("size", [21, 64])
def test_a_key_just_inside_and_just_outside_the_window(kind, dtype, dim, size):
    """Token 5's key takes nearly all of every query's weight up to the last position whose window holds it and is gone at the
    next one, in a prompt's portion and in decoding (bfloat16: the tensor-core tiles and the row-wise kernels; latents
    themselves and expanded ones)."""
    cfg, sd = planted(kind, dim, size)
    eng, _ = build(cfg, dtype, max_seq_len=128, page_size=16 if size == 64 else 4, sd=sd)
    at = 10
    toks = [t if t != 5 else 6 for t in prompt(100, 60, 13)]
    toks[at] = 5
    other = list(toks)
    other[at] = 6
    ref, without = R.forward(cfg, sd, toks), R.forward(cfg, sd, other)
    moved = rel_err(without, ref)
    tol = TOL32 if dtype == torch.float32 else 0.04
    last_in = at + size - 1
    assert moved[at:last_in + 1].min() > 5 * tol and moved[last_in + 1:].max() < 1e-9
    for cuts in ([100], [8], [last_in, 2], [last_in + 1, 2, 16]):
        assert rel_err(run_schedule(eng, toks, cuts), ref).max() < tol


@pytest.mark.parametrize("kind", ["attention", "latent_attention"])
@pytest.mark.parametrize("dtype,dim", [(torch.float32, 8), (torch.bfloat16, 64)])
def test_a_key_hundreds_of_tokens_back_without_a_window(kind, dtype, dim):
    cfg, sd = planted(kind, dim, 0, score=14.0)
    eng, _ = build(cfg, dtype, max_seq_len=512, page_size=16, sd=sd)
    toks = [5] + [t if t != 5 else 6 for t in prompt(400, 60, 9)]
    ref, without = R.forward(cfg, sd, toks), R.forward(cfg, sd, [6] + toks[1:])
    tol = TOL32 if dtype == torch.float32 else 0.04
    assert rel_err(without[-50:], ref[-50:]).min() > 5 * tol
    for cuts in ([401], [360], [130, 2, 64, 100, 17, 60]):
        assert rel_err(run_schedule(eng, toks, cuts), ref).max() < tol


@pytest.mark.parametrize("make", ALL)
def test_long_decoding_float32(make):
    """150 tokens one by one: pages fill and follow, windows pass over decoded tokens, the passes' caches grow together."""
    cfg = make()
    eng, sd = build(cfg, torch.float32)
    toks = prompt(150, cfg["vocab"], 11)
    assert rel_err(run_schedule(eng, toks, [3]), R.forward(cfg, sd, toks)).max() < TOL32


def test_greedy_generation_through_the_scheduler():
    """generate() -> RaggedBatcher -> step(): three prompts of one length share steps; tokens equal the oracle's greedy
    continuation (float32 engine: no near-ties at these sizes)."""
    cfg = cfg_a()
    eng, sd = build(cfg, torch.float32, max_batch=3)
    eng.prefill_chunk = 8   # prompts go in portions of at most 8 tokens per step, shared between the requests
    ids = torch.tensor([prompt(13, cfg["vocab"], 40 + i) for i in range(3)])
    out = eng.generate(ids, max_length=13 + 5)
    for b in range(3):
        assert out[b].tolist() == R.greedy(cfg, sd, ids[b].tolist(), 5)
    assert len(eng.slots.free) == 3 and len(eng.kv.free) == eng.kv.num_pages


def test_decode_steps_replayed_as_a_graph_equal_eager_steps():
    """Steps of single tokens are captured once per batch size and replayed; the logits equal the eager launches' bit for
    bit, also when the batch size changes and a sequence leaves in between."""
    cfg = cfg_a()
    outs = []
    for graph in (True, False):
        eng, sd = build(cfg, torch.float32, max_batch=3)
        eng.use_cuda_graph = graph
        seqs = [prompt(30, cfg["vocab"], 60 + i) for i in range(3)]
        slots = [eng.open_sequence() for _ in seqs]
        got = [eng.step([(slots[i], seqs[i][:9]) for i in range(3)])]
        for t in range(9, 20):
            got.append(eng.step([(slots[i], [seqs[i][t]]) for i in range(3)]))
        eng.close_sequence(slots[1])
        for t in range(20, 30):
            got.append(eng.step([(slots[i], [seqs[i][t]]) for i in (0, 2)]))
        outs.append(torch.cat([g.float().cpu() for g in got]))
        if graph:
            assert any(isinstance(v, tuple) for v in eng._graphs.values())
    assert torch.equal(outs[0], outs[1])


def test_a_layer_style_that_tanh_maps_do_not_have_is_refused():
    from dli_b200 import finezen
    from dli_b200.ragged_engine import RaggedEngine

    spec = finezen.spec_from_config(cfg_c())
    spec.layers[0].layer_scale = True
    with pytest.raises(ValueError, match="tanh"):
        RaggedEngine(spec, max_batch=1, max_seq_len=64)
