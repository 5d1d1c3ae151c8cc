"""The Salizen design on the ragged engine against the plain float64 oracle (oracle/salizen_ref.py).

Small made-up configurations with random weights.  The float32 engine must agree with the oracle to ~1e-4 of the
logits' spread at EVERY position — a key one position off at a window's edge, a matrix state lost or taken from another
slot, a wrong previous token, streams mixed in the wrong direction or a sink left out changes logits by orders of
magnitude more — whatever the schedule: whole prompts, token-by-token decoding, portions down to two tokens, mixed
batches, small page pools and reused slots.  The bfloat16 engine is held to a bf16-sized bound and to agreement between
schedules.
"""
import pytest
import torch

pytestmark = pytest.mark.gpu

from oracle import salizen_ref as R  # noqa: E402


def decays(n, lo=0.6):
    return [lo + (0.999 - lo) * k / max(n - 1, 1) for k in range(n)]


def lightning(heads=3, dim=6, vdim=10, decay=None):
    return "lightning", {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay or decays(heads)}


def retention(heads=2, dim=8, vdim=6, rot=6, base=1000.0, decay=None):
    return "retention", {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay or decays(heads, 0.8), "rot": {"base": base, "dims": rot}}


def parallel(heads=4, kv_heads=2, dim=8, size=9, scale=0.4, cap=5.0, rot=4, scaling=None, r_heads=2, r_dim=6, r_vdim=4, tau=3.0, ls=0.7,
             rs=0.4):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "softcap": cap, "mask": {"size": size},
            "rot": {"base": 300.0, "dims": rot}}
    if scaling:
        left["rot"]["scaling"] = scaling
    return "parallel", {"left_scale": ls, "right_scale": rs, "left": left,
                        "right": {"heads": r_heads, "dim": r_dim, "vdim": r_vdim, "tau": tau}}


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, ff=12):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


SCALING = {"factor": 3.0, "low": 1.0, "high": 4.0, "original": 64}


def config(layers, width=48, vocab=97, eps=1e-5, scale=3.0, streams=3, bigram=(53, 13, 5)):
    return {"architecture": "Salizen", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps},
            "embedding": {"scale": scale, "bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))},
            "layers": [{"type": t, "mixer": m, "mlp": mlp} for (t, m), mlp in layers]}


def cfg_a():
    """Every kind of mixer and feed-forward, three streams, frequency scaling that reaches all three of its ranges."""
    return config([(lightning(), dense()), (parallel(scaling=SCALING, rot=8), moe()), (retention(), None),
                   (retention(heads=3, dim=4, vdim=12, rot=4), moe(experts=5, top=3, ff=20)),
                   (parallel(heads=3, kv_heads=1, dim=12, size=16, rot=6, r_heads=3, r_dim=4, r_vdim=8, tau=16.0), dense(24)),
                   (lightning(heads=2, dim=8, vdim=4), moe(experts=3, top=1, ff=8))])


def cfg_b():
    """Values that often coincide taken apart, and extremes: one stream, a window of one position and none at all, no cap,
    every expert chosen, a single expert, decays of 0 and 1, tau 1 (a fast decay per channel), one pair of the table's rows
    only, odd sizes of the recurrent heads, the whole head rotated and none of it."""
    return config([(parallel(heads=2, kv_heads=2, dim=6, size=1, cap=0.5, rot=6, r_heads=1, r_dim=5, r_vdim=3, tau=1.0, ls=1.3, rs=0.2), moe(experts=3, top=3, ff=8)),
                   (lightning(heads=2, dim=7, vdim=5, decay=[0.0, 1.0]), dense(20)),
                   (parallel(heads=1, kv_heads=1, dim=10, size=0, cap=0.0, rot=2, r_heads=2, r_dim=9, r_vdim=2, tau=0.5), moe(experts=1, top=1, ff=16)),
                   (retention(heads=1, dim=4, vdim=7, rot=2, decay=[0.25]), None)],
                  width=40, vocab=53, scale=1.0, streams=1, bigram=(1, 3, 2))


def cfg_c():
    """One layer without a feed-forward; pair hashes beyond 32 bits."""
    return config([(parallel(size=6, cap=2.0), None)], width=32, streams=2, bigram=(101, 3000000019, 70000001))


def build(cfg, dtype, seed=0, max_batch=4, max_seq_len=256, pool=None, page_size=4, std=0.15, sd=None):
    from dli_b200 import salizen
    from dli_b200.ragged_engine import RaggedEngine

    spec = salizen.spec_from_config(cfg)
    if sd is None:
        sd = salizen.random_state_dict(spec, seed=seed, std=std, rank=5)
    eng = RaggedEngine(spec, max_batch=max_batch, max_seq_len=max_seq_len, page_size=page_size, kv_pool_tokens=pool, dtype=dtype)
    eng.load_tensors(salizen.model_tensors(spec, sd))
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
    left out of the second condition — where two experts' logits lie within a few thousandths of each other, bf16 rounding
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


@pytest.mark.parametrize("make", [cfg_a, cfg_b])
def test_sum_of_the_streams_after_every_layer(make):
    cfg = make()
    eng, sd = build(cfg, torch.float32)
    toks = prompt(19, cfg["vocab"], 2)
    layers = []
    R.forward(cfg, sd, toks, layers)
    n = len(cfg["layers"])
    for cuts in ([19], []):
        eng.layer_trace = []
        run_schedule(eng, toks, cuts)
        trace, eng.layer_trace = eng.layer_trace, None
        assert len(trace) == n * (1 if cuts else 19)
        got = trace if cuts else [torch.cat(trace[i::n]) for i in range(n)]
        for g, ref in zip(got, layers):
            assert (g.double().cpu() - ref).abs().max() < 1e-4 * ref.abs().max()


@pytest.mark.parametrize("make", ALL)
@pytest.mark.parametrize("cuts", [[], [1, 1, 2], [2, 2, 3, 5, 7, 11], [17, 2, 16, 3], [30]])
def test_portions_and_decoding_float32(make, cuts):
    """Token by token from the first token; portions of 2..; a prompt then decoding over page borders and over the edges of
    windows of 1, 6, 9 and 16 positions."""
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
    """Sizes of the tensor-core kernels (attention and linear attention, 64 / 128-wide projections) with widths in multiples
    of 64, windows inside one 64-position tile and across tiles."""
    return config([(lightning(heads=2, dim=64, vdim=128), dense(256)),
                   (parallel(heads=4, kv_heads=2, dim=64, size=70, scale=0.125, rot=32, r_heads=2, r_dim=48, r_vdim=72, tau=8.0), moe(experts=10, top=2, ff=64)),
                   (retention(heads=2, dim=128, vdim=64, rot=128), moe(experts=12, top=2, ff=128)),
                   (parallel(heads=2, kv_heads=1, dim=128, size=20, scale=0.09, rot=64, r_heads=1, r_dim=128, r_vdim=64, tau=2.0), dense(128)),
                   (retention(heads=2, dim=32, vdim=40, rot=20), dense(128))],
                  width=128, vocab=200, streams=2)


def test_bfloat16_sizes_of_the_tensor_core_kernels():
    """Projections on the tensor-core GEMMs and the split-K weight stream, attention and the recurrences over portions of 16
    rows and more on the tensor cores, the chosen-experts kernels for decode rows and the all-experts form for portions, the
    row-wise kernels for the other steps; all against the oracle and against each other."""
    cfg = cfg_tc()
    eng, sd = build(cfg, torch.bfloat16, max_seq_len=256, page_size=16, pool=512, std=0.08)
    from dli_b200 import ops
    eng.moe_sel_min_bytes = 0                     # the engine keeps the chosen-experts kernels for large mixtures; here they run
    assert eng._moe_sel_ok(eng.spec.layers[1].moe, 1) and not eng._moe_sel_ok(eng.spec.layers[1].moe, 3)
    for L in eng.spec.layers:
        for m in L.mixer.flat:
            assert ops.attn_ragged_tc_supported(m.dim, m.vdim, torch.bfloat16) if m.kind == "attention" else \
                ops.linattn_tc_supported(m.dim, m.vdim, bool(m.tau), m.qkv_silu, m.rot_dims, torch.bfloat16)
    toks = prompt(230, cfg["vocab"], 6)
    ref = R.forward(cfg, sd, toks)
    whole = run_schedule(eng, toks, [230])
    hold = eng.open_sequence()                 # another sequence holds the first pages of the pool meanwhile
    eng.step([(hold, prompt(40, cfg["vocab"], 7))])
    parts = run_schedule(eng, toks, [70, 3, 64, 20, 50])
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
    slot's matrix states and last token and its pages must not leak into the next sequence."""
    cfg = cfg_a()
    eng, sd = build(cfg, torch.float32, max_batch=2, pool=64, max_seq_len=64, page_size=4)
    for t in eng.slots.tensors.values():
        t.fill_(10000)                          # whatever a slot held before
    assert len(eng.slots.tensors) == len(cfg["layers"]) + 1
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


def mark_token(sd, token):
    """Embedding rows with two channels of their own: channel 0 is large for `token` and 0 for the others, channel 1 is the
    same for all, so that one projection row can be a mark of that token and another a constant query."""
    sd["bigram"].zero_()
    sd["embed"][:, 0], sd["embed"][:, 1] = 0.0, 1.0
    sd["embed"][token, 0] = 3.0


def test_a_state_written_hundreds_of_tokens_back_is_still_read():
    """One retention layer: in the slow head only token 7 has a key, and it stands at position 0; every later query asks for
    it.  Without that write the slow head's output is zero, so a state that is lost at any step, or decays twice, shows at
    every later position of 400 (decoded one by one, or in portions)."""
    from dli_b200 import salizen

    cfg = config([(retention(heads=2, dim=4, vdim=4, rot=2, decay=[0.999, 0.01]), None)], width=16, vocab=40, streams=2)
    eng, sd = build(cfg, torch.float32, max_seq_len=512)
    mark_token(sd, 7)
    for k, ch in (("q", 1), ("k", 0)):
        sd["l0.mix." + k][:4].zero_()
        sd["l0.mix." + k][3, ch] = 2.0          # a dimension that is not rotated
    sd["l0.mix.o"] *= 4.0
    eng.load_tensors(salizen.model_tensors(eng.spec, sd))
    toks = [7] + [t if t != 7 else 8 for t in prompt(400, 40, 9)]
    ref, without = R.forward(cfg, sd, toks), R.forward(cfg, sd, [8] + toks[1:])
    assert rel_err(without[-50:], ref[-50:]).min() > 50 * TOL32
    for cuts in ([401], [2], [130, 2, 64, 100]):
        assert rel_err(run_schedule(eng, toks, cuts), ref).max() < TOL32


@pytest.mark.parametrize("dtype,dim", [(torch.float32, 8), (torch.bfloat16, 64)])
def test_a_key_just_inside_and_just_outside_the_window(dtype, dim):
    """One attention layer in which token 5's key has the capped score of every query: its share is nearly 1 up to the last
    position whose window holds it and gone at the next one, in a prompt's portion and in decoding (bfloat16: the
    tensor-core tiles and the row-wise kernel)."""
    from dli_b200 import salizen

    size = 21
    cfg = config([(parallel(heads=2, kv_heads=2, dim=dim, size=size, scale=dim ** -0.5, cap=9.0, rot=2, r_heads=1, r_dim=4, r_vdim=4, rs=0.0, ls=1.0), None)],
                 width=64, vocab=60, streams=2)
    eng, sd = build(cfg, dtype, max_seq_len=128)
    mark_token(sd, 5)
    for g in range(2):
        sd["l0.mix.left.q"][g * dim:(g + 1) * dim].zero_()
        sd["l0.mix.left.q"][g * dim + 3, 1] = 20.0
        sd["l0.mix.left.k"][g * dim + 3].zero_()
        sd["l0.mix.left.k"][g * dim + 3, 0] = 20.0
    eng.load_tensors(salizen.model_tensors(eng.spec, sd))
    at = 10
    toks = [t if t != 5 else 6 for t in prompt(70, 60, 13)]
    toks[at] = 5
    other = list(toks)
    other[at] = 6
    ref, without = R.forward(cfg, sd, toks), R.forward(cfg, sd, other)
    moved = rel_err(without, ref)
    tol = TOL32 if dtype == torch.float32 else 0.04
    last_in = at + size - 1
    assert moved[at:last_in + 1].min() > 5 * tol and moved[last_in + 1:].max() < 1e-9
    for cuts in ([70], [8], [last_in, 2], [last_in + 1, 2, 16]):
        assert rel_err(run_schedule(eng, toks, cuts), ref).max() < tol


def test_the_previous_token_is_carried_between_steps():
    """A pair table with large rows: the first position has its own row, every other depends on the token before it, also
    when that token came with an earlier step or the slot served another sequence before."""
    cfg = cfg_c()
    eng, sd = build(cfg, torch.float32)
    from dli_b200 import salizen
    sd["bigram"] = sd["bigram"] * 20.0
    eng.load_tensors(salizen.model_tensors(eng.spec, sd))
    toks = prompt(30, cfg["vocab"], 5)
    ref = R.forward(cfg, sd, toks)
    swapped = [toks[1], toks[0]] + toks[2:]
    assert rel_err(R.forward(cfg, sd, swapped)[:3], ref[:3]).min() > 100 * TOL32
    other = eng.open_sequence()                # a second live sequence whose last token lies in another slot
    eng.step([(other, prompt(6, cfg["vocab"], 8))])
    for cuts in ([30], [], [4, 2, 2, 9]):
        assert rel_err(run_schedule(eng, toks, cuts), ref).max() < TOL32
    eng.close_sequence(other)


@pytest.mark.parametrize("make", [cfg_a, cfg_b])
def test_long_decoding_float32(make):
    """150 tokens one by one: the states are carried 150 times, pages fill and follow, windows pass over decoded tokens."""
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
