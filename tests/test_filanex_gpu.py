"""Filanex on the device against the plain implementation: each mechanism alone (fed in portions beside another request),
keys just inside and just outside a chunk in prompts and in decoding while pages of earlier chunks go back, a far key
that dominates inside a long chunk, a cap that binds, a stretched rotation of neighbouring pairs, the gate per element in
every attention kernel, biases and the exact gelu in every path of the products, experts limited to the groups whose two
best scores sum highest, the previous token carried from step to step, a loop's passes with caches of their own, whole
models under every way of cutting the work, slots and pages used again, long decoding through captured graphs, and greedy
generation through the entry point and its scheduler."""
import numpy as np
import pytest
import torch

from tests.filanex_configs import FILANEX, drawn_filanex, plain_inputs, write_filanex_dir
from tests.plain import filanex_plain as plain
from tests.replay_helpers import collect, max_live_tokens, trace_mixed, trace_portions, trace_tail_decode, trace_whole
from tests.test_fadosun_gpu import _rel, _weights
from tests.test_pepapel_gpu import _run_mixer
from tests.test_zufusun_gpu import _run_feed_forward, attention_kernel, replay  # noqa: F401  (attention_kernel: a fixture)

pytestmark = pytest.mark.gpu

# A position's error is norm(got - want) / norm(want) over its logits.  Rounding is 1e-6 in float32 and 1e-2 in bfloat16
# except where a router's close call falls the other way.  A fault of a mechanism (a key too many, a lost previous token, a
# gate or a bias left out, a chunk's edge one off) is 1e-2 or more in float32 at every position it touches.
TOL = {"float32": dict(median=5e-6, worst=3e-4), "bfloat16": dict(median=3e-2, worst=None, over=0.06, above=0.12)}
MIX_TOL = {torch.float32: 2e-5, torch.bfloat16: 2e-2}


def assert_close(got, want, dtype, what="", over=None):
    errs = sorted((float(np.linalg.norm(rows[p] - want[r][p]) / max(np.linalg.norm(want[r][p]), 1e-30)), r, p)
                  for r, rows in got.items() for p in rows)
    assert errs and all(np.isfinite(e[0]) for e in errs), f"{what} {dtype}: no output or a NaN"
    t = TOL[dtype]
    median, worst = errs[len(errs) // 2][0], errs[-1]
    assert median < t["median"], f"{what} {dtype}: median error {median:.3g}"
    if t["worst"] is not None:
        assert worst[0] < t["worst"], f"{what} {dtype}: worst error {worst[0]:.3g} at {worst[1:]}"
    else:
        n = sum(e[0] > t["above"] for e in errs)
        assert n <= max(2, int((over or t["over"]) * len(errs))), f"{what} {dtype}: {n} of {len(errs)} positions over {t['above']}, worst {worst}"


@pytest.fixture(scope="module")
def dirs(tmp_path_factory):
    return {name: write_filanex_dir(name, str(tmp_path_factory.mktemp("filanex_" + name))) for name in FILANEX}


@pytest.fixture(scope="module")
def plain_logits(dirs):
    cache, inputs = {}, {}

    def get(name, requests):
        if name not in inputs:
            inputs[name] = plain_inputs(dirs[name])
        out = {}
        for rid, toks in requests.items():
            key = (name, tuple(toks))
            if key not in cache:
                cache[key] = plain.forward(*inputs[name], toks).numpy()
            out[rid] = cache[key]
        return out

    return get


def make_requests(name, lengths, seed):
    rng = np.random.default_rng(seed)
    return {f"r{i}": rng.integers(0, FILANEX[name]["json"]["vocab"], size=n).tolist() for i, n in enumerate(lengths)}


LENGTHS = {"a": (1, 2, 37, 130), "b": (3, 18, 65, 110), "c": (2, 70, 140), "d": (1, 25, 90)}


# ------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("page", [16, 64])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(FILANEX))
@pytest.mark.parametrize("mode", ["whole", "tail", "portions", "mixed"])
def test_replay_modes(name, dtype, mode, page, dirs, plain_logits):
    """Whole prompts, a decoded tail (chunk edges pass under decoded tokens), portions down to two tokens (and single
    ones), and four live requests whose slots and pages are used again, against each request alone in the plain
    implementation."""
    requests = make_requests(name, LENGTHS[name], seed=5)
    if mode == "mixed":
        requests = make_requests(name, LENGTHS[name] + (40, 21, 66, 9), seed=6)
    steps = {"whole": trace_whole, "tail": lambda r: trace_tail_decode(r, tail=45),
             "portions": lambda r: trace_portions(r, sizes=(7, 2, 19, 1, 3, 33, 2, 16, 5, 64)),
             "mixed": lambda r: trace_mixed(r, live=4, seed=3)}[mode](requests)
    outputs, _ = replay(dirs[name], dtype, steps, max_live_tokens(steps, round_to=page), page_tokens=page)
    assert_close(collect(steps, outputs), plain_logits(name, requests), dtype, f"{name} {mode}")


@pytest.mark.parametrize("seed", range(10))
def test_configurations_drawn_at_random(seed, tmp_path):
    """Layer orders, loops, sizes, head counts, chunks, groups and constants drawn from a seed: whole prompts, portions and
    a mixed batch in float32 (the sharper comparison), the mixed batch in bfloat16."""
    cfg = drawn_filanex(seed)
    d = write_filanex_dir(cfg, str(tmp_path), seed=seed)
    inputs = plain_inputs(d)
    rng = np.random.default_rng(100 + seed)
    requests = {f"r{i}": rng.integers(0, cfg["vocab"], size=n).tolist()
                for i, n in enumerate((1, 2, int(rng.integers(30, 90)), int(rng.integers(100, 160)), 47, 19))}
    want = {rid: plain.forward(*inputs, toks).numpy() for rid, toks in requests.items()}
    for dtype, modes in (("float32", ("whole", "portions", "mixed")), ("bfloat16", ("mixed",))):
        for mode in modes:
            steps = {"whole": trace_whole, "portions": lambda r: trace_portions(r, sizes=(7, 2, 19, 1, 3, 33, 2, 16, 5, 64)),
                     "mixed": lambda r: trace_mixed(r, live=4, seed=seed)}[mode](requests)
            page = (16, 64)[seed % 2]
            outputs, _ = replay(d, dtype, steps, max_live_tokens(steps, round_to=page), page_tokens=page)
            # (a single choice among many experts in every pass of a loop: close calls are more frequent than elsewhere)
            assert_close(collect(steps, outputs), want, dtype, f"drawn {seed} {mode}", over=0.15)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_through_graphs_equals_the_prompt(dtype, dirs, plain_logits):
    """300 tokens one by one (captured graphs after the second step; the previous token's slot, the router's grouping, the
    pages that go back and the key splits all inside them) against the whole sequence."""
    requests = make_requests("a", (300,), seed=11)
    steps = trace_tail_decode(requests, tail=299)
    outputs, runner = replay(dirs["a"], dtype, steps, 320)
    assert runner.graph_replays > 250
    assert_close(collect(steps, outputs), plain_logits("a", requests), dtype, "long decoding")
    eager, _ = replay(dirs["a"], dtype, steps, 320, cuda_graphs=False)
    assert max(float(np.abs(outputs[k] - eager[k]).max()) for k in outputs) < (1e-5 if dtype == "float32" else 1e-1)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_long_prompt_then_decoding(dtype, dirs, plain_logits):
    """900 tokens at a real model's head sizes: chunks of 256, 100 and 77 that end inside portions, angles of hundreds of
    positions: as one prompt with a decoded tail and as portions of 400."""
    requests = make_requests("c", (900,), seed=17)
    for steps in (trace_tail_decode(requests, tail=24), trace_portions(requests, sizes=(400, 37, 400, 2))):
        outputs, _ = replay(dirs["c"], dtype, steps, 960, page_tokens=64, max_batch_tokens=1024)
        assert_close(collect(steps, outputs), plain_logits("c", requests), dtype, "long prompt")


def test_a_request_longer_than_the_pool(dirs, plain_logits):
    """Every layer of this model works in chunks: a pool of 384 tokens serves a request of 700, because the pages of chunks
    that have passed come back while it runs."""
    requests = make_requests("c", (700,), seed=19)
    steps = trace_portions(requests, sizes=(64, 30, 1, 1, 50))
    outputs, _ = replay(dirs["c"], "float32", steps, 384, page_tokens=16)
    assert_close(collect(steps, outputs), plain_logits("c", requests), "float32", "longer than the pool")


@pytest.mark.parametrize("name", ["a", "b"])
def test_a_slot_used_again_starts_anew(name, dirs, plain_logits):
    """One slot only: the second request gets the pages the first left and the slot with the first's last token in it."""
    requests = make_requests(name, (90, 75, 33), seed=21)
    steps = trace_portions(requests, sizes=(40, 3, 1, 31))
    outputs, _ = replay(dirs[name], "float32", steps, 96, max_requests=1)
    assert_close(collect(steps, outputs), plain_logits(name, requests), "float32", "one slot")


@pytest.mark.parametrize("name", ["a", "b"])
def test_greedy_generation_through_the_engine(name, dirs):
    """Greedy tokens from ``ember_b200.load(...).generate`` (scheduler, portions of 16, few pages, four prompts of unequal
    length, three slots; decode steps launched before the ids of the step before are back, so the token and the previous
    token are read on the device) against greedy decoding with the plain implementation."""
    import ember_b200
    cfg, W = plain_inputs(dirs[name])
    prompts = list(make_requests(name, (5, 40, 1, 23), seed=31).values())
    llm = ember_b200.load(dirs[name], dtype="float32", kv_cache_tokens=256, max_batch_tokens=64, max_seqs=3, prefill_chunk=16,
                          page_tokens=16)
    got = llm.generate(prompts, max_tokens=14, ignore_eos=True)
    for p, ids in zip(prompts, got):
        seq = list(p)
        for _ in range(14):
            seq.append(int(plain.forward(cfg, W, seq)[-1].argmax()))
        assert list(ids) == seq[len(p):]
    assert llm.runner.cache.check() == ""


def test_generation_under_preemption_keeps_the_previous_token(dirs):
    """So few pages that requests are preempted and admitted again into used slots: the same tokens as with room for all."""
    import ember_b200
    prompts = list(make_requests("a", (30, 28, 35, 31), seed=33).values())
    outs = []
    for tokens in (1024, 144):
        llm = ember_b200.load(dirs["a"], dtype="float32", kv_cache_tokens=tokens, max_batch_tokens=64, max_seqs=4, prefill_chunk=16, page_tokens=16)
        outs.append(llm.generate(prompts, max_tokens=40, ignore_eos=True))
        preempted = llm.engine.stats.preemptions
    assert preempted > 0 and outs[0] == outs[1]


# --------------------------------------------------------------------------------- the embedding, alone
@pytest.mark.parametrize("table_dtype,bigram_dtype", [(torch.bfloat16, torch.bfloat16), (torch.float32, torch.float32), (torch.bfloat16, torch.float32)])
def test_bigram_embedding_carries_the_previous_token(table_dtype, bigram_dtype):
    """Runs of one and several tokens beside one another, over three steps; multipliers whose products pass 2^31; slots
    that hold another request's token; tokens that are still on the device (negative: the id the sampler left)."""
    from ember_b200 import ops
    V, H, B, a, b = 1000, 72, 501, 2000003, 1999993
    g = torch.Generator().manual_seed(1)
    table, extra = torch.randn(V, H, generator=g).to(table_dtype), torch.randn(B + 1, H, generator=g).to(bigram_dtype)
    seqs = {s: torch.randint(0, V, (12,), generator=g).tolist() for s in range(3)}
    want = {s: plain.embed({"embedding": {"bigram": {"buckets": B, "mul_prev": a, "mul_cur": b}}},
                           {"embed": table, "bigram": extra}, t, torch.float64) for s, t in seqs.items()}
    dev = "cuda"
    state = torch.full((5, 1), 999, dtype=torch.int32, device=dev)            # whatever the slot's last owner left
    err = torch.zeros(1, dtype=torch.int32, device=dev)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)            # noqa: E731
    at = {0: 0, 1: 0, 2: 0}
    slot = {0: 3, 1: 0, 2: 4}
    for step in ([(0, 5), (1, 1)], [(2, 7), (0, 1), (1, 2)], [(1, 1), (2, 5), (0, 6)], [(1, 1)]):
        toks, pos, seq, qs, rows = [], [], [], [0], []
        for i, (s, n) in enumerate(step):
            toks += seqs[s][at[s]:at[s] + n]
            pos += range(at[s], at[s] + n)
            rows += [(s, p) for p in range(at[s], at[s] + n)]
            seq += [i] * n
            qs.append(qs[-1] + n)
            at[s] += n
        prev_ids = i32([7, toks[-1], 9])
        if len(step) == 1:
            toks[-1] = -2                                                     # row 1 of the sampler's output
        out = torch.zeros(len(toks), H, device=dev)
        ops.embed_bigram(i32(toks), table.to(dev), extra.to(dev), out, B, a, b, i32(pos), i32(seq), i32(qs), i32([slot[s] for s, _ in step]),
                         state, scale=1.0, err=err, prev_ids=prev_ids)
        for r, (s, p) in enumerate(rows):
            assert float((out[r].cpu().double() - want[s][p]).abs().max()) < 1e-6, (step, s, p)
        for s, _ in step:
            assert int(state[slot[s], 0]) == seqs[s][at[s] - 1]
    assert int(err.item()) == 0 and int(state[1, 0]) == 999


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hidden", [64, 100])
def test_reentry_mixes_the_stream_with_the_embedding_output(dtype, hidden):
    """x <- W [x; x0], the first time (x is x0) and again with another x; the columns of x come first."""
    from ember_b200.config import ConcatReentrySpec
    from ember_b200.parts import build_part
    from tests.test_parts_gpu import Bench, store_of
    g = torch.Generator().manual_seed(hidden)
    w = (0.1 * torch.randn(hidden, 2 * hidden, generator=g)).bfloat16()
    part = build_part("reentry", ConcatReentrySpec(size=hidden, name="in"), "loop.")
    b = Bench({}, dtype)
    part.load(store_of({"loop.in": w}), b.rt)
    x0, x1 = torch.randn(20, hidden, generator=g), torch.randn(20, hidden, generator=g)
    for separate in (False, True):
        ctx = b.ctx([("r", 17)])
        h = x0.to(b.dev).clone()
        if separate:
            part.keep(ctx, h)
            part.forward(ctx, h)
        else:
            part.forward(ctx, h, first=True)
        assert _rel(h[:17].cpu(), plain.lin(torch.cat([x0, x0], -1).double(), w)[:17]) < MIX_TOL[dtype]
        assert torch.equal(h[17:].cpu(), x0[17:])
        h = x1.to(b.dev).clone()
        part.forward(ctx, h)
        want = plain.lin(torch.cat([x1, x0], -1).double(), w)[:17]
        assert _rel(h[:17].cpu(), want) < MIX_TOL[dtype]
        assert _rel(plain.lin(torch.cat([x0, x1], -1).double(), w)[:17], want) > 0.3
        b.cache.release("r")


# -------------------------------------------------------------------------------------- the mixer, alone
def _spec(heads, kv, dim, vdim, hidden, scale=0.2, softcap=0.0, chunk=0, rot=None):
    from ember_b200.config import NoPositionSpec, RotarySpec, SinkAttentionSpec
    pos = NoPositionSpec()
    if rot:
        sc = rot.get("scaling")
        kw = dict(scaling_factor=sc["factor"], scaling_original=sc["original"], scaling_fast=sc["fast"], scaling_slow=sc["slow"]) if sc else {}
        pos = RotarySpec(head_dim=dim, rotary_dim=rot["dims"], theta=rot["base"], frequency_precision="float64", layout="interleaved", **kw)
    return SinkAttentionSpec(hidden_size=hidden, num_heads=heads, num_kv_heads=kv, head_dim=dim, value_dim=vdim, scale=scale,
                             sink=False, softcap=softcap, chunk=chunk, position=pos, element_gate=True)


def _m(heads, kv, dim, vdim, scale=0.2, softcap=0.0, chunk=0, rot=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if softcap:
        m["softcap"] = softcap
    if chunk:
        m["mask"] = {"size": chunk}
    if rot:
        m["rot"] = rot
    return m


def _want(x, w, m):
    return plain.attention_mixer(x.double(), {k: v.double() for k, v in w.items()}, "m.", m)


YARN = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}
MIXER_CASES = [
    (6, 2, 16, 24, 64, 4.0, 20, {"dims": 16, "base": 1e4, "scaling": YARN}),
    (4, 1, 20, 12, 100, 0.0, 16, {"dims": 8, "base": 77.0}),
    (2, 2, 128, 128, 128, 30.0, 64, {"dims": 64, "base": 1e6, "scaling": YARN}),
    (3, 3, 18, 300, 72, 1.0, 33, {"dims": 2, "base": 10.0}),
    (40, 1, 8, 8, 64, 2.0, 0, None),
    (4, 1, 64, 32, 64, 40.0, 7, {"dims": 64, "base": 500.0, "scaling": {**YARN, "factor": 1.0}}),
    (1, 1, 48, 16, 64, 5.0, 1, {"dims": 46, "base": 500.0}),
    (6, 2, 40, 56, 64, 3.0, 120, {"dims": 40, "base": 2e4, "scaling": {**YARN, "factor": 16.0}}),
]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv,dim,vdim,hidden,softcap,chunk,rot", MIXER_CASES)
def test_attention_alone(dtype, heads, kv, dim, vdim, hidden, softcap, chunk, rot, attention_kernel):
    """Whole and partial rotations of neighbouring pairs, stretched and not, caps from one that flattens most scores to
    none, chunks from one position to longer than the sequence, values wider and narrower than keys, forty query heads on
    one key head, the gate per element."""
    spec = _spec(heads, kv, dim, vdim, hidden, 0.5, softcap, chunk, rot)
    w = _weights(spec, seed=heads, std=0.15)
    x = torch.randn(90, hidden, generator=torch.Generator().manual_seed(2)).bfloat16()
    want = _want(x, w, _m(heads, kv, dim, vdim, 0.5, softcap, chunk, rot))
    assert _rel(_run_mixer(spec, w, x, dtype), want) < MIX_TOL[dtype]


@pytest.mark.parametrize("dense", [True, False], ids=["TMA-fed kernels", "shared-row kernels"])
@pytest.mark.parametrize("heads,kv,dim,softcap,chunk,rot", [
    (8, 1, 128, 25.0, 50, {"dims": 64, "base": 1e4, "scaling": YARN}), (4, 2, 64, 0.0, 64, {"dims": 64, "base": 500.0}),
    (2, 2, 128, 0.7, 7, {"dims": 16, "base": 1e6}), (16, 1, 64, 3.0, 300, {"dims": 32, "base": 1e4, "scaling": YARN}),
    (12, 4, 128, 40.0, 0, {"dims": 128, "base": 1e4, "scaling": YARN}), (6, 2, 64, 5.0, 0, None), (4, 4, 128, 300.0, 90, None)])
def test_layers_on_the_engines_dense_attention_kernels(dense, heads, kv, dim, softcap, chunk, rot, monkeypatch):
    """Keys and values of one size, 64 or 128: bfloat16 steps go to the kernels Qwen3's attention uses, which take the
    chunk, the cap and the gate per element (a group of three query heads a key head takes the mma.sync form for portions
    too); switched off, the same layer runs on the shared-row kernels with the gate as a pass of its own."""
    from ember_b200.parts.sink_attention import SinkAttention
    monkeypatch.setattr(SinkAttention, "DENSE_KERNELS", dense)
    spec = _spec(heads, kv, dim, dim, 128, 0.5, softcap, chunk, rot)
    w = _weights(spec, seed=heads, std=0.15)
    x = torch.randn(200, 128, generator=torch.Generator().manual_seed(8)).bfloat16()
    want = _want(x, w, _m(heads, kv, dim, dim, 0.5, softcap, chunk, rot))
    got = _run_mixer(spec, w, x, torch.bfloat16, portions=((130, 3), (60, 20), (1, 1), (1, 1), (1, 1), (7, 2)))
    assert _rel(got, want) < MIX_TOL[torch.bfloat16]
    for t in (49, 50, 51, 63, 64, 65, 127, 128, 129, 130, 189, 190, 191, 192, 193, 199):
        assert _rel(got[t], want[t]) < 3 * MIX_TOL[torch.bfloat16], t


@pytest.mark.parametrize("merge", ["cluster", "buffers"])
@pytest.mark.parametrize("chunk,at", [(700, 690), (700, 1399), (700, 705), (0, 1399), (900, 1250), (70, 1399)])
def test_single_tokens_over_split_keys_in_a_chunk(chunk, at, merge, monkeypatch):
    """A decoded token whose chunk is cut into key splits that start where the chunk does (inside a tile of 64 keys), merged
    in a cluster or through buffers; the gate joins behind the merge."""
    from ember_b200 import ops
    heads, kv, dim, page = 4, 2, 128, 16
    g = torch.Generator().manual_seed(at)
    n = at + 1
    q = torch.randn(1, heads, dim, generator=g).bfloat16()
    k, v = torch.randn(n, kv, dim, generator=g).bfloat16(), torch.randn(n, kv, dim, generator=g).bfloat16()
    gate = torch.randn(1, 24 + heads * dim, generator=g)
    pages = (n + page - 1) // page
    order = torch.randperm(pages, generator=g)
    kp, vp = (torch.zeros(pages, kv, page, dim, dtype=torch.bfloat16) for _ in range(2))
    for p in range(n):
        kp[order[p // page], :, p % page], vp[order[p // page], :, p % page] = k[p], v[p]
    table = order.to(torch.int32)[None].clone()
    if chunk:
        table[0, :at // chunk * chunk // page] = -1                           # given back
    splits, keys, _ = (3, 320, True) if chunk != 70 else (2, 128, True)
    if not chunk:
        splits, keys = 6, 256
    dev = "cuda"
    tiles = torch.tensor([[0, 0, 1, at]], dtype=torch.int32, device=dev)
    out = torch.zeros(1, heads, dim, dtype=torch.bfloat16, device=dev)
    kw = {}
    if merge == "buffers":
        kw = dict(part_o=torch.zeros(heads * splits * dim, device=dev), part_ml=torch.zeros(heads * splits * 2, device=dev))
    ops.attention_tc(q.to(dev), kp.to(dev), vp.to(dev), out, 1, heads, kv, dim, tiles, 1, table.to(dev), page, 0, 0.3, splits, keys,
                     softcap=9.0, chunk=chunk, gate=gate.to(dev), gate_col=24, **kw)
    torch.cuda.synchronize()
    lo = at // chunk * chunk if chunk else 0
    mask = (torch.arange(n) >= lo)[None]
    want = plain.capped_attention(q.double(), k.double(), v.double(), 0.3, mask, 9.0)
    want = want * torch.sigmoid(gate[:, 24:].double()).reshape(1, heads, dim)
    assert _rel(out.cpu(), want) < 1e-2


def test_the_gate_the_cap_and_the_stretching_are_there():
    """Each of the three switched off in the plain implementation changes the result by much more than the tolerance."""
    rot = {"dims": 16, "base": 500.0, "scaling": {"factor": 8.0, "original": 32, "fast": 4.0, "slow": 0.5}}
    spec = _spec(2, 1, 32, 32, 64, 1.0, 3.0, 50, rot)
    w = _weights(spec, seed=3, std=0.3)
    x = torch.randn(120, 64, generator=torch.Generator().manual_seed(4)).bfloat16()
    m = _m(2, 1, 32, 32, 1.0, 3.0, 50, rot)
    want = _want(x, w, m)
    assert _rel(_want(x, w, {**m, "softcap": 0.0}), want) > 0.2
    assert _rel(_want(x, {**w, "m.g": torch.zeros_like(w["m.g"])}, m), want) > 0.2
    assert _rel(_want(x, w, {**m, "rot": {"dims": 16, "base": 500.0}}), want) > 0.02
    for portions in (((120, 3),), ((49, 1), (1, 1), (1, 1), (1, 1), (2, 1), (66, 30))):
        assert _rel(_run_mixer(spec, w, x, torch.float32, portions=portions), want) < MIX_TOL[torch.float32]


@pytest.mark.parametrize("portions", [((150, 3),), ((40, 3), (1, 1), (1, 1), (1, 1), (37, 30), (2, 1), (68, 1)), ((38, 1),) + ((1, 1),) * 5 + ((35, 1),) + ((1, 1),) * 5 + ((35, 1),) + ((1, 1),) * 5 + ((27, 1),),
                                      ((39, 1), (1, 1), (40, 1), (40, 1), (30, 1))])
def test_keys_just_inside_and_just_outside_a_chunk(portions):
    """Chunks of 40 with pages of 16.  The query at 40 sees itself alone and the one at 79 sees 40 .. 79: with a chunk's
    edge one off, position 40 (or 39) would see one key more or fewer, which changes its result by a large part.  Checked
    row by row around every edge, in a prompt's portion, at a portion's first token and for single tokens."""
    rot = {"dims": 4, "base": 100.0}
    spec = _spec(2, 1, 16, 16, 64, 1.0, 0.0, 40, rot)
    w = _weights(spec, seed=4, std=0.1)
    x = torch.randn(150, 64, generator=torch.Generator().manual_seed(6)).bfloat16()
    m = _m(2, 1, 16, 16, 1.0, 0.0, 40, rot)
    want = _want(x, w, m)
    for off in (39, 41):
        moved = _want(x, w, {**m, "mask": {"size": off}})
        assert min(_rel(moved[t], want[t]) for t in (40, 80, 120)) > 0.02
    got = _run_mixer(spec, w, x, torch.float32, portions=portions)
    for t in (0, 1, 38, 39, 40, 41, 78, 79, 80, 81, 118, 119, 120, 121, 149):
        assert _rel(got[t], want[t]) < 1e-4, t
    assert _rel(got, want) < 1e-4


@pytest.mark.parametrize("portions", [((200, 3),), ((120, 3), (40, 30), (38, 1), (1, 1), (1, 1)), ((2, 1),) * 50 + ((100, 1),)])
def test_a_far_key_that_dominates_is_seen_across_pages_and_portions(portions):
    """A chunk of 300: key 5 is made large along the direction the late queries point in, so that among two hundred keys it
    has most of the weight; lost (a page too few, a page given back too early) the result changes wholly."""
    spec = _spec(2, 1, 16, 24, 64, 1.5, 60.0, 300)
    w = _weights(spec, seed=4, std=0.1)
    x = torch.randn(200, 64, generator=torch.Generator().manual_seed(6))
    x[150:] = x[5] + 0.3 * x[150:]                           # late queries and key 5 come from nearly the same direction
    x[5] *= 2.5                                              # and key 5 is longer than the late keys
    x = x.bfloat16()
    w["m.q"] = w["m.k"].repeat(2, 1)                         # q and k projections alike: q_t . k_5 is large for t >= 150
    m = _m(2, 1, 16, 24, 1.5, 60.0, 300)
    want = _want(x, w, m)
    gone = x.clone()
    gone[5] = 0
    assert min(_rel(a, b) for a, b in zip(_want(gone, w, m)[150:], want[150:])) > 0.3
    assert _rel(_run_mixer(spec, w, x, torch.float32, portions=portions), want) < 1e-4


# ------------------------------------------------------------------------------------------ feed-forwards
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hidden,ff", [(64, 40), (100, 30), (128, 256), (72, 1000)])
def test_dense_feed_forward_alone(dtype, hidden, ff):
    """Biases on both projections, stored and added; without them the result is far away."""
    from ember_b200.config import MLPSpec
    spec = MLPSpec(hidden_size=hidden, intermediate_size=ff, names=("up", "down"), bias=True)
    g = torch.Generator().manual_seed(ff)
    w = {f"f.{n}": (0.3 * torch.randn(s, generator=g)).bfloat16()
         for n, s in (("up", (ff, hidden)), ("down", (hidden, ff)), ("up.b", (ff,)), ("down.b", (hidden,)))}
    w["f.down.b"] = (w["f.down.b"].float() * 10).bfloat16()
    x = torch.randn(90, hidden, generator=g).bfloat16()
    want = plain.dense_ff(x.double(), {k: v.double() for k, v in w.items()}, "f.")
    for gone in ("f.up.b", "f.down.b"):
        assert _rel(plain.dense_ff(x.double(), {k: v.double() * (k != gone) for k, v in w.items()}, "f."), want) > 0.05
    got, _, _ = _run_feed_forward(spec, w, x, dtype)
    assert _rel(got, want) < MIX_TOL[dtype]


@pytest.mark.parametrize("M,N,K", [(1, 128, 64), (7, 200, 72), (16, 2048, 512), (30, 300, 2048), (64, 2048, 6144), (128, 384, 128), (128, 1000, 4096),
                                   (129, 96, 64), (300, 2048, 512), (513, 250, 1024), (600, 512, 6144), (2048, 2048, 2048), (2304, 520, 640)])
@pytest.mark.parametrize("split_mode", [0, 1, 2, 4])
def test_biases_and_exact_gelu_in_every_path_of_the_product(M, N, K, split_mode):
    """K in one part and in several (clusters, atomics into scratch and into the residual, units of a persistent walk, pairs
    of SMs), token tiles of 16 to 128 and whole prompts, widths that are no multiple of a tile: the bias joins once."""
    from ember_b200 import ops
    g = torch.Generator().manual_seed(M + N)
    a, w = torch.randn(M, K, generator=g).bfloat16(), (K ** -0.5 * torch.randn(N, K, generator=g)).bfloat16()
    bias, start = torch.randn(N, generator=g), torch.randn(M, N, generator=g)
    dev = "cuda"
    z = (a.to(dev).double() @ w.to(dev).double().T + bias.to(dev).double()).cpu()
    ad, wd, bd = a.to(dev), w.to(dev), bias.to(dev)
    for epi, want, tol in ((ops.EPI_STORE, z, 5e-3), (ops.EPI_STORE_F32, z, 1e-5), (ops.EPI_GELU, plain.gelu(z), 5e-3),
                           (ops.EPI_ADD_F32, z + start.double(), 1e-5)):
        out = start.to(dev).to(torch.bfloat16 if epi in (ops.EPI_STORE, ops.EPI_GELU) else torch.float32).clone()
        ops.gemm_tc(ad, wd, out, M, epi, split_mode=split_mode, bias=bd)
        assert _rel(out.cpu(), want) < tol, (epi, split_mode)
        if split_mode == 0:
            out = start.to(dev).to(out.dtype).clone()
            ops.gemm_simt(ad, wd, out, M, epi, bias=bd)
            assert _rel(out.cpu(), want) < tol, (epi, "simt")


ROUTED_CASES = [
    # hidden, ff, experts, top, groups
    (64, 40, 6, 2, (3, 2)), (100, 30, 3, 3, None), (96, 24, 5, 1, (5, 1)), (128, 256, 48, 4, (8, 3)), (64, 50, 8, 2, (4, 2)),
    (64, 32, 6, 3, (2, 1)), (64, 16, 1, 1, (1, 1)), (72, 20, 64, 6, (32, 20)),
]


def _routed(hidden, ff, experts, top, groups, seed, spread=4.0):
    from ember_b200.config import RoutedMLPSpec
    spec = RoutedMLPSpec(hidden_size=hidden, intermediate_size=ff, experts=experts, top=top, limit=0.0, alpha=1.0, up_offset=0.0,
                         scoring="sigmoid", correction=False, renormalize=True, renorm_eps=1e-20, groups=groups[0] if groups else 0,
                         keep_groups=groups[1] if groups else 0, group_score="top2")
    g = torch.Generator().manual_seed(seed)
    w = {"f.router": (spread * 0.1 * torch.randn(experts, hidden, generator=g)).bfloat16()}
    for e in range(experts):
        for n, s in (("gate", (ff, hidden)), ("up", (ff, hidden)), ("down", (hidden, ff))):
            w[f"f.e{e}.{n}"] = (0.3 * torch.randn(s, generator=g)).bfloat16()
    router = {"experts": experts, "top": top}
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return spec, w, {"kind": "moe", "expert": {"ff": ff}, "router": router}


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hidden,ff,experts,top,groups", ROUTED_CASES)
def test_routed_feed_forward_alone(dtype, hidden, ff, experts, top, groups):
    """Sigmoid scores divided by their sum, groups kept and dropped by their two best scores, groups of one and of all, as
    many choices as experts, forty-eight and sixty-four experts (more than a warp has lanes), thirty-two groups."""
    spec, w, mlp = _routed(hidden, ff, experts, top, groups, seed=experts + top)
    x = torch.randn(90, hidden, generator=torch.Generator().manual_seed(5)).bfloat16()
    W = {k: v.double() for k, v in w.items()}
    want = plain.moe_ff(x.double(), W, "f.", mlp)
    if groups and 1 < groups[1] < groups[0]:
        free, _ = plain.route(x.double(), W, "f.", {"experts": experts, "top": top})
        kept, _ = plain.route(x.double(), W, "f.", mlp["router"])
        assert (free.sort(-1).values != kept.sort(-1).values).any()
    got, _, _ = _run_feed_forward(spec, w, x, dtype)
    errs = sorted(_rel(got[t], want[t]) for t in range(90))
    # a token whose choice is a close call may fall the other way in bfloat16 (the router reads the rounded input)
    assert errs[len(errs) // 2] < MIX_TOL[dtype] and errs[-3 if dtype == torch.bfloat16 else -1] < 10 * MIX_TOL[dtype]


@pytest.mark.parametrize("E,groups,keep,top", [(12, 4, 2, 3), (40, 5, 2, 4), (96, 3, 1, 6), (6, 6, 3, 2), (64, 32, 3, 4)])
def test_the_router_on_the_device_chooses_what_the_plain_one_does(E, groups, keep, top):
    """The choices themselves, from given logits: a group with one high score and nothing beside it loses against two good
    ones; groups wider than a warp; groups of one."""
    from ember_b200 import ops
    T = 128
    logits = (2.0 * torch.randn(T, E, generator=torch.Generator().manual_seed(E))).float()
    logits[: T // 2, 0] = 9.0
    logits[: T // 2, 1: E // groups] = -9.0                                   # group 0: one score near 1, the others near 0
    chosen, weights = plain.route(logits.double(), {"r.router": torch.eye(E, dtype=torch.float64)}, "r.",
                                  {"experts": E, "top": top, "groups": {"count": groups, "keep": keep}})
    sel = torch.zeros(T * top, dtype=torch.int32, device="cuda")
    wgt = torch.zeros(T * top, dtype=torch.float32, device="cuda")
    ops.moe_route(logits.cuda(), T, top, sel, wgt, rule=(None, 1.0, True, "sigmoid", groups, keep, "top2", 1e-20))
    torch.cuda.synchronize()
    same = [sorted(a) == sorted(b) for a, b in zip(sel.view(T, top).cpu().tolist(), chosen.tolist())]
    assert sum(same) >= T - 1                                                # (float32 sums of two scores may tie)
    w = torch.where(torch.tensor(same)[:, None], wgt.view(T, top).cpu().double().sort(-1).values - weights.sort(-1).values, torch.zeros(()).double())
    assert float(w.abs().max()) < 1e-6
    if E // groups > 1:
        largest, _ = plain.route(logits.double(), {"r.router": torch.eye(E, dtype=torch.float64)}, "r.", {"experts": E, "top": top})
        assert (largest[: T // 2] == 0).any() and not (chosen[: T // 2] == 0).all(-1).any()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_experts_of_prompt_portions_on_tensor_cores(dtype, tmp_path):
    """A portion of more than 256 tokens takes the per-expert product on the tensor cores in bfloat16 (gathered rows)."""
    att = {"heads": 4, "kv_heads": 2, "dim": 32, "vdim": 32, "scale": 0.18, "softcap": 20.0, "mask": {"size": 150}, "rot": {"dims": 16, "base": 1e4}}
    cfg = {"architecture": "Filanex", "vocab": 300, "width": 128, "norm": {"eps": 1e-5}, "embedding": {"bigram": {"buckets": 97, "mul_prev": 5, "mul_cur": 11}},
           "loop": {"start": 0, "stop": 1, "times": 2},
           "layers": [{"type": "attention", "mixer": att, "mlp": {"kind": "moe", "expert": {"ff": 64}, "router": {"experts": 8, "top": 3, "groups": {"count": 4, "keep": 2}}}},
                      {"type": "attention", "mixer": att, "mlp": {"kind": "dense", "ff": 264}}]}
    d = write_filanex_dir(cfg, str(tmp_path), seed=5)
    inputs = plain_inputs(d)
    toks = np.random.default_rng(3).integers(0, 300, size=420).tolist()
    requests = {"r0": toks}
    want = {"r0": plain.forward(*inputs, toks).numpy()}
    steps = trace_portions(requests, sizes=(300, 2, 118))
    outputs, _ = replay(d, dtype, steps, 448, max_batch_tokens=512)
    assert_close(collect(steps, outputs), want, dtype, "experts on tensor cores")


@pytest.mark.parametrize("N,K", [(96, 64), (512, 200), (1000, 1024), (2048, 512)])
@pytest.mark.parametrize("counts", [(0, 1, 127, 128, 129, 0), (300,), (5, 700, 0, 0, 33, 256, 2, 64), tuple([3] * 200)])
def test_grouped_products_in_one_launch(N, K, counts):
    """Rows in groups against weights of their own: empty groups, groups of one row, of a tile exactly and of a row more, two
    hundred groups; rows behind the last group stay as they are.  Stored in fp32 and bfloat16, and silu(gate) up."""
    from ember_b200 import ops
    g = torch.Generator().manual_seed(N + len(counts))
    G, M = len(counts), sum(counts) + 7
    a = torch.randn(M, K, generator=g).bfloat16().cuda()
    w = (K ** -0.5 * torch.randn(G, N, K, generator=g)).bfloat16().cuda()
    bounds = [0]
    for c in counts:
        bounds.append(bounds[-1] + c)
    offsets = torch.tensor(bounds, dtype=torch.int32, device="cuda")
    err = torch.zeros(1, dtype=torch.int32, device="cuda")
    z = torch.cat([a[bounds[i]:bounds[i + 1]].double() @ w[i].double().T for i in range(G)])
    for epi, want, dt, tol in ((ops.EPI_STORE_F32, z, torch.float32, 1e-5), (ops.EPI_STORE, z, torch.bfloat16, 5e-3),
                               (ops.EPI_SILU_MUL, torch.nn.functional.silu(z[:, 0::2]) * z[:, 1::2], torch.bfloat16, 5e-3)):
        out = torch.full((M, want.shape[1]), 7.0, dtype=dt, device="cuda")
        ops.gemm_tc_grouped(a, w, out, M, offsets, epi, err=err)
        assert _rel(out[:bounds[-1]].cpu(), want.cpu()) < tol, epi
        assert float((out[bounds[-1]:].float() - 7.0).abs().max()) == 0.0
    assert int(err.item()) == 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_router_of_long_steps_is_the_router_of_short_ones(dtype):
    """From 1,024 tokens on a block routes four tokens: the same choices and weights, bit by bit, as in steps of 500."""
    from ember_b200 import ops
    T, E, K, top = 1303, 24, 132, 3
    g = torch.Generator().manual_seed(4)
    x, w = torch.randn(T, K, generator=g).to(dtype).cuda(), torch.randn(E, K, generator=g).cuda()
    rule = (None, 1.0, True, "sigmoid", 6, 2, "top2", 1e-20)
    outs = []
    for pieces in ((T,), (500, 500, T - 1000)):
        sel, wgt, at = torch.zeros(T * top, dtype=torch.int32, device="cuda"), torch.zeros(T * top, device="cuda"), 0
        for n in pieces:
            ops.moe_router(x[at:at + n].contiguous(), w, n, top, sel[at * top:], wgt[at * top:], rule=rule)
            at += n
        outs.append((sel.cpu(), wgt.cpu()))
    assert torch.equal(outs[0][0], outs[1][0]) and torch.equal(outs[0][1], outs[1][1])
