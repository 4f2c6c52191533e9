"""Malusun on the device against the plain implementation: each mechanism alone (fed in portions beside another request), the
scan's state and the convolution's inputs carried from step to step, keys just inside and just outside a window in prompts
and in decoding, a far key that dominates, distance slopes and the fixed sink in every attention kernel, values blended with
an earlier layer's, experts weighed at their input beside a shared expert, relu squared in every path of the products, the
norms around a sublayer in one kernel, whole models under every way of cutting the work, slots and pages used again, long
decoding through captured graphs, and greedy generation through the entry point and its scheduler."""
import numpy as np
import pytest
import torch

from tests.malusun_configs import MALUSUN, drawn_malusun, plain_inputs, write_malusun_dir
from tests.plain import malusun_plain as plain
from tests.replay_helpers import collect, max_live_tokens, trace_mixed, trace_portions, trace_tail_decode, trace_whole
from tests.test_fadosun_gpu import _rel, _weights
from tests.test_pepapel_gpu import _run_mixer
from tests.test_zufusun_gpu import _run_feed_forward, attention_kernel, replay  # noqa: F401  (attention_kernel: a fixture)

pytestmark = pytest.mark.gpu

# A position's error is norm(got - want) / norm(want) over its logits.  Rounding is 1e-6 in float32 and 1e-2 in bfloat16
# except where a router's close call falls the other way.  A fault of a mechanism (a key too many, a lost state, a sink or a
# slope left out, a window's edge one off) is 1e-2 or more in float32 at every position it touches.
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
    return {name: write_malusun_dir(name, str(tmp_path_factory.mktemp("malusun_" + name))) for name in MALUSUN}


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
    return {f"r{i}": rng.integers(0, MALUSUN[name]["json"]["vocab"], size=n).tolist() for i, n in enumerate(lengths)}


LENGTHS = {"a": (1, 2, 37, 130), "b": (3, 18, 65, 110), "c": (2, 70, 140), "d": (1, 25, 90)}


# ------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("page", [16, 64])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(MALUSUN))
@pytest.mark.parametrize("mode", ["whole", "tail", "portions", "mixed"])
def test_replay_modes(name, dtype, mode, page, dirs, plain_logits):
    """Whole prompts, a decoded tail (windows pass over decoded tokens), portions down to two tokens (and single ones), and
    four live requests whose slots and pages are used again, against each request alone in the plain implementation."""
    requests = make_requests(name, LENGTHS[name], seed=5)
    if mode == "mixed":
        requests = make_requests(name, LENGTHS[name] + (40, 21, 66, 9), seed=6)
    steps = {"whole": trace_whole, "tail": lambda r: trace_tail_decode(r, tail=60),
             "portions": lambda r: trace_portions(r, sizes=(7, 2, 19, 1, 3, 33, 2, 16, 5, 64)),
             "mixed": lambda r: trace_mixed(r, live=4, seed=3)}[mode](requests)
    outputs, _ = replay(dirs[name], dtype, steps, max_live_tokens(steps, round_to=page), page_tokens=page)
    assert_close(collect(steps, outputs), plain_logits(name, requests), dtype, f"{name} {mode}")


@pytest.mark.parametrize("seed", range(12))
def test_configurations_drawn_at_random(seed, tmp_path):
    """Layer orders, sizes, head counts, windows and constants drawn from a seed: whole prompts, portions and a mixed batch in
    float32 (the sharper comparison), the mixed batch in bfloat16."""
    cfg = drawn_malusun(seed)
    d = write_malusun_dir(cfg, str(tmp_path), seed=seed)
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
            assert_close(collect(steps, outputs), want, dtype, f"drawn {seed} {mode}", over=0.15)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_through_graphs_equals_the_prompt(dtype, dirs, plain_logits):
    """300 tokens one by one (captured graphs after the second step; state rows, carried inputs, blended values, the router's
    grouping and the pages that go back all inside them) against the whole sequence."""
    requests = make_requests("a", (300,), seed=11)
    steps = trace_tail_decode(requests, tail=299)
    outputs, runner = replay(dirs["a"], dtype, steps, 320)
    assert runner.graph_replays > 250
    assert_close(collect(steps, outputs), plain_logits("a", requests), dtype, "long decoding")
    eager, _ = replay(dirs["a"], dtype, steps, 320, cuda_graphs=False)
    assert max(float(np.abs(outputs[k] - eager[k]).max()) for k in outputs) < (1e-5 if dtype == "float32" else 1e-1)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_long_prompt_then_decoding(dtype, dirs, plain_logits):
    """900 tokens at a real model's head sizes: windows of 100, 256 and 300 whose edges pass inside portions, a scan of hundreds
    of tokens: as one prompt with a decoded tail and as portions of 400."""
    requests = make_requests("c", (900,), seed=17)
    for steps in (trace_tail_decode(requests, tail=24), trace_portions(requests, sizes=(400, 37, 400, 2))):
        outputs, _ = replay(dirs["c"], dtype, steps, 960, page_tokens=64, max_batch_tokens=1024)
        assert_close(collect(steps, outputs), plain_logits("c", requests), dtype, "long prompt")


def test_a_request_longer_than_the_pool(dirs, plain_logits):
    """Every attention layer of this model has a window: a pool of 512 tokens serves a request of 800, because the pages the
    windows have passed come back while it runs."""
    requests = make_requests("c", (800,), seed=19)
    steps = trace_portions(requests, sizes=(64, 30, 1, 1, 50))
    outputs, _ = replay(dirs["c"], "float32", steps, 512, page_tokens=16)
    assert_close(collect(steps, outputs), plain_logits("c", requests), "float32", "longer than the pool")


@pytest.mark.parametrize("name", ["a", "b", "d"])
def test_a_slot_used_again_starts_anew(name, dirs, plain_logits):
    """One slot only: the second request gets the pages the first left and the slot with the first's state in it."""
    requests = make_requests(name, (90, 75, 1, 33), seed=21)
    steps = trace_portions(requests, sizes=(40, 3, 1, 31))
    outputs, _ = replay(dirs[name], "float32", steps, 96, max_requests=1)
    assert_close(collect(steps, outputs), plain_logits(name, requests), "float32", "one slot")


@pytest.mark.parametrize("name", ["a", "b"])
def test_greedy_generation_through_the_engine(name, dirs):
    """Greedy tokens from ``ember_b200.load(...).generate`` (scheduler, portions of 16, few pages, four prompts of unequal
    length, three slots) against greedy decoding with the plain implementation."""
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


def test_generation_under_preemption_starts_states_anew(dirs):
    """So few pages that requests are preempted and admitted again into used slots: the same tokens as with room for all."""
    import ember_b200
    prompts = list(make_requests("b", (30, 28, 35, 31), seed=33).values())
    outs = []
    for tokens in (1024, 144):
        llm = ember_b200.load(dirs["b"], dtype="float32", kv_cache_tokens=tokens, max_batch_tokens=64, max_seqs=4, prefill_chunk=16, page_tokens=16)
        outs.append(llm.generate(prompts, max_tokens=40, ignore_eos=True))
        preempted = llm.engine.stats.preemptions
    assert preempted > 0 and outs[0] == outs[1]


# ---------------------------------------------------------------------------------- the scan, alone
SCAN_CASES = [
    # hidden, inner, state, dt_rank, conv
    (64, 96, 16, 8, 4), (100, 77, 5, 3, 2), (128, 256, 24, 16, 3), (72, 40, 1, 1, 1), (64, 33, 40, 12, 6), (96, 130, 128, 8, 4), (64, 48, 200, 5, 9),
    (64, 128, 8, 128, 4), (64, 64, 33, 64, 2)]


def _scan_weights(spec, seed):
    w = _weights(spec, seed=seed, std=0.15)
    g = torch.Generator().manual_seed(seed + 50)
    w["m.conv.b"] = 0.3 * torch.randn(w["m.conv.b"].shape, generator=g)
    w["m.x"] = 2.0 * w["m.x"]
    w["m.dt.b"] = -3.0 + 1.5 * torch.randn(w["m.dt.b"].shape, generator=g)
    return {k: v.bfloat16() for k, v in w.items()}


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hidden,inner,state,dt_rank,conv", SCAN_CASES)
@pytest.mark.parametrize("portions", [((150, 7),), ((40, 7), (3, 1), (1, 1), (2, 2), (64, 19), (1, 1), (33, 1), (6, 3)), ((5, 1),) + ((1, 1),) * 20 + ((125, 2),)])
def test_selective_scan_alone(dtype, hidden, inner, state, dt_rank, conv, portions):
    """From one state a channel to two hundred, channel counts that fill no block, one tap to nine, ranks the tensor cores take
    and not; whole, in portions that end anywhere in a chunk of the kernel, and token by token."""
    from ember_b200.config import SelectiveScanSpec
    spec = SelectiveScanSpec(hidden_size=hidden, inner=inner, state_size=state, dt_rank=dt_rank, conv_taps=conv)
    w = _scan_weights(spec, inner)
    x = torch.randn(150, hidden, generator=torch.Generator().manual_seed(2)).bfloat16()
    want = plain.mamba_mixer(x.double(), {k: v.double() for k, v in w.items()}, "m.", {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv})
    assert _rel(_run_mixer(spec, w, x, dtype, portions=portions), want) < MIX_TOL[dtype]


def test_the_parts_of_the_scan_are_there():
    """Steps, decays, the skip, the gate, the convolution and its bias: each left out of the plain implementation changes the
    result by much more than the tolerance, so does a state or a carried input lost at a portion's edge."""
    from ember_b200.config import SelectiveScanSpec
    spec = SelectiveScanSpec(hidden_size=64, inner=96, state_size=16, dt_rank=8, conv_taps=4)
    w = _scan_weights(spec, 1)
    W = {k: v.double() for k, v in w.items()}
    x = torch.randn(100, 64, generator=torch.Generator().manual_seed(4)).bfloat16()
    m = {"inner": 96, "state": 16, "dt_rank": 8, "conv": 4}
    want = plain.mamba_mixer(x.double(), W, "m.", m)
    for name, t in (("m.D", torch.zeros(96)), ("m.A_log", torch.full((96, 16), -9.0)), ("m.dt", torch.zeros(96, 8)), ("m.conv.b", torch.zeros(96)),
                    ("m.dt.b", torch.full((96,), -1.0)), ("m.conv", torch.tensor([[0.0, 0.0, 0.0, 1.0]]).repeat(96, 1))):
        assert _rel(plain.mamba_mixer(x.double(), {**W, name: t.double()}, "m.", m), want) > 0.02, name
    anew = plain.mamba_mixer(x[50:].double(), W, "m.", m)                     # nothing carried over position 50
    assert _rel(anew[0], want[50]) > 0.05 and _rel(anew[5], want[55]) > 0.01
    for portions in (((50, 3), (50, 1)), ((49, 1), (1, 1), (1, 1), (49, 9))):
        got = _run_mixer(spec, w, x, torch.float32, portions=portions)
        for t in (48, 49, 50, 51, 55, 99):
            assert _rel(got[t], want[t]) < 1e-4, t


@pytest.mark.parametrize("C,taps,col,ld", [(64, 2, 0, 64), (64, 3, 4, 80), (37, 4, 3, 50), (128, 4, 0, 130), (66, 4, 0, 66), (24, 6, 0, 24)])
@pytest.mark.parametrize("silu", [True, False])
def test_convolution_over_runs_and_steps(C, taps, col, ld, silu):
    """Runs of one and of several tokens beside one another (blocks of several tokens cross runs in long steps), four channels a
    thread and one, taps in registers and not; the carried inputs after every step; the rounded copy."""
    from ember_b200 import ops
    g = torch.Generator().manual_seed(C + taps)
    dev = "cuda"
    w, b = torch.randn(C, taps, generator=g), torch.randn(C, generator=g)
    n = 700
    seqs = {s: torch.randn(n, C, generator=g) for s in range(3)}
    act = plain.silu if silu else (lambda z: z)
    want = {s: act(plain.causal_conv(x.double(), w.double(), b.double())) for s, x in seqs.items()}
    carry = torch.zeros(5, 8 + (taps - 1) * C, device=dev)
    slot, at = {0: 4, 1: 0, 2: 2}, {0: 0, 1: 0, 2: 0}
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)            # noqa: E731
    for step in ([(0, 5), (1, 1), (2, 2)], [(0, 1), (1, 1), (2, 1)], [(2, 330), (0, 3), (1, 40)], [(1, 1), (0, 1)], [(0, 600), (2, 300), (1, 500)],
                 [(2, 1)]):
        rows, seq, qs = [], [], [0]
        for i, (s, k) in enumerate(step):
            rows.append(seqs[s][at[s]:at[s] + k])
            seq += [i] * k
            qs.append(qs[-1] + k)
        T = qs[-1]
        x = torch.randn(T, ld, generator=g)
        x[:, col:col + C] = torch.cat(rows)
        out, rounded = torch.zeros(T, C, device=dev), torch.zeros(T, C, device=dev, dtype=torch.bfloat16)
        ops.conv_silu(x.to(dev), col, w.to(dev), b.to(dev), carry, 8, i32(seq), i32(qs), i32([slot[s] for s, _ in step]), out, T, len(step),
                      silu=silu, rounded=rounded)
        got = out.cpu()
        assert torch.equal(rounded.cpu(), got.bfloat16())
        for i, (s, k) in enumerate(step):
            assert _rel(got[qs[i]:qs[i + 1]], want[s][at[s]:at[s] + k]) < 2e-6, (step, s)
            at[s] += k
            last = torch.cat([torch.zeros(taps - 1, C), seqs[s][:at[s]]])[-(taps - 1):] if taps > 1 else torch.zeros(0, C)
            assert torch.equal(carry[slot[s], 8:].cpu().view(taps - 1, C), last)
    assert float(carry[[1, 3]].abs().max()) == 0.0


# -------------------------------------------------------------------------------------- attention, alone
def _spec(kind, heads, kv, dim, vdim, hidden, scale=0.2, window=0, rot=None, value_mix=""):
    from ember_b200.config import NoPositionSpec, RotarySpec, SinkAttentionSpec
    second = kind == "attention_2"
    pos = RotarySpec(head_dim=dim, rotary_dim=rot[0], theta=rot[1], frequency_precision="float64") if rot else NoPositionSpec()
    return SinkAttentionSpec(hidden_size=hidden, num_heads=heads, num_kv_heads=kv, head_dim=dim, value_dim=vdim, scale=scale, window=window,
                             bias=second, sink=second, fixed_sink=0.0 if second else None, slope_span=8.0 if second else 0.0, position=pos,
                             value_mix=value_mix)


def _m(heads, kv, dim, vdim, scale=0.2, window=0, rot=None, v_mix=False):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix}
    if window:
        m["mask"] = {"size": window}
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    return m


def _attention_weights(spec, seed, std=0.15):
    w = _weights(spec, seed=seed, std=std)
    g = torch.Generator().manual_seed(seed + 50)
    return {k: (0.5 * torch.randn(v.shape, generator=g) if k.endswith(".b") else v).bfloat16() for k, v in w.items()}


def _want(kind, x, w, m, shared=None):
    return plain.attention_mixer(x.double(), {k: v.double() for k, v in w.items()}, "m.", kind, m, {} if shared is None else shared)


MIXER_CASES = [
    ("attention", 6, 2, 16, 24, 64, 20, (16, 1e4)), ("attention", 4, 1, 20, 12, 100, 16, (8, 77.0)), ("attention", 3, 3, 18, 300, 72, 0, (2, 10.0)),
    ("attention", 40, 1, 8, 8, 64, 33, None), ("attention", 1, 1, 48, 16, 64, 1, (46, 500.0)),
    ("attention_2", 6, 2, 16, 24, 64, 20, None), ("attention_2", 4, 1, 20, 12, 100, 16, None), ("attention_2", 1, 1, 32, 32, 64, 0, None),
    ("attention_2", 40, 1, 8, 16, 64, 33, None), ("attention_2", 3, 3, 64, 32, 64, 1, None), ("attention_2", 9, 3, 128, 48, 128, 64, None),
    ("attention_2", 7, 7, 24, 40, 64, 2, None)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("kind,heads,kv,dim,vdim,hidden,window,rot", MIXER_CASES)
def test_attention_alone(dtype, kind, heads, kv, dim, vdim, hidden, window, rot, attention_kernel):
    """Both kinds: partial rotations, windows of one key to none, values wider and narrower than keys, forty query heads on one
    key head, head counts that are no power of two (the slopes' exponents are then no integers), biases."""
    spec = _spec(kind, heads, kv, dim, vdim, hidden, 0.5, window, rot)
    w = _attention_weights(spec, heads)
    x = torch.randn(90, hidden, generator=torch.Generator().manual_seed(2)).bfloat16()
    want = _want(kind, x, w, _m(heads, kv, dim, vdim, 0.5, window, rot))
    assert _rel(_run_mixer(spec, w, x, dtype), want) < MIX_TOL[dtype]


@pytest.mark.parametrize("dense", [True, False], ids=["TMA-fed kernels", "shared-row kernels"])
@pytest.mark.parametrize("kind,heads,kv,dim,window,rot", [
    ("attention", 8, 1, 128, 50, (64, 1e4)), ("attention", 4, 2, 64, 64, (64, 500.0)), ("attention", 12, 4, 128, 90, None),
    ("attention_2", 8, 1, 128, 50, None), ("attention_2", 4, 2, 64, 64, None), ("attention_2", 12, 4, 128, 0, None),
    ("attention_2", 16, 1, 64, 130, None), ("attention_2", 4, 4, 128, 7, None), ("attention_2", 2, 2, 128, 1, None)])
def test_layers_on_the_engines_dense_attention_kernels(dense, kind, heads, kv, dim, window, rot, monkeypatch):
    """Keys and values of one size, 64 or 128: bfloat16 steps go to the kernels Qwen3's attention uses, which take the window,
    the slopes and the sink (a group of three query heads a key head takes the mma.sync form for portions too); switched off,
    the same layer runs on the shared-row kernels."""
    from ember_b200.parts.sink_attention import SinkAttention
    monkeypatch.setattr(SinkAttention, "DENSE_KERNELS", dense)
    spec = _spec(kind, heads, kv, dim, dim, 128, 0.5, window, rot)
    w = _attention_weights(spec, heads)
    x = torch.randn(200, 128, generator=torch.Generator().manual_seed(8)).bfloat16()
    want = _want(kind, x, w, _m(heads, kv, dim, dim, 0.5, window, rot))
    got = _run_mixer(spec, w, x, torch.bfloat16, portions=((130, 3), (60, 20), (1, 1), (1, 1), (1, 1), (7, 2)))
    assert _rel(got, want) < MIX_TOL[torch.bfloat16]
    for t in (0, 1, 6, 7, 49, 50, 51, 63, 64, 65, 127, 128, 129, 130, 189, 190, 191, 192, 193, 199):
        assert _rel(got[t], want[t]) < 3 * MIX_TOL[torch.bfloat16], t


@pytest.mark.parametrize("merge", ["one split", "cluster", "buffers"])
@pytest.mark.parametrize("window,at,softcap,sink", [(0, 1399, 0.0, 0.0), (700, 1399, 0.0, 2.0), (0, 900, 6.0, -1.0), (300, 310, 0.0, 40.0), (0, 5, 0.0, 0.0)])
def test_single_tokens_over_split_keys_with_slopes_and_a_sink(window, at, softcap, sink, merge):
    """A decoded token's keys in one split and in several, merged in a cluster or through buffers: the slopes count distances
    from the token in every split, the sink joins once, whatever its size."""
    from ember_b200 import ops
    heads, kv, dim, page = 4, 2, 128, 16
    g = torch.Generator().manual_seed(at)
    n = at + 1
    q = torch.randn(1, heads, dim, generator=g).bfloat16()
    k, v = torch.randn(n, kv, dim, generator=g).bfloat16(), torch.randn(n, kv, dim, generator=g).bfloat16()
    slopes, sinks = torch.tensor([0.25, 0.01, 0.002, 0.0]), sink + torch.arange(heads) * 0.5
    pages = (n + page - 1) // page
    order = torch.randperm(pages, generator=g)
    kp, vp = (torch.zeros(pages, kv, page, dim, dtype=torch.bfloat16) for _ in range(2))
    for p in range(n):
        kp[order[p // page], :, p % page], vp[order[p // page], :, p % page] = k[p], v[p]
    dev = "cuda"
    out = torch.zeros(1, heads, dim, dtype=torch.bfloat16, device=dev)
    splits, keys = (1, 0) if merge == "one split" else (6, 256)
    kw = dict(part_o=torch.zeros(heads * splits * dim, device=dev), part_ml=torch.zeros(heads * splits * 2, device=dev)) if merge == "buffers" else {}
    tiles = torch.tensor([[0, 0, 1, at]], dtype=torch.int32, device=dev)
    ops.attention_tc(q.to(dev), kp.to(dev), vp.to(dev), out, 1, heads, kv, dim, tiles, 1, order.to(torch.int32)[None].to(dev), page, window, 0.3,
                     splits, keys, softcap=softcap, slopes=slopes.to(dev), sink=sinks.to(dev), **kw)
    torch.cuda.synchronize()
    want = torch.zeros(heads, dim, dtype=torch.float64)
    gap = (at - torch.arange(n)).double()
    for h in range(heads):
        s = (k[:, h // 2].double() @ q[0, h].double()) * 0.3
        s = softcap * torch.tanh(s / softcap) if softcap else s
        s = s - float(slopes[h]) * gap
        if window:
            s = s.masked_fill(gap >= window, float("-inf"))
        p = torch.softmax(torch.cat([s, sinks[h:h + 1].double()]), 0)[:-1]
        want[h] = p @ v[:, h // 2].double()
    for h in range(heads):
        if float(want[h].norm()) > 1e-4:
            assert _rel(out[0, h].cpu(), want[h]) < 1.5e-2, h
        else:
            assert float(out[0, h].float().norm()) < 2e-4, h


@pytest.mark.parametrize("kind", ["attention", "attention_2"])
@pytest.mark.parametrize("portions", [((150, 3),), ((40, 3), (1, 1), (1, 1), (1, 1), (37, 30), (2, 1), (68, 1)),
                                      ((38, 1),) + ((1, 1),) * 5 + ((35, 1),) + ((1, 1),) * 5 + ((35, 1),) + ((1, 1),) * 5 + ((27, 1),)])
def test_keys_just_inside_and_just_outside_a_window(kind, portions):
    """A window of 40 with pages of 16.  Value 30 stands out and query t sees it up to t = 69: with the window's edge one off,
    position 69 would lose it or 70 would gain it.  Checked row by row around that edge and at the first tokens."""
    spec = _spec(kind, 2, 1, 16, 16, 64, 0.2, 40)
    w = _attention_weights(spec, 4, std=0.1)
    x = torch.randn(150, 64, generator=torch.Generator().manual_seed(6))
    x[30] *= 12.0
    x = x.bfloat16()
    m = _m(2, 1, 16, 16, 0.2, 40)
    w["m.q"] = 0.05 * w["m.q"]                               # near-even weights: the far key is not lost among them
    want = _want(kind, x, w, m)
    for off, at in ((39, 69), (41, 70)):
        assert _rel(_want(kind, x, w, {**m, "mask": {"size": off}})[at], want[at]) > 0.02
    got = _run_mixer(spec, w, x, torch.float32, portions=portions)
    for t in (0, 1, 2, 29, 30, 31, 38, 39, 40, 41, 68, 69, 70, 71, 79, 80, 110, 149):
        assert _rel(got[t], want[t]) < 1e-4, t
    assert _rel(got, want) < 1e-4


def test_slopes_the_sink_and_the_biases_are_there():
    """Each left out of the plain implementation changes the result by much more than the tolerance; so does the other reading
    of the slopes (slope j instead of slope (i - j)), which the sink tells apart."""
    spec = _spec("attention_2", 4, 2, 32, 32, 64, 0.3, 50)
    w = _attention_weights(spec, 3)
    W = {k: v.double() for k, v in w.items()}
    x = torch.randn(120, 64, generator=torch.Generator().manual_seed(4)).bfloat16()
    m = _m(4, 2, 32, 32, 0.3, 50)
    want = _want("attention_2", x, w, m)
    for b in ("m.q.b", "m.k.b", "m.v.b"):
        assert _rel(_want("attention_2", x, {**w, b: torch.zeros_like(w[b])}, m), want) > 0.02, b
    assert _rel(plain.attention_mixer(x.double(), {k[:-2] if k.endswith(".b") else k: v for k, v in W.items() if not k.endswith(".b")}, "m.",
                                      "attention", m, {}), want) > 0.2
    for portions in (((120, 3),), ((49, 1), (1, 1), (1, 1), (1, 1), (2, 1), (66, 30))):
        assert _rel(_run_mixer(spec, w, x, torch.float32, portions=portions), want) < MIX_TOL[torch.float32]


@pytest.mark.parametrize("portions", [((200, 3),), ((120, 3), (40, 30), (38, 1), (1, 1), (1, 1)), ((2, 1),) * 50 + ((100, 1),)])
def test_a_far_key_that_dominates_is_seen_across_pages_and_portions(portions):
    """A window of 300: key 5 is made large along the direction the late queries point in, so that among two hundred keys it
    has most of the weight in spite of its distance; lost (a page given back too early) the result changes wholly."""
    spec = _spec("attention_2", 2, 1, 16, 24, 64, 1.5, 300)
    w = _attention_weights(spec, 4, std=0.1)
    x = torch.randn(200, 64, generator=torch.Generator().manual_seed(6))
    x[150:] = x[5] + 0.3 * x[150:]
    x[5] *= 6.0
    x = x.bfloat16()
    w["m.q"], w["m.q.b"] = w["m.k"].repeat(2, 1), torch.zeros(32).bfloat16()
    m = _m(2, 1, 16, 24, 1.5, 300)
    want = _want("attention_2", x, w, m)
    gone = x.clone()
    gone[5] = 0
    assert min(_rel(a, b) for a, b in zip(_want("attention_2", gone, w, m)[150:], want[150:])) > 0.1
    assert _rel(_run_mixer(spec, w, x, torch.float32, portions=portions), want) < 1e-4


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("vdim,kv", [(24, 2), (64, 1), (10, 3)])
def test_values_blend_with_the_source_layers_for_the_same_token(dtype, vdim, kv):
    """A source layer and two that blend, of both kinds, run one after the other on inputs of their own in portions beside
    another request: the cached values are the blended ones (later portions read them), the source's are its own."""
    from ember_b200.parts import build_part
    from tests.test_parts_gpu import Bench, store_of
    hidden = 64
    kinds = (("attention_2", "source"), ("attention", "mix"), ("attention_2", "mix"))
    specs = [_spec(k, 2 * kv, kv, 64, vdim, hidden, 0.3, 30, (16, 1e3) if k == "attention" else None, mix) for k, mix in kinds]
    ws = [_attention_weights(s, 7 + i) for i, s in enumerate(specs)]
    g = torch.Generator().manual_seed(vdim)
    xs = [torch.randn(100, hidden, generator=g).bfloat16() for _ in specs]
    for w, lam in zip(ws[1:], (0.7, 0.4)):
        w["m.vmix"] = torch.tensor(lam).bfloat16()
    shared, want = {}, []
    for (k, _), s, w, x in zip(kinds, specs, ws, xs):
        want.append(_want(k, x, w, _m(2 * kv, kv, 64, vdim, 0.3, 30, (16, 1e3) if k == "attention" else None, True), shared))
    alone = [_want(k, x, w, _m(2 * kv, kv, 64, vdim, 0.3, 30, (16, 1e3) if k == "attention" else None)) for (k, _), x, w in zip(kinds, xs, ws)]
    assert _rel(alone[0], want[0]) < 1e-12 and _rel(alone[1], want[1]) > 0.2 and _rel(alone[2], want[2]) > 0.1
    parts = [build_part("mixer", s, "m.") for s in specs]
    b = Bench({i: p.cache_need() for i, p in enumerate(parts)}, dtype, capacity=512)
    for p, w in zip(parts, ws):
        p.load(store_of(w), b.rt)
    got = [torch.zeros(100, hidden) for _ in parts]
    at = 0
    for n, m in ((37, 5), (1, 2), (1, 1), (2, 30), (59, 1)):
        ctx = b.ctx([("o", m), ("x", n)], tile_sizes=tuple(k for p in parts for k in p.tile_requests()))
        for i, p in enumerate(parts):
            x = torch.zeros(256, hidden, device=b.dev, dtype=dtype)
            x[:m] = torch.randn(m, hidden, generator=g).to(dtype)
            x[m:m + n] = xs[i][at:at + n].to(dtype)
            out = torch.full((256, hidden), 7.0, device=b.dev)
            p.forward(ctx, x, out, b.storage.layer(i), accumulate=False)
            got[i][at:at + n] = out[m:m + n].cpu()
        at += n
    assert at == 100 and int(b.err.item()) == 0
    for i in range(3):
        assert _rel(got[i], want[i]) < MIX_TOL[dtype], i


# ------------------------------------------------------------------------------------------ feed-forwards
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hidden,ff", [(64, 40), (100, 30), (128, 256), (72, 1000)])
def test_dense_feed_forward_alone(dtype, hidden, ff):
    from ember_b200.config import MLPSpec
    spec = MLPSpec(hidden_size=hidden, intermediate_size=ff, names=("up", "down"), activation="square_relu")
    g = torch.Generator().manual_seed(ff)
    w = {f"f.{n}": (0.3 * torch.randn(s, generator=g)).bfloat16() for n, s in (("up", (ff, hidden)), ("down", (hidden, ff)))}
    x = torch.randn(90, hidden, generator=g).bfloat16()
    want = plain.dense_ff(x.double(), {k: v.double() for k, v in w.items()}, "f.")
    got, _, _ = _run_feed_forward(spec, w, x, dtype)
    assert _rel(got, want) < MIX_TOL[dtype]


@pytest.mark.parametrize("M,N,K", [(1, 128, 64), (7, 200, 72), (16, 2048, 512), (30, 300, 2048), (64, 2048, 6144), (128, 384, 128), (128, 1000, 4096),
                                   (129, 96, 64), (300, 2048, 512), (513, 250, 1024), (2048, 2048, 2048), (2304, 520, 640)])
@pytest.mark.parametrize("split_mode", [0, 1, 2, 4])
def test_square_relu_in_every_path_of_the_product(M, N, K, split_mode):
    """K in one part and in several, token tiles of 16 to 128 and whole prompts, widths that are no multiple of a tile."""
    from ember_b200 import ops
    g = torch.Generator().manual_seed(M + N)
    a, w = torch.randn(M, K, generator=g).bfloat16().cuda(), (K ** -0.5 * torch.randn(N, K, generator=g)).bfloat16().cuda()
    want = (torch.relu(a.double() @ w.double().T) ** 2).cpu()
    for fn in ("tc",) + (("simt",) if split_mode == 0 else ()):
        out = torch.zeros(M, N, dtype=torch.bfloat16, device="cuda")
        if fn == "tc":
            ops.gemm_tc(a, w, out, M, ops.EPI_SQUARE_RELU, split_mode=split_mode)
        else:
            ops.gemm_simt(a, w, out, M, ops.EPI_SQUARE_RELU)
        assert _rel(out.cpu(), want) < 5e-3, fn


@pytest.mark.parametrize("M,N,K", [(129, 160, 1024), (300, 130, 2048), (2048, 160, 4096), (700, 512, 1088), (2100, 96, 1024), (64, 160, 4096), (300, 600, 2048)])
@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_narrow_products_of_prompt_portions(M, N, K, dtype):
    """Few columns and many tokens: added into zeros with K in parts (whatever the buffer held), or stored."""
    from types import SimpleNamespace
    from ember_b200.parts.linear import Linear
    g = torch.Generator().manual_seed(M + N)
    a, w = torch.randn(M, K, generator=g).to(dtype).cuda(), (K ** -0.5 * torch.randn(N, K, generator=g)).to(dtype).cuda()
    out = torch.full((M + 1, N), 7.0, device="cuda")
    Linear(w).store_f32(SimpleNamespace(err=None, stream=None), a, out, M)
    assert _rel(out[:M].cpu(), (a.double() @ w.double().T).cpu()) < 1e-5 and float((out[M] - 7.0).abs().max()) == 0.0


ROUTED_CASES = [
    # hidden, ff, experts, top, shared
    (64, 40, 6, 2, 32), (100, 30, 3, 3, 50), (96, 24, 5, 1, 0), (128, 256, 48, 4, 128), (64, 50, 8, 1, 64), (64, 16, 1, 1, 8), (72, 20, 64, 6, 0)]


def _routed(hidden, ff, experts, top, shared, seed, spread=1.0):
    from ember_b200.config import RoutedMLPSpec
    spec = RoutedMLPSpec(hidden_size=hidden, intermediate_size=ff, experts=experts, top=top, limit=0.0, alpha=1.0, up_offset=0.0,
                         scoring="sigmoid", weigh="input", shared_size=shared)
    g = torch.Generator().manual_seed(seed)
    w = {"f.router": (spread * 0.1 * torch.randn(experts, hidden, generator=g)).bfloat16()}
    names = [(f"e{e}", ff) for e in range(experts)] + ([("shared", shared)] if shared else [])
    for p, size in names:
        for n, s in (("gate", (size, hidden)), ("up", (size, hidden)), ("down", (hidden, size))):
            w[f"f.{p}.{n}"] = (0.3 * torch.randn(s, generator=g)).bfloat16()
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        mlp["shared"] = {"ff": shared}
    return spec, w, mlp


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hidden,ff,experts,top,shared", ROUTED_CASES)
def test_routed_feed_forward_alone(dtype, hidden, ff, experts, top, shared):
    """Weights on the experts' inputs (not on their outputs: that is far away), a shared expert of another size than the
    others or none, a single choice, as many choices as experts, sixty-four experts; stored and added."""
    spec, w, mlp = _routed(hidden, ff, experts, top, shared, seed=experts + top)
    x = torch.randn(90, hidden, generator=torch.Generator().manual_seed(5)).bfloat16()
    W = {k: v.double() for k, v in w.items()}
    want = plain.moe_ff(x.double(), W, "f.", mlp)
    if top < experts:
        chosen, weights = plain.route(x.double(), W, "f.", top)
        at_output = sum(weights[:, i:i + 1] * torch.cat([plain.expert(x[t:t + 1].double(), W, f"f.e{int(chosen[t, i])}.") for t in range(90)])
                        for i in range(top))
        assert _rel(at_output, want - (plain.expert(x.double(), W, "f.shared.") if shared else 0)) > 0.03
    got, _, _ = _run_feed_forward(spec, w, x, dtype)
    errs = sorted(_rel(got[t], want[t]) for t in range(90))
    # a token whose choice is a close call may fall the other way in bfloat16 (the router reads the rounded input)
    assert errs[len(errs) // 2] < MIX_TOL[dtype] and errs[-3 if dtype == torch.bfloat16 else -1] < 10 * MIX_TOL[dtype]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_experts_of_prompt_portions_on_tensor_cores(dtype, tmp_path):
    """A portion of more than 256 tokens takes the grouped product on the tensor cores in bfloat16 (weighted gathered rows)."""
    att = {"heads": 4, "kv_heads": 2, "dim": 32, "vdim": 32, "scale": 0.18, "mask": {"size": 150}, "v_mix": True}
    moe = {"kind": "moe", "expert": {"ff": 64}, "router": {"experts": 8, "top": 3}, "shared": {"ff": 96}}
    cfg = {"architecture": "Malusun", "vocab": 300, "width": 128, "norm": {"eps": 1e-5}, "embedding": {"scale": 5.0},
           "layers": [{"type": "attention", "mixer": {**att, "rot": {"dims": 16, "base": 1e4}}, "mlp": moe},
                      {"type": "mamba1", "mixer": {"inner": 160, "state": 12, "dt_rank": 16, "conv": 4}, "mlp": {"kind": "dense", "ff": 264}},
                      {"type": "attention_2", "mixer": att, "mlp": moe}]}
    d = write_malusun_dir(cfg, str(tmp_path), seed=5)
    inputs = plain_inputs(d)
    toks = np.random.default_rng(3).integers(0, 300, size=420).tolist()
    requests = {"r0": toks}
    want = {"r0": plain.forward(*inputs, toks).numpy()}
    steps = trace_portions(requests, sizes=(300, 2, 118))
    outputs, _ = replay(d, dtype, steps, 448, max_batch_tokens=512)
    assert_close(collect(steps, outputs), want, dtype, "experts on tensor cores")


# ----------------------------------------------------------------------------------------------- norms
@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows,width", [(1, 64), (5, 100), (33, 2048), (3, 77), (2, 20000)])
def test_norm_add_norm_is_the_three_one_after_the_other(rows, width, out_dtype):
    from ember_b200 import ops
    g = torch.Generator().manual_seed(width)
    y, h = 3.0 * torch.randn(rows, width, generator=g), torch.randn(rows, width, generator=g)
    w1, w2 = 0.3 * torch.randn(width, generator=g), 0.3 * torch.randn(width, generator=g)
    new = h.double() + plain.rms_norm(y.double(), w1, 1e-5)
    want = plain.rms_norm(new, w2, 1e-3)
    hd, out = h.cuda(), torch.zeros(rows + 1, width, dtype=out_dtype, device="cuda")
    ops.norm_add_norm(y.cuda(), (1.0 + w1).cuda(), 1e-5, hd, (1.0 + w2).cuda(), 1e-3, out, rows)
    assert _rel(hd.cpu(), new) < 1e-6 and _rel(out[:rows].cpu(), want) < (1e-6 if out_dtype == torch.float32 else 5e-3)
    assert float(out[rows].float().abs().max()) == 0.0


def test_the_norms_between_layers_ride_on_the_additions(dirs):
    """A step of a Malusun model launches one norm of its own at the start (and the final one): the others are part of the
    kernels that add to the stream, and a layer without a feed-forward hands its successor its rows too."""
    from ember_b200 import StepEntry, ops
    from ember_b200.engine.runner import ModelRunner
    counts = {}
    for name in ("a", "b"):
        runner = ModelRunner.from_dir(dirs[name], dtype="float32", capacity_tokens=64, max_batch_tokens=64, max_requests=1, page_tokens=16)
        calls = []
        norm, both = ops.rmsnorm, ops.norm_add_norm
        ops.rmsnorm = lambda *a, **k: (calls.append("norm"), norm(*a, **k))[1]
        ops.norm_add_norm = lambda *a, **k: (calls.append("both"), both(*a, **k))[1]
        try:
            assert runner.admit("r") and runner.reserve("r", 3)
            runner.step([StepEntry("r", [1, 2, 3], (2,))])
        finally:
            ops.rmsnorm, ops.norm_add_norm = norm, both
        counts[name] = (calls.count("norm"), calls.count("both"))
    assert counts["a"] == (2, 9) and counts["b"] == (2, 8)
