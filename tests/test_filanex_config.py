"""Filanex without a device: reading config.json, the order of runs, the tensors a model declares, what its layers and its
embedding ask of the cache, pages of chunks that have passed, the random-weights folder, the command line, and the plain
implementation's own mechanisms on cases whose answer is known."""
import json
import math

import pytest
import torch

from tests.filanex_configs import FILANEX, drawn_filanex, filanex_config, plain_inputs, write_filanex_dir
from tests.plain import filanex_plain as plain


def test_registered_and_resolved_by_the_architecture_key():
    from ember_b200.config import FilanexConfig, config_from_dict, registered_architectures
    assert "Filanex" in registered_architectures()
    cfg = config_from_dict(FILANEX["a"]["json"])
    assert isinstance(cfg, FilanexConfig) and cfg.width == 128 and cfg.bigram == (211, 7, 3) and cfg.loop == (1, 3, 2)
    for name in FILANEX:
        assert config_from_dict(filanex_config(name).to_json()) == filanex_config(name)
    assert filanex_config("d").bigram is None and filanex_config("d").loop is None and filanex_config("c").bigram is None


def test_run_order_marks_the_first_layer_of_every_pass():
    cfg = filanex_config("a")
    assert cfg.order() == ((0, 0, False), (1, 0, True), (2, 0, False), (1, 1, True), (2, 1, False), (3, 0, False))
    spec = cfg.to_model_spec()
    assert [(e.layer, e.instance, e.reentry) for e in spec.schedule] == list(cfg.order()) and spec.reentry is not None
    assert plain.run_order(FILANEX["a"]["json"]) == [(l, r) for l, _, r in cfg.order()]
    assert [e.reentry for e in filanex_config("c").to_model_spec().schedule] == [False, False, True]       # run once: still mixed
    assert filanex_config("d").to_model_spec().reentry is None


@pytest.mark.parametrize("name", sorted(FILANEX))
def test_cache_needs(name):
    """Pages for every run of every layer, a chunk's worth at a time where there is a mask; one int32 a request for the
    embedding's previous token."""
    from ember_b200.model.causal_lm import CausalLM
    cfg, j = filanex_config(name), FILANEX[name]["json"]
    needs = CausalLM(cfg.to_model_spec()).cache_needs()
    kv = 0
    for i, t, _ in cfg.order():
        m, n = j["layers"][i]["mixer"], needs[i if t == 0 else (i, "", t)]
        chunk = (m.get("mask") or {}).get("size", 0)
        assert (n.kind, n.chunk, n.window) == ("window" if chunk else "full", chunk, 0)
        assert (n.num_kv_heads, n.head_dim, n.value_dim or n.head_dim) == (m["kv_heads"], m["dim"], m["vdim"])
        kv += 2 * m["kv_heads"] * (m["dim"] + m["vdim"])
    bigram = bool((j.get("embedding") or {}).get("bigram"))
    assert ((-1, "bigram") in needs) == bigram
    if bigram:
        n = needs[(-1, "bigram")]
        assert (n.kind, n.state_shape, n.state_dtype) == ("state", (1,), "int32")
    assert cfg.kv_bytes_per_token(2) == kv and cfg.state_bytes_per_request() == (4 if bigram else 0)


def test_pages_of_chunks_that_have_passed_go_back():
    """Chunks of 40 on pages of 16 beside layers that keep everything: once a chunk is full the pages wholly before the next
    chunk's first key are free (its edge lies inside a page: 40 = 2 pages and a half, so that page stays), and never
    one that a later query still sees."""
    from ember_b200.cache.manager import CacheManager
    from ember_b200.parts.base import CacheNeed
    full, chunk = CacheNeed("full", 2, 16), CacheNeed("window", 2, 16, chunk=40)
    m = CacheManager({0: full, 1: chunk}, 16, 400, 2)
    m.admit("a")
    m.admit("b")
    held = 0
    for upto in list(range(1, 131)) + [133, 160, 161, 200, 239, 240, 241, 300]:
        assert m.ensure("a", upto)
        m.advance("a", upto)
        first = upto // 40 * 40 // 16                             # the page of the first key the next token may see
        t = m.get("a").tables[1]
        assert all(p == -1 for p in t[:first]) and all(p >= 0 for p in t[first:]) and m.check() == ""
        held = max(held, sum(p >= 0 for p in t))
    assert held <= 6 and len(m.get("a").tables[0]) == 19 and all(p >= 0 for p in m.get("a").tables[0])
    m.reset("a")
    assert m.ensure("a", 50) and m.check() == ""
    m.release("a")
    m.release("b")
    assert m.used_pages() == [0, 0] and m.check() == ""
    # a chunk group serves requests longer than its pool; the smallest pool is what is reported
    only = CacheManager({0: chunk}, 16, 96, 1)
    only.admit("long")
    for at in range(0, 4000, 25):
        assert only.ensure("long", at + 25)
        only.advance("long", at + 25)
    assert only.pool_tokens() == 96 and only.check() == ""


def test_decode_splits_under_a_chunk_cover_the_chunk_and_nothing_else():
    """Whatever the context, a chunk of 512 is cut over its own 575 keys at most (it may start inside a tile of 64)."""
    from ember_b200.parts.attention import plan_decode_splits
    for ctx in (100, 512, 1024, 16384):
        for n in (1, 8, 64):
            for chunk in (64, 512, 3000):
                splits, keys, in_cluster = plan_decode_splits(n, ctx, 0, 8, 128, 148, 8, 3.0, 6.4e6, chunk=chunk)
                reach = min(ctx, chunk + 63)
                assert splits * keys >= reach > (splits - 1) * keys and keys % 64 == 0 and (not in_cluster or splits <= 8)
    assert plan_decode_splits(8, 16384, 0, 8, 128, 148, 8, 3.0, 6.4e6, chunk=512)[2]


def test_bad_configurations_are_refused_when_read():
    from ember_b200.config import ConfigError, config_from_dict
    good = FILANEX["a"]["json"]
    for edit in (lambda c: c.pop("width"), lambda c: c["norm"].pop("eps"), lambda c: c["layers"][0].update(type="gla"),
                 lambda c: c["layers"][1]["mixer"].pop("scale"), lambda c: c["layers"][1]["mlp"].update(kind="glu"),
                 lambda c: c.update(layers=[]), lambda c: c["layers"][0]["mlp"]["router"].update(top=5),
                 lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4),
                 lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=4),
                 lambda c: c["layers"][0]["mixer"]["rot"].update(dims=34), lambda c: c["layers"][0]["mixer"]["rot"].update(dims=5),
                 lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), lambda c: c["layers"][0]["mixer"].update(kv_heads=3),
                 lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), lambda c: c["layers"][0]["mixer"].update(softcap=-1.0),
                 lambda c: c["loop"].update(stop=9), lambda c: c["loop"].update(times=0), lambda c: c["loop"].update(start=3),
                 lambda c: c["embedding"]["bigram"].update(buckets=0), lambda c: c["embedding"]["bigram"].pop("mul_cur")):
        c = json.loads(json.dumps(good))
        edit(c)
        with pytest.raises(ConfigError):
            config_from_dict(c)


@pytest.mark.parametrize("name", sorted(FILANEX))
def test_random_folder_declares_what_the_plain_implementation_reads(name, tmp_path):
    d = write_filanex_dir(name, str(tmp_path))
    cfg, W = plain_inputs(d)
    layers = []
    logits = plain.forward(cfg, W, [5, 17, 3, 98, 41, 7, 7, 60], layers_out=layers)
    assert logits.shape == (8, cfg["vocab"]) and bool(torch.isfinite(logits).all()) and len(layers) == len(filanex_config(name).order())
    from ember_b200.config import load_config
    from ember_b200.model.causal_lm import CausalLM
    declared = {x.name: tuple(x.shape) for x in CausalLM(load_config(d).to_model_spec()).weight_decls()}
    assert declared == {k: tuple(v.shape) for k, v in W.items()}


def test_drawn_configurations_are_read():
    from ember_b200.config import config_from_dict
    for seed in range(60):
        c = drawn_filanex(seed)
        back = config_from_dict(config_from_dict(c).to_json()).to_json()
        assert all(back.get(k) == c.get(k) for k in ("layers", "loop", "embedding", "vocab", "width"))


def test_interleaved_rows_are_put_in_the_rotate_half_order():
    """Elements 0, 2, .. of the rotated part, then 1, 3, ..; what is not rotated stays; the same for every head."""
    from ember_b200.config import RotarySpec, SinkAttentionSpec
    from ember_b200.parts import build_part
    spec = SinkAttentionSpec(hidden_size=8, num_heads=2, num_kv_heads=1, head_dim=6, value_dim=4, sink=False,
                             position=RotarySpec(head_dim=6, rotary_dim=4, layout="interleaved", frequency_precision="float64"))
    part = build_part("mixer", spec, "m.")
    got = part._half_order(torch.arange(12.0)[:, None].repeat(1, 3), 2)
    assert got[:, 0].tolist() == [0, 2, 1, 3, 4, 5, 6, 8, 7, 9, 10, 11]


# ------------------------------------------------------------------ the plain implementation on known cases
def test_plain_bigram_rows_hash_the_pair_and_mark_the_start():
    b = {"buckets": 10, "mul_prev": 7, "mul_cur": 3}
    assert plain.bigram_rows([4, 5, 4, 4], b) == [10, (28 + 15) % 10, (35 + 12) % 10, (28 + 12) % 10]
    W = {"embed": torch.zeros(6, 2), "bigram": torch.arange(11.0)[:, None].repeat(1, 2)}
    x = plain.embed({"embedding": {"bigram": b}}, W, [4, 5], torch.float64)
    assert x[:, 0].tolist() == [10.0, 3.0]


def test_plain_rotation_turns_neighbours_with_stretched_frequencies():
    x = torch.zeros(3, 1, 6, dtype=torch.float64)
    x[:, 0, 2] = 1.0                                                          # pairs (0, 1), (2, 3); 4 and 5 pass
    x[:, 0, 5] = 9.0
    y = plain.rotate_pairs(x, {"dims": 4, "base": 100.0})
    assert abs(float(y[2, 0, 2]) - math.cos(2 * 0.1)) < 1e-12 and abs(float(y[2, 0, 3]) - math.sin(0.2)) < 1e-12
    assert float(y[2, 0, 0]) == 0.0 and float(y[1, 0, 5]) == 9.0
    # 16 elements, base 10000, made for 1000 positions: dim(32) = 16 ln(1000 / 64 pi) / (2 ln 10000) = 1.39.. -> lo 1,
    # dim(1) = 16 ln(1000 / 2 pi) / (2 ln 10000) = 4.40.. -> hi 5: pairs 0 and 1 keep their frequency, from 5 on it is divided
    f, mag = plain.frequencies({"dims": 16, "base": 10000.0, "scaling": {"factor": 8.0, "original": 1000, "fast": 32.0, "slow": 1.0}}, torch.float64)
    plain_f, one = plain.frequencies({"dims": 16, "base": 10000.0}, torch.float64)
    ratio = (f / plain_f).tolist()
    assert ratio[:2] == [1.0, 1.0] and all(abs(r - 0.125) < 1e-12 for r in ratio[5:]) and abs(ratio[3] - (0.5 / 8 + 0.5)) < 1e-12
    assert one == 1.0 and abs(mag - (0.1 * math.log(8.0) + 1.0)) < 1e-12


def test_plain_mask_counts_chunks_from_the_start():
    m = plain.visible(7, 3)
    assert m[2].tolist() == [True, True, True, False, False, False, False]
    assert m[3].tolist() == [False, False, False, True, False, False, False]
    assert m[5].tolist() == [False, False, False, True, True, True, False]
    assert plain.visible(4)[3].tolist() == [True] * 4


def test_plain_router_scores_a_group_by_its_two_best():
    W = {"r.router": torch.eye(6, dtype=torch.float64)}
    h = torch.tensor([[3.0, -9.0, 1.0, 0.9, 0.0, 0.5]], dtype=torch.float64)
    s = torch.sigmoid(h)[0]
    # groups (0, 1), (2, 3), (4, 5): the first has the largest score but a tiny second; 1.0 and 0.9 sum higher
    chosen, weights = plain.route(h, W, "r.", {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}})
    assert chosen[0].tolist() == [2, 3] and torch.allclose(weights[0], s[[2, 3]] / (s[2] + s[3]))
    chosen, _ = plain.route(h, W, "r.", {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 2}})
    assert chosen[0].tolist() == [2, 3]                                       # (4, 5) is the second group: 0.5 + 0.62
    chosen, _ = plain.route(h, W, "r.", {"experts": 6, "top": 2, "groups": {"count": 6, "keep": 2}})
    assert chosen[0].tolist() == [0, 2]                                       # groups of one
    chosen, _ = plain.route(h, W, "r.", {"experts": 6, "top": 2})
    assert chosen[0].tolist() == [0, 2]


def test_plain_feed_forwards():
    z = torch.tensor([-3.0, 0.0, 1.5], dtype=torch.float64)
    assert torch.allclose(plain.gelu(z), torch.nn.functional.gelu(z))
    W = {"f.up": torch.ones(1, 2, dtype=torch.float64), "f.up.b": torch.tensor([2.0], dtype=torch.float64),
         "f.down": torch.ones(2, 1, dtype=torch.float64), "f.down.b": torch.tensor([5.0, -1.0], dtype=torch.float64)}
    y = plain.dense_ff(torch.tensor([[0.5, -1.0]], dtype=torch.float64), W, "f.")
    g = 1.5 * 0.5 * (1 + math.erf(1.5 / math.sqrt(2)))
    assert torch.allclose(y, torch.tensor([[g + 5.0, g - 1.0]], dtype=torch.float64))


def test_plain_sublayers_read_one_norm_and_add_at_once():
    """A layer whose mixer is switched off by its gate (sigmoid of -80) is the feed-forward of the same normed input."""
    cfg = {"norm": {"eps": 1e-5}, "layers": [{"type": "attention", "mixer": {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 2, "scale": 1.0}, "mlp": {"kind": "dense", "ff": 3}}]}
    g = torch.Generator().manual_seed(0)
    W = {n: torch.randn(s, generator=g, dtype=torch.float64) for n, s in (
        ("embed", (5, 2)), ("head", (5, 2)), ("final.norm", (2,)), ("l0.norm1", (2,)), ("l0.mix.q", (2, 2)), ("l0.mix.k", (2, 2)), ("l0.mix.v", (2, 2)),
        ("l0.mix.g", (2, 2)), ("l0.mix.o", (2, 2)), ("l0.mlp.up", (3, 2)), ("l0.mlp.up.b", (3,)), ("l0.mlp.down", (2, 3)), ("l0.mlp.down.b", (2,)))}
    layers = []
    plain.forward(cfg, W, [1, 4, 2], layers_out=layers)
    x = W["embed"][[1, 4, 2]]
    h = plain.rms_norm(x, W["l0.norm1"], 1e-5)
    want = x + plain.attention_mixer(h, W, "l0.mix.", cfg["layers"][0]["mixer"]) + plain.dense_ff(h, W, "l0.mlp.")
    assert torch.allclose(layers[0], want)


def test_the_command_line_writes_and_describes_a_random_model(tmp_path, capsys):
    """``random`` makes a folder from a config.json of this design, ``info`` reads it back through the registry."""
    from ember_b200.cli import main
    cfg = tmp_path / "config.json"
    cfg.write_text(json.dumps(FILANEX["b"]["json"]))
    out = tmp_path / "model"
    assert main(["random", "--config", str(cfg), "--out", str(out), "--seed", "3"]) == 0
    capsys.readouterr()
    assert main(["info", "-m", str(out)]) == 0
    text = capsys.readouterr().out
    assert "filanex: 4 layers, layers 0..3 x 3" in text and "state per request" in text
    W = plain_inputs(str(out))[1]
    assert W["bigram"].shape == (14, 100) and W["loop.in"].shape == (100, 200) and W["l0.mix.g"].shape == (24, 100)
