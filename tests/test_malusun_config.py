"""Malusun without a device: reading config.json, the tensors a model declares, what its layers ask of the cache, which layer
hands out its values, the random-weights folder, the command line, and the plain implementation's own mechanisms on cases
whose answer is known."""
import json
import math

import pytest
import torch

from tests.malusun_configs import MALUSUN, drawn_malusun, malusun_config, plain_inputs, write_malusun_dir
from tests.plain import malusun_plain as plain


def test_registered_and_resolved_by_the_architecture_key():
    from ember_b200.config import MalusunConfig, config_from_dict, registered_architectures
    assert "Malusun" in registered_architectures()
    cfg = config_from_dict(MALUSUN["a"]["json"])
    assert isinstance(cfg, MalusunConfig) and cfg.width == 128 and cfg.embedding_scale == 8.0
    for name in MALUSUN:
        assert config_from_dict(malusun_config(name).to_json()) == malusun_config(name)
    assert malusun_config("d").embedding_scale == 1.0


def test_the_first_blending_layer_is_the_source():
    assert [malusun_config(n).value_source() for n in "abcd"] == [1, 0, 0, -1]
    mixes = lambda n: [getattr(l.part("mixer")[0], "value_mix", None) for l in malusun_config(n).to_model_spec().layers]     # noqa: E731
    assert mixes("a") == [None, "source", "mix", "", ""] and mixes("b") == ["source", None, "mix", "mix", None]
    assert mixes("d") == [None, "", None, ""]


@pytest.mark.parametrize("name", sorted(MALUSUN))
def test_cache_needs(name):
    """Pages in a window where there is a mask, all of them where not; one state row a request for a scan, which also holds
    the convolution's last inputs."""
    from ember_b200.model.causal_lm import CausalLM
    cfg, j = malusun_config(name), MALUSUN[name]["json"]
    needs = CausalLM(cfg.to_model_spec()).cache_needs()
    kv = state = 0
    for i, l in enumerate(j["layers"]):
        m, n = l["mixer"], needs[i]
        if l["type"] == "mamba1":
            floats = m["inner"] * (m["state"] + m["conv"] - 1)
            assert (n.kind, n.state_shape, n.state_dtype) == ("state", (floats,), "float32")
            state += 4 * floats
            continue
        window = (m.get("mask") or {}).get("size", 0)
        assert (n.kind, n.window, n.keep_first) == ("window" if window else "full", window, 0)
        assert (n.num_kv_heads, n.head_dim, n.value_dim or n.head_dim) == (m["kv_heads"], m["dim"], m["vdim"])
        kv += 2 * m["kv_heads"] * (m["dim"] + m["vdim"])
    assert cfg.kv_bytes_per_token(2) == kv and cfg.state_bytes_per_request() == state


def test_the_distance_slopes_and_the_sink_are_constants_of_the_design():
    spec = malusun_config("a").to_model_spec().layers[2].part("mixer")[0]
    assert (spec.slope_span, spec.sink, spec.fixed_sink, spec.bias) == (8.0, True, 0.0, True)
    plain_layer = malusun_config("a").to_model_spec().layers[1].part("mixer")[0]
    assert (plain_layer.slope_span, plain_layer.sink, plain_layer.bias) == (0.0, False, False)


def test_bad_configurations_are_refused_when_read():
    from ember_b200.config import ConfigError, config_from_dict
    good = MALUSUN["a"]["json"]
    for edit in (lambda c: c.pop("width"), lambda c: c["norm"].pop("eps"), lambda c: c["layers"][0].update(type="gla"),
                 lambda c: c["layers"][0]["mixer"].pop("dt_rank"), lambda c: c["layers"][0]["mixer"].update(state=0),
                 lambda c: c["layers"][0]["mixer"].update(state=1000), lambda c: c["layers"][0]["mixer"].update(conv=0),
                 lambda c: c["layers"][1]["mixer"].pop("scale"), lambda c: c["layers"][1]["mlp"].update(kind="glu"),
                 lambda c: c.update(layers=[]), lambda c: c["layers"][0]["mlp"]["router"].update(top=7),
                 lambda c: c["layers"][1]["mixer"]["rot"].update(dims=34), lambda c: c["layers"][1]["mixer"]["rot"].update(dims=5),
                 lambda c: c["layers"][1]["mixer"].update(kv_heads=3), lambda c: c["layers"][1]["mixer"]["mask"].update(size=0),
                 lambda c: c["layers"][2]["mixer"].update(vdim=32), lambda c: c["layers"][0]["mlp"]["shared"].update(ff=0),
                 lambda c: c["embedding"].update(scale="8")):
        c = json.loads(json.dumps(good))
        edit(c)
        with pytest.raises(ConfigError):
            config_from_dict(c)


@pytest.mark.parametrize("name", sorted(MALUSUN))
def test_random_folder_declares_what_the_plain_implementation_reads(name, tmp_path):
    d = write_malusun_dir(name, str(tmp_path))
    cfg, W = plain_inputs(d)
    layers = []
    logits = plain.forward(cfg, W, [5, 17, 3, 98, 41, 7, 7, 60], layers_out=layers)
    assert logits.shape == (8, cfg["vocab"]) and bool(torch.isfinite(logits).all()) and len(layers) == len(cfg["layers"])
    from ember_b200.config import load_config
    from ember_b200.model.causal_lm import CausalLM
    mcfg = load_config(d)
    declared = {x.name: tuple(x.shape) for x in CausalLM(mcfg.to_model_spec()).weight_decls()}
    unread = {f"l{mcfg.value_source()}.mix.vmix"}                             # the source's own factor is not read
    assert declared == {k: tuple(v.shape) for k, v in W.items() if k not in unread}


def test_drawn_configurations_are_read():
    from ember_b200.config import config_from_dict
    for seed in range(200):
        c = drawn_malusun(seed)
        back = config_from_dict(config_from_dict(c).to_json()).to_json()
        assert all(back.get(k) == c.get(k) for k in ("layers", "embedding", "vocab", "width"))


# ------------------------------------------------------------------ the plain implementation on known cases
def test_plain_norm_weights_are_distances_from_one():
    x = torch.tensor([[3.0, -4.0]], dtype=torch.float64)
    y = plain.rms_norm(x, torch.tensor([0.0, 0.5], dtype=torch.float64), 0.0)
    r = math.sqrt(12.5)
    assert torch.allclose(y, torch.tensor([[3.0 / r, -6.0 / r]], dtype=torch.float64))


def test_plain_convolution_meets_the_current_token_with_its_last_tap():
    x = torch.arange(1.0, 6.0, dtype=torch.float64)[:, None]
    y = plain.causal_conv(x, torch.tensor([[100.0, 10.0, 1.0]], dtype=torch.float64), torch.tensor([0.5], dtype=torch.float64))
    assert y[:, 0].tolist() == [1.5, 12.5, 123.5, 234.5, 345.5]


def test_plain_scan_is_the_recurrence():
    """One channel, one state: S_t = e^(-a d_t) S_(t-1) + d_t x_t B_t, y = S C + D x; a second call goes on from the state."""
    t64 = lambda *v: torch.tensor(v, dtype=torch.float64)                     # noqa: E731
    x, d, B, C = t64(1.0, 2.0, -1.0)[:, None], t64(0.5, 0.25, 1.0)[:, None], t64(2.0, 1.0, 3.0)[:, None], t64(1.0, 5.0, 0.5)[:, None]
    A, D = t64(-2.0)[:, None], t64(10.0)
    y, S = plain.selective_scan(x, d, A, B, C, D)
    s1 = 0.5 * 1.0 * 2.0
    s2 = math.exp(-0.5) * s1 + 0.25 * 2.0 * 1.0
    s3 = math.exp(-2.0) * s2 - 3.0
    assert torch.allclose(y[:, 0], t64(s1 + 10.0, 5.0 * s2 + 20.0, 0.5 * s3 - 10.0)) and abs(float(S) - s3) < 1e-12
    first, S1 = plain.selective_scan(x[:1], d[:1], A, B[:1], C[:1], D)
    rest, S2 = plain.selective_scan(x[1:], d[1:], A, B[1:], C[1:], D, S1)
    assert torch.allclose(torch.cat([first, rest]), y) and torch.allclose(S2, S)


def test_plain_rotation_pairs_halves_and_passes_the_rest():
    x = torch.zeros(3, 1, 6, dtype=torch.float64)
    x[:, 0, 1] = 1.0                                                          # pairs (0, 2), (1, 3); 4 and 5 pass
    x[:, 0, 5] = 9.0
    y = plain.rotate_half(x, {"dims": 4, "base": 100.0})
    assert abs(float(y[2, 0, 1]) - math.cos(0.2)) < 1e-12 and abs(float(y[2, 0, 3]) - math.sin(0.2)) < 1e-12
    assert float(y[2, 0, 0]) == 0.0 and float(y[1, 0, 5]) == 9.0


def test_plain_window_slopes_and_sink():
    assert plain.visible(5, 2)[3].tolist() == [False, False, True, True, False] and plain.visible(3)[2].tolist() == [True] * 3
    assert plain.slopes(4) == [2.0 ** -2, 2.0 ** -4, 2.0 ** -6, 2.0 ** -8] and plain.slopes(1) == [2.0 ** -8]
    # equal keys: scores 0 and -slope; the sink's own score is 0
    q, k = torch.zeros(2, 1, 4, dtype=torch.float64), torch.zeros(2, 1, 4, dtype=torch.float64)
    v = torch.tensor([[[1.0]], [[0.0]]], dtype=torch.float64)
    o = plain.biased_attention(q, k, v, 1.0, plain.visible(2))
    e = math.exp(-(2.0 ** -8))
    assert abs(float(o[0]) - 0.5) < 1e-12 and abs(float(o[1]) - e / (2.0 + e)) < 1e-12
    # scores far above the sink's: an ordinary softmax
    big = plain.biased_attention(torch.full_like(q, 30.0), torch.full_like(k, 30.0), v, 1.0, plain.visible(2))
    assert abs(float(big[1]) - e / (1.0 + e)) < 1e-12


def test_plain_values_blend_with_the_first_layers():
    v, first = torch.tensor([[[2.0]]], dtype=torch.float64), torch.tensor([[[10.0]]], dtype=torch.float64)
    assert float(plain.mix_values(v, first, torch.tensor(0.25))) == 4.0


def test_plain_experts_read_the_weighted_input():
    """One expert of width one: silu(g w h) (u w h), not w silu(g h) (u h); the shared expert reads h itself."""
    one = lambda x: torch.tensor([[x]], dtype=torch.float64)                  # noqa: E731
    W = {"m.router": one(2.0), "m.e0.gate": one(1.5), "m.e0.up": one(-1.0), "m.e0.down": one(3.0),
         "m.shared.gate": one(0.5), "m.shared.up": one(1.0), "m.shared.down": one(1.0)}
    h = one(0.7)
    s = 1.0 / (1.0 + math.exp(-1.4))
    silu = lambda z: z / (1.0 + math.exp(-z))                                 # noqa: E731
    want = 3.0 * silu(1.5 * s * 0.7) * (-s * 0.7) + silu(0.35) * 0.7
    got = plain.moe_ff(h, W, "m.", {"router": {"experts": 1, "top": 1}, "shared": {"ff": 1}})
    assert abs(float(got) - want) < 1e-12
    assert abs(3.0 * s * silu(1.05) * -0.7 + silu(0.35) * 0.7 - want) > 0.05
    assert float(plain.dense_ff(one(-2.0), {"f.up": one(1.0), "f.down": one(1.0)}, "f.")) == 0.0
    assert float(plain.dense_ff(one(3.0), {"f.up": one(1.0), "f.down": one(2.0)}, "f.")) == 18.0


def test_the_command_line_writes_and_describes_a_random_model(tmp_path, capsys):
    """``random`` makes a folder from a config.json of this design, ``info`` reads it back through the registry."""
    from ember_b200.cli import main
    cfg = tmp_path / "config.json"
    cfg.write_text(json.dumps(MALUSUN["b"]["json"]))
    out = tmp_path / "model"
    assert main(["random", "--config", str(cfg), "--out", str(out), "--seed", "3"]) == 0
    capsys.readouterr()
    assert main(["info", "-m", str(out)]) == 0
    text = capsys.readouterr().out
    assert "malusun: 5 layers" in text and "state per request" in text
    W = plain_inputs(str(out))[1]
    assert W["l1.mix.A_log"].shape == (77, 5) and W["l3.mix.q.b"].shape == (180,) and W["l2.mix.vmix"].shape == ()
