"""Decoder language models, host side: configuration reader and registry (no GPU needed), and the plain
statement's own consistency."""
import copy
import json
import os

import numpy as np
import pytest

import lm_plain as plain
from lm_models import as_float, attention, config, delta, error, latent, tokens, weights, write_folder


@pytest.fixture(scope="module")
def lm_mod(pkg):
    return pkg


GOOD = config([delta(), attention(), attention(window=0, rot=0, softcap=0, ff=0)], loop=(1, 2, 2))


def test_a_configuration_is_accepted(lm_mod):
    lm_mod.check_config(GOOD)
    lm_mod.check_config(json.dumps(GOOD, indent=3))
    lm_mod.check_config({**GOOD, "loop": None, "something_else": {"x": [1, "a\\\"\\u00e9", None, True]}})


@pytest.mark.parametrize("change,what", [
    (lambda c: c.update(architecture="Other"), "not registered"),
    (lambda c: c.pop("architecture"), "not registered"),
    (lambda c: c.pop("vocab"), "vocab"),
    (lambda c: c.update(width=0), "width"),
    (lambda c: c.update(width=8.5), "width"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c.update(layers=[]), "layers"),
    (lambda c: c["layers"][0].update(type="other"), "other"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=2), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"].pop("conv"), "conv"),
    (lambda c: c["layers"][0]["mixer"].update(dim=300), "256"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=34), "dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("fast"), "fast"),
    (lambda c: c["layers"][1]["mlp"].update(kind="sparse"), "kind"),
    (lambda c: c["layers"][1]["mlp"].pop("ff"), "ff"),
    (lambda c: c["loop"].update(stop=9), "stop"),
    (lambda c: c["loop"].update(times=0), "times"),
])
def test_a_wrong_configuration_is_named(lm_mod, change, what):
    c = copy.deepcopy(GOOD)
    change(c)
    with pytest.raises(ValueError, match=what):
        lm_mod.check_config(c)


LATENT = config([latent(), latent(kv_from=0, window=40, ff=30, experts=6, top=2), latent(kv_rank=32, ff=0)])


def test_latent_configurations_are_accepted(lm_mod):
    lm_mod.check_config(LATENT)
    lm_mod.check_config({**LATENT, "something_else": 1})
    lm_mod.check_config(config([latent(window=0, rot_dim=0)]))
    lm_mod.check_config(config([latent(kv_rank=1, q_rank=1, heads=1, dim=1, vdim=1, rot_dim=2, ff=1, experts=1, top=1)]))


@pytest.mark.parametrize("change,what", [
    (lambda c: c["layers"][0].update(type="attention"), "attention"),
    (lambda c: c["layers"][0]["mixer"].pop("q_rank"), "q_rank"),
    (lambda c: c["layers"][0]["mixer"].pop("vdim"), "vdim"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"].update(kv_rank=0), "kv_rank"),
    (lambda c: c["layers"][2]["mixer"].update(kv_rank=5000), "large"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(keep_first=2), "first"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=10), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=5), "dims"),
    (lambda c: c["layers"][1]["mixer"].update(kv_from=1), "kv_from"),
    (lambda c: c["layers"][1]["mixer"].update(kv_from=2), "kv_from"),
    (lambda c: c["layers"][1]["mixer"].update(kv_from=-1), "kv_from"),
    (lambda c: c["layers"][1]["mixer"].update(kv_rank=40), "kv_from"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(base=9.0), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=1, kv_rank=48), "kv_from"),
    (lambda c: c["layers"][0]["mlp"].update(kind="gated"), "kind"),
    (lambda c: c["layers"][0]["mlp"].pop("kind"), "kind"),
    (lambda c: c["layers"][0]["mlp"].pop("ff"), "ff"),
    (lambda c: c["layers"][1]["mlp"]["expert"].pop("ff"), "ff"),
    (lambda c: c["layers"][1]["mlp"].pop("router"), "experts"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=7), "top"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=0), "top"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(experts=5000), "experts"),
])
def test_a_wrong_latent_configuration_is_named(lm_mod, change, what):
    c = copy.deepcopy(LATENT)
    change(c)
    with pytest.raises(ValueError, match=what):
        lm_mod.check_config(c)


@pytest.mark.parametrize("text", ["", "{", "[1, 2", '{"a" 1}', '{"a": tru}', '{"a": "x', '{"a": 1} x', "[" * 200])
def test_malformed_json_is_reported(lm_mod, text):
    with pytest.raises(ValueError, match="config.json"):
        lm_mod.check_config(text)


def test_loading_without_a_gpu_fails_loudly(lm_mod, tmp_path):
    import torch
    with pytest.raises(RuntimeError, match="config.json"):
        lm_mod.LanguageModel(str(tmp_path / "nowhere"))
    if not torch.cuda.is_available():
        with pytest.raises(RuntimeError):
            lm_mod.LanguageModel(write_folder(tmp_path, GOOD, weights(GOOD, 1)))


def test_model_folder_round_trip(tmp_path):
    w = weights(GOOD, 1)
    cfg, got = plain.load_folder(write_folder(tmp_path, GOOD, w))
    assert cfg == json.loads(json.dumps(GOOD))
    want = as_float(w)
    assert set(got) == set(want) and all(np.array_equal(got[n], want[n]) for n in want)


def test_statement_is_causal_and_windowed():
    """Later tokens change nothing; a token behind the window and not kept changes nothing."""
    cfg = config([attention(window=8, keep=2, ff=0)], width=48, vocab=50)
    w = as_float(weights(cfg, 4))
    t = tokens(cfg, 30, 1)
    base = plain.forward(w, cfg, t)[0]
    for at in (0, 1, 2, 21, 22, 29):
        other = list(t)
        other[at] = (t[at] + 1) % 50
        d = np.abs(plain.forward(w, cfg, other)[0] - base).max(axis=1)
        assert np.all(d[:at] == 0.0)
        assert (d[29] > 0) == (at < 2 or at >= 22)


def test_delta_rule_in_two_pieces():
    rng = np.random.default_rng(0)
    q, k, v = rng.standard_normal((20, 6)), rng.standard_normal((20, 6)), rng.standard_normal((20, 5))
    b, g = rng.uniform(size=20), rng.uniform(size=20)
    o, S = plain.delta_rule(q, k, v, b, g)
    o1, S1 = plain.delta_rule(q[:7], k[:7], v[:7], b[:7], g[:7])
    o2, S2 = plain.delta_rule(q[7:], k[7:], v[7:], b[7:], g[7:], S1)
    assert np.allclose(np.concatenate([o1, o2]), o) and np.allclose(S, S2)


def test_yarn_frequencies():
    f, m = plain.rope_frequencies({"dims": 16, "base": 10000.0})
    assert m == 1.0 and np.allclose(f, 10000.0 ** (-np.arange(8) / 8))
    y, m = plain.rope_frequencies({"dims": 16, "base": 10000.0, "scaling": {"factor": 5.0, "original": 1500, "fast": 40, "slow": 2}})
    assert np.isclose(m, 0.1 * np.log(5.0) + 1)
    assert np.allclose(y[0], f[0]) and np.allclose(y[-1], f[-1] / 5) and np.all(y <= f) and np.all(y >= f / 5 * (1 - 1e-12))


def test_statement_of_the_latent_attention():
    """Causal and windowed; a layer that reads another's latents sees as far as its own window, not the other's."""
    cfg = config([latent(window=5, ff=0, heads=2), latent(window=0, kv_from=0, heads=3, ff=0)], width=48, vocab=50)
    w = as_float(weights(cfg, 4))
    w["l0.mix.o"][:] = 0.0
    t = tokens(cfg, 30, 1)
    base, taps = plain.forward(w, cfg, t)
    assert np.array_equal(taps[0], w["embed"][t])
    for at in (0, 21, 29):
        other = list(t)
        other[at] = (t[at] + 1) % 50
        d = np.abs(plain.forward(w, cfg, other)[0] - base).max(axis=1)
        assert np.all(d[:at] == 0.0) and np.all(d[at:] > 0.0)
    cfg["layers"][1]["mixer"]["mask"] = {"size": 8}
    base = plain.forward(w, cfg, t)[0]
    for at in (20, 21, 22, 23):
        other = list(t)
        other[at] = (t[at] + 1) % 50
        assert (np.abs(plain.forward(w, cfg, other)[0] - base).max(axis=1)[29] > 0) == (at >= 22)


def test_rotation_of_neighbours():
    """The product of a rotated query and key depends on their distance only; what is not rotated passes unchanged."""
    rng = np.random.default_rng(3)
    q, k = rng.standard_normal((1, 10)), rng.standard_normal((1, 10))
    rot = {"dims": 8, "base": 500.0}
    at = lambda x, p: plain.rotate_neighbours(x, [p], rot)[0]
    assert np.isclose(at(q, 7) @ at(k, 3), at(q, 104) @ at(k, 100)) and not np.isclose(at(q, 7) @ at(k, 3), at(q, 7) @ at(k, 4))
    assert np.array_equal(at(q, 9)[8:], q[0, 8:])
    one = plain.rotate_neighbours(np.eye(10)[:1], [2], rot)[0]
    assert np.isclose(one[0], np.cos(2.0)) and np.isclose(one[1], np.sin(2.0))


def test_routing():
    z = np.array([[1.0, 5.0, -2.0, 3.0]])
    chosen, p = plain.route(z, np.eye(4), 2)
    assert chosen.tolist() == [[1, 3]] and np.allclose(p, [[1 / (1 + np.exp(-2.0)), 1 / (1 + np.exp(2.0))]])
    assert plain.route(z, np.eye(4), 1)[1].tolist() == [[1.0]]


def test_one_expert_is_a_dense_feed_forward():
    dense, moe = config([latent(ff=20)], width=40), config([latent(ff=20, experts=1, top=1)], width=40)
    w = as_float(weights(moe, 6))
    t = tokens(dense, 12, 2)
    a = plain.forward(w, moe, t)[0]
    w["l0.mlp.up"], w["l0.mlp.down"] = w["l0.mlp.e0.up"], w["l0.mlp.e0.down"]
    assert error(plain.forward(w, dense, t)[0], a) < 1e-12
