"""Nololix without a device: the folder reader and its errors, and the oracle's own properties - each mechanism alone, and
that a fault in any of them shows in the logits of the test models by far more than rounding."""

import copy

import numpy as np
import pytest

import layer_list_testlib as ll
import nololix_oracle as no
import nololix_testlib as nl
import q38_testlib as tl  # noqa: F401  (loads the package)
from q38b200 import engine as eng


@pytest.mark.parametrize("name", sorted(nl.CONFIGS))
def test_model_folders_open(tmp_path, name):
    cfg = nl.CONFIGS[name]
    folder, _ = nl.make_model(tmp_path / name, cfg)
    m = eng.Model(folder)
    assert (m.architecture, m.vocab, m.hidden, m.layers) == ("Nololix", cfg["vocab"], cfg["width"], len(cfg["layers"]))
    kinds = [x["type"] for x in cfg["layers"]]
    assert f"{kinds.count('retention')} retention / {kinds.count('latent_attention')} latent attention" in m.summary()
    assert ("times" in m.summary()) == bool(cfg["loop"])
    m.close()


def test_optional_entries(tmp_path):
    """No loop, no rotation, one stream without hyper-connections, no scale: left out altogether."""
    cfg = nl.config(40, 30, [nl.retention(2, 8, 8, (0.9, 0.8)), nl.latent(2, 8, 8, 8, 8)])
    t = {k: v for k, v in nl.random_tensors(cfg, 1).items() if ".hc" not in k}
    for key in ("loop", "streams", "embedding", "residual_mult"):
        del cfg[key]
    del cfg["norm"]["groups"], cfg["layers"][0]["mixer"]["rot"], cfg["layers"][1]["mlp"]
    eng.Model(ll.write_model(tmp_path / "m", cfg, t)).close()


def test_bad_folders_are_refused(tmp_path):
    cfg = nl.CONFIGS["mixed"]
    tensors = nl.random_tensors(cfg, 3)

    def refused(match, change_cfg=None, change=None):
        c, t = copy.deepcopy(cfg), dict(tensors)
        if change_cfg:
            change_cfg(c)
        if change:
            change(t)
        with pytest.raises(eng.EngineError, match=match):
            eng.Model(ll.write_model(tmp_path / "bad", c, t))

    refused("missing key 'vocab'", lambda c: c.pop("vocab"))
    refused("mixer 'mingru' is not part", lambda c: c["layers"][0].update(type="mingru"))
    refused("feed-forward 'routed'", lambda c: c["layers"][0]["mlp"].update(kind="routed"))
    refused("4 decays for 5 heads", lambda c: c["layers"][0]["mixer"]["decay"].pop())
    refused("26 rotated dimensions of 24", lambda c: c["layers"][0]["mixer"]["rot"].update(dims=26))
    refused("5 norm groups of a width of 112", lambda c: c["norm"].update(groups=5))
    refused("loop over layers 3 .. 4", lambda c: c["loop"].update(start=3, stop=5))
    refused("17 residual streams", lambda c: c.update(streams=17))
    refused(r"l0.hc1.in: shape \[3\], expected \[4\]", lambda c: c.update(streams=4))
    refused("'l1.mix.dkv.norm' not found", change=lambda t: t.pop("l1.mix.dkv.norm"))
    refused("'l0.mlp.act' not found", change=lambda t: t.pop("l0.mlp.act"))
    refused(r"l3.mix.uk: shape \[128, 72\], expected \[128, 80\]", lambda c: c["layers"][3]["mixer"].update(kv_rank=80),
            lambda t: t.update({"l3.mix.dkv": np.zeros((80, 112)), "l3.mix.dkv.norm": np.zeros(80)}))


def test_oracle_mechanisms_alone():
    rng = np.random.default_rng(0)
    # parts of a row are normed on their own; one part is the ordinary norm
    x = rng.standard_normal((4, 12))
    y = no.rms_norm(x, 2.0, 0.0, 3)
    assert np.allclose(np.mean(y.reshape(4, 3, 4) ** 2, axis=2), 4.0)
    assert np.allclose(no.rms_norm(x, 1.0, 1e-3), x / np.sqrt(np.mean(x * x, axis=1, keepdims=True) + 1e-3))
    # a rotation keeps lengths, turns products by the distance only, and leaves the other dimensions alone
    q, k = rng.standard_normal((2, 7, 3, 10))
    pos = np.arange(7)
    a, b = no.rope(q, pos, 6, 100.0), no.rope(k, pos, 6, 100.0)
    assert np.allclose(np.linalg.norm(a, axis=2), np.linalg.norm(q, axis=2)) and np.array_equal(a[:, :, 6:], q[:, :, 6:])
    a2, b2 = no.rope(q, pos + 40, 6, 100.0), no.rope(k, pos + 40, 6, 100.0)
    assert np.allclose(np.einsum("ihd,jhd->hij", a, b), np.einsum("ihd,jhd->hij", a2, b2))
    # the recurrence is a weighted sum over the past, whole or from a carried state
    v, decay = rng.standard_normal((7, 3, 4)), np.array([0.9, 0.5, 1.0])
    o, S = no.retention(q, k, v, decay)
    w = np.einsum("ihd,jhd->hij", q, k) * np.tril(decay[:, None, None] ** (pos[:, None] - pos[None]))
    assert np.allclose(o, np.einsum("hij,jhv->ihv", w, v))
    o1, S1 = no.retention(q[:3], k[:3], v[:3], decay)
    o2, S2 = no.retention(q[3:], k[3:], v[3:], decay, S1)
    assert np.allclose(np.concatenate([o1, o2]), o) and np.allclose(S2, S)
    # attention: weights sum to one, the first token sees itself only
    ones = no.softmax_attention(q, k, np.ones((7, 3, 2)), 0.5)
    assert np.allclose(ones, 1.0) and np.allclose(no.softmax_attention(q, k, v, 0.5)[0], v[0])
    # the latent form: a head's key matrix may meet the query instead of the latent, its value matrix the output
    c, uk, uv = rng.standard_normal((7, 5)), rng.standard_normal((3, 10, 5)), rng.standard_normal((3, 4, 5))
    plain = no.softmax_attention(q, np.einsum("hdr,jr->jhd", uk, c), np.einsum("hvr,jr->jhv", uv, c), 0.3)
    absorbed = no.softmax_attention(np.einsum("hdr,ihd->ihr", uk, q), np.repeat(c[:, None], 3, 1), np.repeat(c[:, None], 3, 1), 0.3)
    assert np.allclose(np.einsum("hvr,ihr->ihv", uv, absorbed), plain)
    # the activation is continuous with slope 1/2 at zero
    e = 1e-6
    assert abs(no.xielu(np.array(0.0), 0.3, -0.2)) == 0
    assert np.allclose([(no.xielu(np.array(s * e), 0.3, -0.2)) / (s * e) for s in (1, -1)], 0.5, atol=1e-5)
    # one stream with in = out = mix = 1 is the ordinary residual sum; all streams change at once
    y = rng.standard_normal((4, 12))
    assert np.allclose(no.hyper_update(x[None], y, np.ones((1, 1)), np.ones(1), 0.5)[0], x + 0.5 * y)
    mix = rng.standard_normal((2, 2))
    z = no.hyper_update(np.stack([x, 2 * x]), 0 * y, mix, np.ones(2), 1.0)
    assert np.allclose(z[1], (mix[0, 1] + 2 * mix[1, 1]) * x)
    assert no.run_order({"layers": [0] * 4, "loop": {"start": 1, "stop": 3, "times": 2}}) == [0, 1, 2, 1, 2, 3]


def _each(suffix, f):
    def change(t, c):
        hit = [k for k in t if k.endswith(suffix)]
        assert hit
        t.update({k: f(t[k]) for k in hit})
    return change


def _mixers(kind, f):
    return lambda t, c: [f(x["mixer"]) for x in c["layers"] if x["type"] == kind]


FAULTS = {
    "streams mixed the other way": _each(".mix", lambda v: v.T),
    "streams not mixed": _each(".mix", lambda v: np.eye(len(v))),
    "wrong weight into a stream": _each(".out", lambda v: v[::-1]),
    "only one stream read": _each(".in", lambda v: v * (np.arange(len(v)) == 0)),
    "residual factor": lambda t, c: c.update(residual_mult=1.0),
    "embedding scale": lambda t, c: c["embedding"].update(scale=1.0),
    "norm over the whole row": lambda t, c: c["norm"].update(groups=1),
    "eps": lambda t, c: c["norm"].update(eps=1e-2),
    "one pass less": lambda t, c: c["loop"].update(times=1),
    "loop one layer short": lambda t, c: c["loop"].update(stop=2),
    "decays of heads swapped": _mixers("retention", lambda m: m["decay"].reverse()),
    "decay forgets more": _mixers("retention", lambda m: m.update(decay=[d * 0.98 for d in m["decay"]])),
    "rotation base": _mixers("retention", lambda m: m["rot"].update(base=m["rot"]["base"] * 4.0)),
    "rotation left out": _mixers("retention", lambda m: m["rot"].update(dims=0)),
    "scale of the scores": _mixers("latent_attention", lambda m: m.update(scale=m["scale"] * 2.0)),
    "no latent norm weight": _each(".dkv.norm", lambda v: np.ones_like(v)),
    "no query latent norm weight": _each(".dq.norm", lambda v: np.ones_like(v)),
    "output gate stuck": _each(".mix.g", lambda v: v * 0),
    "activation parameters swapped": _each(".mlp.act", lambda v: v[::-1]),
    "heads' key matrices swapped": _each(".uk", lambda v: v[::-1]),
}


@pytest.mark.parametrize("fault", sorted(FAULTS))
def test_every_mechanism_shows_in_the_logits(fault):
    cfg = nl.CONFIGS["mixed"]
    tensors = nl.random_tensors(cfg, 5)
    tokens = np.random.default_rng(1).integers(0, cfg["vocab"], 40)
    want = no.Model(cfg, tensors).logits(tokens)
    c, t = copy.deepcopy(cfg), dict(tensors)
    FAULTS[fault](t, c)
    got = no.Model(c, t).logits(tokens)
    assert np.sqrt(np.mean((got - want)[20:] ** 2)) > (1e-3 if fault == "eps" else 0.05) * np.sqrt(np.mean(want ** 2))


def test_a_lost_state_and_a_lost_pass_state_show(monkeypatch):
    """Retention that starts from nothing in the middle of the sequence, and attention that lost its first page."""
    cfg = nl.CONFIGS["mixed"]
    tensors = nl.random_tensors(cfg, 6)
    tokens = np.random.default_rng(2).integers(0, cfg["vocab"], 100)
    model = no.Model(cfg, tensors)
    want = model.logits(tokens)
    plain = no.retention

    def forgets(q, k, v, decay, state=None):
        a, _ = plain(q[:64], k[:64], v[:64], decay)
        b, _ = plain(q[64:], k[64:], v[64:], decay)
        return np.concatenate([a, b]), None
    monkeypatch.setattr(no, "retention", forgets)
    lost = model.logits(tokens)
    assert np.allclose(lost[:64], want[:64])
    assert np.sqrt(np.mean((lost - want)[64:] ** 2)) > 0.05 * np.sqrt(np.mean(want ** 2))
