"""Fegenex without a device: the folder reader and its errors, and the oracle's own properties - each mechanism alone, and
that a fault in any of them shows in the logits of the test models by far more than rounding."""

import copy
import json

import numpy as np
import pytest

import fegenex_oracle as fo
import layer_list_testlib as ll
import q38_testlib as tl  # noqa: F401  (loads the package)
from q38b200 import engine as eng


@pytest.mark.parametrize("name", sorted(ll.CONFIGS))
def test_model_folders_open(tmp_path, name):
    cfg = ll.CONFIGS[name]
    folder, _ = ll.make_model(tmp_path / name, cfg)
    m = eng.Model(folder)
    assert (m.architecture, m.vocab, m.hidden, m.layers) == ("Fegenex", cfg["vocab"], cfg["width"], len(cfg["layers"]))
    assert m.max_positions == cfg["max_positions"]
    assert f"{sum(x['type'] == 'mingru' for x in cfg['layers'])} minGRU" in m.summary()
    m.close()


def test_bad_folders_are_refused(tmp_path):
    cfg = ll.CONFIGS["mixed"]
    tensors = ll.random_tensors(cfg, 3)

    def refused(match, change_cfg=None, change=None):
        c, t = copy.deepcopy(cfg), dict(tensors)
        if change_cfg:
            change_cfg(c)
        if change:
            change(t)
        with pytest.raises(eng.EngineError, match=match):
            eng.Model(ll.write_model(tmp_path / "bad", c, t))

    refused("not in this build", lambda c: c.update(architecture="Nothing"))
    refused("read from .q38 files", lambda c: c.update(architecture="Qwen3.8"))
    refused("missing key 'vocab'", lambda c: c.pop("vocab"))
    refused("mixer 'loop' is not part", lambda c: c["layers"][0].update(type="loop"))
    refused("feed-forward 'routed'", lambda c: c["layers"][0]["mlp"].update(kind="routed"))
    refused("6 query heads over 4", lambda c: c["layers"][1]["mixer"].update(kv_heads=4))
    refused("'l1.mix.talk' not found", change=lambda t: t.pop("l1.mix.talk"))
    refused(r"l1.mix.k: shape \[80, 112\], expected \[160, 112\]", lambda c: c["layers"][1]["mixer"].update(dim=80),
            lambda t: t.update({"l1.mix.q": np.zeros((480, 112))}) or t.update({"l1.mix.q.b": np.zeros(480)}))
    folder = ll.write_model(tmp_path / "cut", cfg, tensors)
    data = (folder / "model.safetensors").read_bytes()
    (folder / "model.safetensors").write_bytes(data[:len(data) // 2])
    with pytest.raises(eng.EngineError, match="outside the file"):
        eng.Model(folder)
    (folder / "config.json").write_text("{")
    with pytest.raises(eng.EngineError, match="malformed configuration"):
        eng.Model(folder)


def test_oracle_mechanisms_alone():
    rng = np.random.default_rng(0)
    # a rotation keeps lengths, turns scores by the distance only, and leaves the other dimensions alone
    q, k = rng.standard_normal((2, 7, 3, 10))
    pos = np.arange(7)
    a, b = fo.rope(q, pos, 6, 100.0), fo.rope(k, pos, 6, 100.0)
    assert np.allclose(np.linalg.norm(a, axis=2), np.linalg.norm(q, axis=2)) and np.array_equal(a[:, :, 6:], q[:, :, 6:])
    a2, b2 = fo.rope(q, pos + 40, 6, 100.0), fo.rope(k, pos + 40, 6, 100.0)
    assert np.allclose(np.einsum("ihd,jhd->hij", a, b), np.einsum("ihd,jhd->hij", a2, b2))
    # identity mixing is plain grouped attention; a constant value passes through weights that sum to the row of T
    v = np.ones((7, 1, 4))
    T = rng.standard_normal((3, 3))
    out = fo.mixed_head_attention(a, b[:, :1], v, 0.5, T)
    assert np.allclose(out, T.sum(1)[None, :, None])
    # recurrences: token by token from a carried state equals the whole
    z = [rng.standard_normal(s) for s in ((5, 4), 5, (5, 4), 5, (5, 4), (4, 5))]
    h = rng.standard_normal((9, 4))
    assert fo.min_gru(h, *z).shape == (9, 4)
    x, w = rng.standard_normal((6, 2)), rng.standard_normal((2, 3))
    y = fo.causal_conv(x, w, np.zeros(2))
    assert np.allclose(y[0], w[:, 2] * x[0]) and np.allclose(y[5], w[:, 2] * x[5] + w[:, 1] * x[4] + w[:, 0] * x[3])
    u = rng.standard_normal((6, 4))
    ra = rng.standard_normal((2, 2, 2))
    s = fo.rg_lru(u, ra, np.zeros((2, 2)), ra, np.zeros((2, 2)), np.full(4, 30.0))
    i = fo.sigmoid(fo.block_linear(u, ra, np.zeros((2, 2))))
    assert np.allclose(s, i * u, atol=1e-6)  # a decay to nothing leaves the gated input


FAULTS = {
    "no head mixing": lambda t, c: t.update({k: np.eye(len(v)) for k, v in t.items() if k.endswith("talk")}),
    "mixing matrix transposed": lambda t, c: t.update({k: v.T for k, v in t.items() if k.endswith("talk")}),
    "no value blending": lambda t, c: t.update({k: np.array(0.0) for k in t if k.endswith("vmix")}),
    "no positions": lambda t, c: t.update(pos=t["pos"] * 0),
    "projection bias lost": lambda t, c: t.update({k: v * 0 for k, v in t.items() if k.endswith("o.b")}),
    "convolution reversed": lambda t, c: t.update({k: v[:, ::-1] for k, v in t.items() if k.endswith("conv")}),
    "gates of blocks swapped": lambda t, c: t.update({k: v[::-1] for k, v in t.items() if k.endswith(".ra")}),
    "slower decay": lambda t, c: t.update({k: v - 1.0 for k, v in t.items() if k.endswith("lam")}),
    "rotation base": lambda t, c: [x["mixer"]["rot"].update(base=x["mixer"]["rot"]["base"] * 1.2) for x in c["layers"]
                                   if x["type"] == "attention"],
    "eps": lambda t, c: c["norm"].update(eps=1e-2),
}


@pytest.mark.parametrize("fault", sorted(FAULTS))
def test_every_mechanism_shows_in_the_logits(fault):
    cfg = ll.CONFIGS["mixed"]
    tensors = ll.random_tensors(cfg, 5)
    tokens = np.random.default_rng(1).integers(0, cfg["vocab"], 40)
    want = fo.Model(cfg, tensors).logits(tokens)
    c, t = copy.deepcopy(cfg), dict(tensors)
    FAULTS[fault](t, c)
    got = fo.Model(c, t).logits(tokens)
    assert np.sqrt(np.mean((got - want)[20:] ** 2)) > (1e-3 if fault == "eps" else 0.03) * np.sqrt(np.mean(want ** 2))


def test_family_builds_name_disjoint_sources_and_known_architectures():
    from q38b200 import build
    seen = set()
    for family in build.FAMILIES.values():
        for kind, folder, suffix in (("cu", build.CSRC, ".cu"), ("host", build.HOST / "src", ".cpp")):
            for stem in family[kind]:
                assert (folder / (stem + suffix)).exists() and (kind, stem) not in seen
                seen.add((kind, stem))
    assert set(build.ARCHITECTURE_FAMILY.values()) == set(build.FAMILIES)


def test_runner_options_struct_matches_the_library_defaults():
    o = eng.default_runner_options()
    assert (o.max_batch, o.prefill_chunk, o.kv_dtype, o.compute_dtype) == (8, 1024, -1, 0)
    assert json.dumps(o.max_context) == "262144"
