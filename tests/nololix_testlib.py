"""Random Nololix models on disk for the tests."""

from __future__ import annotations

import numpy as np

import layer_list_testlib as ll
import nololix_oracle as no


def retention(heads, dim, vdim, decay, rot_dims=0, base=10000.0, ff=None):
    assert len(decay) == heads
    return {"type": "retention",
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay), "rot": {"base": base, "dims": rot_dims}},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def latent(heads, dim, vdim, q_rank, kv_rank, scale=None, ff=None):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                      "scale": dim ** -0.5 if scale is None else scale},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(width, vocab, layers, groups=1, streams=1, loop=None, scale=1.0, mult=1.0, eps=1e-5):
    return {"architecture": "Nololix", "width": width, "vocab": vocab, "embedding": {"scale": scale},
            "norm": {"eps": eps, "groups": groups}, "streams": streams, "residual_mult": mult,
            "loop": None if loop is None else dict(zip(("start", "stop", "times"), loop)), "layers": layers}


def random_tensors(cfg, seed, qk_gain=1.5):
    """Weights of O(1) activations; gains away from 1, the streams' mixing matrices away from the identity and from
    symmetry, activation parameters of both signs, so that nothing drops out by accident."""
    rng = np.random.default_rng(seed)
    W, V, s = cfg["width"], cfg["vocab"], cfg["streams"]
    t = {}

    def mat(name, n, k, gain=1.0):
        t[name] = rng.standard_normal((n, k)) * gain / np.sqrt(k)

    def gains(name, n):
        t[name] = rng.uniform(0.6, 1.4, n)

    t["embed"] = rng.standard_normal((V, W))
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        x = p + "mix."
        H = m["heads"]
        for q in (1, 2) if layer["mlp"] else (1,):
            gains(f"{p}norm{q}", W)
            t[f"{p}hc{q}.in"] = rng.uniform(-0.5, 1.0, s) + 0.3
            t[f"{p}hc{q}.out"] = rng.uniform(0.6, 1.4, s)
            t[f"{p}hc{q}.mix"] = np.eye(s) * rng.uniform(0.7, 1.0, s) + 0.2 * rng.standard_normal((s, s))
        if layer["type"] == "retention":
            mat(x + "q", H * m["dim"], W, qk_gain)
            mat(x + "k", H * m["dim"], W, qk_gain)
            mat(x + "v", H * m["vdim"], W)
            mat(x + "g", H * m["vdim"], W)
        else:
            mat(x + "dq", m["q_rank"], W)
            gains(x + "dq.norm", m["q_rank"])
            mat(x + "uq", H * m["dim"], m["q_rank"], qk_gain)
            mat(x + "dkv", m["kv_rank"], W)
            gains(x + "dkv.norm", m["kv_rank"])
            mat(x + "uk", H * m["dim"], m["kv_rank"], qk_gain)
            mat(x + "uv", H * m["vdim"], m["kv_rank"])
            mat(x + "g", H * m["vdim"], W)
        mat(x + "o", W, H * m["vdim"])
        if layer["mlp"]:
            ff = layer["mlp"]["ff"]
            mat(p + "mlp.up", ff, W)
            mat(p + "mlp.down", W, ff)
            t[p + "mlp.act"] = rng.uniform(-1.0, 1.0, 2)
    gains("final.norm", W)
    mat("head", V, W)
    return {k: ll.bf16_round(v) for k, v in t.items()}


def make_model(folder, cfg, seed=1, **kw):
    tensors = random_tensors(cfg, seed, **kw)
    return ll.write_model(folder, cfg, tensors), no.Model(cfg, tensors)


# Sizes that share nothing with one another: one to five streams, norms over the whole row and over parts, heads
# of odd sizes (values the vector kernels cannot take among them), no, partial and full rotation, decays up to 1, latents on
# either side of the tensor-core kernels' instances, layers without a feed-forward, a loop at the start, in the middle, at the
# end, and none.
CONFIGS = {
    "mixed": config(112, 130, [retention(5, 24, 40, (0.9, 0.97, 0.99, 0.995, 0.999), 16, 500.0, ff=72), latent(3, 20, 24, 36, 44, ff=100),
                               retention(2, 48, 20, (0.98, 0.5), 48), latent(4, 32, 12, 28, 72, scale=0.3)],
                    groups=7, streams=3, loop=(1, 3, 2), scale=3.0, mult=0.4),
    "retention": config(72, 67, [retention(1, 136, 20, (0.995,), 0, ff=40), retention(3, 9, 33, (1.0, 0.25, 0.96), 6, 50.0),
                                 retention(2, 64, 128, (0.9, 0.999), 32, ff=36)], groups=1, streams=1, eps=1e-6),
    "latent": config(96, 200, [latent(20, 16, 8, 24, 200, ff=64), latent(2, 40, 56, 72, 128), latent(7, 12, 20, 8, 24, scale=0.5)],
                     groups=3, streams=2, loop=(0, 3, 2), scale=0.7, mult=0.6),
    "odd": config(63, 57, [latent(3, 21, 24, 33, 100, ff=35), retention(3, 14, 11, (0.95, 0.99, 0.9), 10, ff=41), latent(5, 40, 9, 17, 75)],
                  groups=9, streams=4, loop=(0, 2, 2), scale=2.0, mult=0.4),
    "wide": config(200, 96, [latent(2, 72, 100, 120, 300, ff=136), retention(4, 40, 72, (0.99, 0.93, 0.997, 0.9999), 24, ff=88),
                             retention(1, 16, 8, (0.9,), 16)], groups=10, streams=5, loop=(2, 3, 3), scale=8.0, mult=0.4),
}
