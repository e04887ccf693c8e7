"""Random Fegenex models on disk (config.json + model.safetensors, written here byte by byte) for the tests."""

from __future__ import annotations

import json
import struct

import numpy as np

import fegenex_oracle as fo


def f32_to_bf16_bits(a):
    u = np.array(a, dtype=np.float32, order="C").view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def bf16_round(a):
    return (f32_to_bf16_bits(a).astype(np.uint32) << 16).view(np.float32)


def attention(heads, kv_heads, dim, vdim, rot_dims, base=10000.0, scale=None, v_mix=True, ff=None):
    return {"type": "attention",
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "v_mix": v_mix,
                      "rot": {"base": base, "dims": rot_dims}, "scale": dim ** -0.5 if scale is None else scale},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def mingru(width, ff=None):
    return {"type": "mingru", "mixer": {"width": width}, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def rglru(width, blocks, conv, ff=None):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(width, vocab, layers, max_positions=512, eps=1e-5):
    return {"architecture": "Fegenex", "width": width, "vocab": vocab, "max_positions": max_positions, "norm": {"eps": eps},
            "layers": layers}


def random_tensors(cfg, seed, qk_gain=1.5):
    """Weights of O(1) activations; decays spread over short and long memories, mixing matrices with both signs, gains and
    biases away from 1 and 0, so that nothing drops out by accident."""
    rng = np.random.default_rng(seed)
    W, V = cfg["width"], cfg["vocab"]
    t = {}

    def mat(name, n, k, gain=1.0):
        t[name] = rng.standard_normal((n, k)) * gain / np.sqrt(k)

    def vec(name, n, std=0.3, mean=0.0):
        t[name] = mean + std * rng.standard_normal(n)

    t["embed"] = rng.standard_normal((V, W))
    t["pos"] = 0.5 * rng.standard_normal((cfg["max_positions"], W))
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        for name in ("norm1", "norm1b") + (("norm2", "norm2b") if layer["mlp"] else ()):
            t[p + name] = np.array(rng.uniform(0.7, 1.3))
        x = p + "mix."
        if layer["type"] == "attention":
            H, G = m["heads"], m["kv_heads"]
            for name, n, gain in (("q", H * m["dim"], qk_gain), ("k", G * m["dim"], qk_gain), ("v", G * m["vdim"], 1.0)):
                mat(x + name, n, W, gain)
                vec(x + name + ".b", n)
            mat(x + "o", W, H * m["vdim"])
            vec(x + "o.b", W)
            t[x + "talk"] = np.eye(H) + 0.5 * rng.standard_normal((H, H))
            if m["v_mix"]:
                t[x + "vmix"] = np.array(rng.uniform(0.3, 0.7))
        elif layer["type"] == "mingru":
            for name in "zxg":
                mat(x + name, m["width"], W)
            vec(x + "z.b", m["width"], 1.0, -3.0)
            vec(x + "x.b", m["width"])
            mat(x + "o", W, m["width"])
        else:
            w, nb = m["width"], m["blocks"]
            bs = w // nb
            for name in "yx":
                mat(x + name, w, W)
                vec(x + name + ".b", w)
            t[x + "conv"] = 0.5 * rng.standard_normal((w, m["conv"]))
            vec(x + "conv.b", w)
            for name in ("ra", "ri"):
                t[x + name] = rng.standard_normal((nb, bs, bs)) / np.sqrt(bs)
                t[x + name + ".b"] = 0.3 * rng.standard_normal((nb, bs))
            vec(x + "lam", w, 1.0, -4.0)
            mat(x + "o", W, w)
        if layer["mlp"]:
            ff = layer["mlp"]["ff"]
            mat(p + "mlp.gate", ff, W)
            mat(p + "mlp.up", ff, W)
            mat(p + "mlp.down", W, ff)
    t["final.norm"] = np.array(1.1)
    mat("head", V, W)
    return {k: bf16_round(v) for k, v in t.items()}


def write_safetensors(path, tensors):
    head, data, at = {}, [], 0
    for name, a in tensors.items():
        raw = f32_to_bf16_bits(a).tobytes()
        head[name] = {"dtype": "BF16", "shape": list(np.shape(a)), "data_offsets": [at, at + len(raw)]}
        data.append(raw)
        at += len(raw)
    text = json.dumps(head).encode()
    text += b" " * (-len(text) % 8)
    path.write_bytes(struct.pack("<Q", len(text)) + text + b"".join(data))


def write_model(folder, cfg, tensors):
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    write_safetensors(folder / "model.safetensors", tensors)
    return folder


def make_model(folder, cfg, seed=1, **kw):
    tensors = random_tensors(cfg, seed, **kw)
    return write_model(folder, cfg, tensors), fo.Model(cfg, tensors)


# Sizes that share nothing with one another: grouped and single kv heads, odd head sizes, one and several convolution taps,
# blocks of many sizes, feed-forwards on any kind of layer, value blending that starts late, is absent, or skips a layer.
CONFIGS = {
    "mixed": config(112, 130, [rglru(96, 3, 3, ff=72), attention(6, 2, 40, 24, 16, base=500.0), mingru(80, ff=100),
                               attention(4, 1, 20, 48, 20, scale=0.3, ff=64), attention(3, 3, 32, 16, 8)], 400),
    "recurrent": config(72, 67, [mingru(40), rglru(56, 1, 1), mingru(72, ff=36), rglru(64, 8, 5)], 300, eps=1e-6),
    "attention": config(96, 200, [attention(2, 2, 64, 96, 32, v_mix=False), attention(8, 2, 24, 32, 12, base=2000.0),
                                  attention(5, 5, 16, 8, 4, v_mix=False, ff=50), attention(16, 4, 48, 16, 48)], 600),
    "wide": config(200, 96, [attention(8, 1, 72, 136, 24, ff=136), rglru(160, 4, 4), attention(1, 1, 128, 136, 64),
                             mingru(144)], 260),
}
