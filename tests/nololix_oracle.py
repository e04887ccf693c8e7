"""A plain, slow implementation of the Nololix design in numpy float64: one function per mechanism, whole sequences only,
no cache and no batching. Test oracle; it shares no code with the product path."""

from __future__ import annotations

import numpy as np


def rms_norm(x, w, eps, groups=1):
    """Every one of `groups` equal consecutive parts of the last axis over its own root mean square, then times w."""
    parts = x.reshape(x.shape[:-1] + (groups, -1))
    parts = parts / np.sqrt(np.mean(parts * parts, axis=-1, keepdims=True) + eps)
    return parts.reshape(x.shape) * w


def sigmoid(x):
    return np.where(x >= 0, 1.0 / (1.0 + np.exp(-np.abs(x))), np.exp(-np.abs(x)) / (1.0 + np.exp(-np.abs(x))))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return np.logaddexp(0.0, x)


def xielu(z, p, q):
    """Quadratic above zero, exponential below, half the identity in both."""
    below = np.minimum(z, 0.0)
    return np.where(z > 0, softplus(p) * z * z, (0.5 + softplus(q)) * (np.expm1(below) - below)) + 0.5 * z


def linear(x, w):
    return x @ w.T


def rope(x, positions, dims, base):
    """x [T, heads, d]; the first `dims` of a head turn, dimension i together with i + dims / 2."""
    half = dims // 2
    out = x.copy()
    for i in range(half):
        ang = positions * base ** (-2.0 * i / dims)
        c, s = np.cos(ang)[:, None], np.sin(ang)[:, None]
        u, v = x[:, :, i], x[:, :, i + half]
        out[:, :, i] = u * c - v * s
        out[:, :, i + half] = v * c + u * s
    return out


def retention(q, k, v, decay, state=None):
    """q, k [T, H, d] (k already scaled), v [T, H, dv] -> outputs [T, H, dv] and the state [H, d, dv] after the last token:
    S = decay S + k v^T, o = S^T q."""
    T, H, d = q.shape
    S = np.zeros((H, d, v.shape[2])) if state is None else state
    out = np.zeros(v.shape)
    g = np.asarray(decay, dtype=np.float64)[:, None, None]
    for t in range(T):
        S = g * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hdv,hd->hv", S, q[t])
    return out, S


def softmax_attention(q, k, v, scale):
    """q, k [T, H, d], v [T, H, dv] -> [T, H, dv], causal."""
    T, H, _ = q.shape
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        s = np.einsum("hd,jhd->hj", q[i], k[:i + 1]) * scale
        e = np.exp(s - s.max(axis=1, keepdims=True))
        out[i] = np.einsum("hj,jhd->hd", e / e.sum(axis=1, keepdims=True), v[:i + 1])
    return out


def retention_mixer(h, positions, m, get, eps):
    T, H, d, dv = len(h), m["heads"], m["dim"], m["vdim"]
    q = rope(linear(h, get("q")).reshape(T, H, d), positions, m["rot"]["dims"], m["rot"]["base"])
    k = rope(linear(h, get("k")).reshape(T, H, d), positions, m["rot"]["dims"], m["rot"]["base"]) * d ** -0.5
    o, _ = retention(q, k, linear(h, get("v")).reshape(T, H, dv), m["decay"])
    o = rms_norm(o, 1.0, eps).reshape(T, -1) * silu(linear(h, get("g")))
    return linear(o, get("o"))


def latent_mixer(h, m, get, eps):
    T, H, d, dv = len(h), m["heads"], m["dim"], m["vdim"]
    q = linear(rms_norm(linear(h, get("dq")), get("dq.norm"), eps), get("uq")).reshape(T, H, d)
    c = rms_norm(linear(h, get("dkv")), get("dkv.norm"), eps)
    k, v = linear(c, get("uk")).reshape(T, H, d), linear(c, get("uv")).reshape(T, H, dv)
    o = softmax_attention(q, k, v, m["scale"]).reshape(T, -1)
    return linear(o * sigmoid(linear(h, get("g"))), get("o"))


def hyper_update(x, y, mix, out, mult):
    """x [s, T, W] streams, all replaced at once from the old ones; mix is [from, to]."""
    return np.einsum("st,sjw->tjw", mix, x) + mult * out[:, None, None] * y[None]


def run_order(cfg):
    """Layer indices in the order they run, the looped span repeated."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


class Model:
    def __init__(self, cfg, tensors):
        self.cfg = cfg
        self.w = {k: np.asarray(v, dtype=np.float64) for k, v in tensors.items()}

    def layers(self, tokens, positions=None):
        """The sum of the streams after every layer run, [runs, T, width]."""
        cfg, w = self.cfg, self.w
        eps, groups, mult = cfg["norm"]["eps"], cfg["norm"]["groups"], cfg["residual_mult"]
        tokens = np.asarray(tokens)
        pos = np.arange(len(tokens)) if positions is None else positions
        x = np.repeat((w["embed"][tokens] * cfg["embedding"]["scale"])[None], cfg["streams"], axis=0)
        out = []
        for n in run_order(cfg):
            p, layer = f"l{n}.", cfg["layers"][n]
            get = lambda name: w[p + "mix." + name]

            def sublayer(q, f, x):
                hc = lambda name: w[f"{p}hc{q}.{name}"]
                u = np.einsum("s,sjw->jw", hc("in"), x)
                return hyper_update(x, f(rms_norm(u, w[f"{p}norm{q}"], eps, groups)), hc("mix"), hc("out"), mult)

            if layer["type"] == "retention":
                x = sublayer(1, lambda h: retention_mixer(h, pos, layer["mixer"], get, eps), x)
            else:
                assert layer["type"] == "latent_attention"
                x = sublayer(1, lambda h: latent_mixer(h, layer["mixer"], get, eps), x)
            if layer["mlp"] is not None:
                a, b = w[p + "mlp.act"]
                x = sublayer(2, lambda h: linear(xielu(linear(h, w[p + "mlp.up"]), a, b), w[p + "mlp.down"]), x)
            out.append(x.sum(axis=0))
        return np.array(out)

    def logits(self, tokens, positions=None):
        cfg = self.cfg
        x = self.layers(tokens, positions)[-1]
        return linear(rms_norm(x, self.w["final.norm"], cfg["norm"]["eps"], cfg["norm"]["groups"]), self.w["head"])
