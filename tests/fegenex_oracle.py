"""A plain, slow implementation of the Fegenex design in numpy float64: one function per mechanism, whole sequences
only, no cache and no batching. Test oracle; it shares no code with the product path."""

from __future__ import annotations

import numpy as np


def rms_norm(x, gain, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * gain


def sigmoid(x):
    return np.where(x >= 0, 1.0 / (1.0 + np.exp(-np.abs(x))), np.exp(-np.abs(x)) / (1.0 + np.exp(-np.abs(x))))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return np.logaddexp(0.0, x)


def gelu_tanh(x):
    return 0.5 * x * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (x + 0.044715 * x ** 3)))


def linear(x, w, b=None):
    y = x @ w.T
    return y if b is None else y + b


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


def mixed_head_attention(q, k, v, scale, talk):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]: causal softmax per head, then the heads' weights are
    combined with talk [H, H] before they meet the values."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        w = np.zeros((H, i + 1))
        for h in range(H):
            s = k[:i + 1, h * G // H] @ q[i, h] * scale
            e = np.exp(s - s.max())
            w[h] = e / e.sum()
        w = talk @ w
        for h in range(H):
            out[i, h] = w[h] @ v[:i + 1, h * G // H]
    return out


def blend_values(v, v_first, lam):
    return (1.0 - lam) * v + lam * v_first.reshape(v.shape)  # the token's values as one vector, however cut into heads


def min_gru(h, Wz, bz, Wx, bx, Wg, Wo, state=None):
    z = sigmoid(linear(h, Wz, bz))
    u = linear(h, Wx, bx)
    cand = np.where(u >= 0, u + 0.5, sigmoid(u))
    S = np.zeros(z.shape[1]) if state is None else state
    rows = []
    for t in range(len(h)):
        S = (1.0 - z[t]) * S + z[t] * cand[t]
        rows.append(S)
    return linear(np.array(rows) * silu(linear(h, Wg)), Wo)


def causal_conv(x, w, b):
    """x [T, C], w [C, taps]; the last column of w meets the current token."""
    T, taps = len(x), w.shape[1]
    out = np.tile(b, (T, 1))
    for t in range(T):
        for j in range(taps):
            if t - (taps - 1 - j) >= 0:
                out[t] = out[t] + w[:, j] * x[t - (taps - 1 - j)]
    return out


def block_linear(x, w, b):
    """w [blocks, n, n], b [blocks, n]: each part of x meets its own square matrix."""
    n = w.shape[1]
    return np.concatenate([x[:, i * n:(i + 1) * n] @ w[i].T + b[i] for i in range(len(w))], axis=1)


def rg_lru(u, ra, rab, ri, rib, lam):
    r, i = sigmoid(block_linear(u, ra, rab)), sigmoid(block_linear(u, ri, rib))
    log_a = -8.0 * r * softplus(lam)
    a, gain = np.exp(log_a), np.sqrt(-np.expm1(2.0 * log_a))
    S = np.zeros(u.shape[1])
    rows = []
    for t in range(len(u)):
        S = a[t] * S + gain[t] * i[t] * u[t]
        rows.append(S)
    return np.array(rows)


class Model:
    def __init__(self, cfg, tensors):
        self.cfg = cfg
        self.w = {k: np.asarray(v, dtype=np.float64) for k, v in tensors.items()}

    def layers(self, tokens, positions=None):
        """The residual stream after every layer, [layers, T, width]."""
        cfg, w = self.cfg, self.w
        eps = cfg["norm"]["eps"]
        tokens = np.asarray(tokens)
        pos = np.arange(len(tokens)) if positions is None else positions
        x = w["embed"][tokens] + w["pos"][pos]
        first = None
        out = []
        for n, layer in enumerate(cfg["layers"]):
            p, m = f"l{n}.", layer["mixer"]
            g = lambda name: w[p + "mix." + name]
            h = rms_norm(x, w[p + "norm1"], eps)
            if layer["type"] == "attention":
                T, H, G = len(tokens), m["heads"], m["kv_heads"]
                q = linear(h, g("q"), g("q.b")).reshape(T, H, m["dim"])
                k = linear(h, g("k"), g("k.b")).reshape(T, G, m["dim"])
                v = linear(h, g("v"), g("v.b")).reshape(T, G, m["vdim"])
                q = rope(q, pos, m["rot"]["dims"], m["rot"]["base"])
                k = rope(k, pos, m["rot"]["dims"], m["rot"]["base"])
                if m["v_mix"]:
                    if first is None:
                        first = v
                    else:
                        v = blend_values(v, first, g("vmix"))
                y = mixed_head_attention(q, k, v, m["scale"], g("talk"))
                y = linear(y.reshape(T, -1), g("o"), g("o.b"))
            elif layer["type"] == "mingru":
                y = min_gru(h, g("z"), g("z.b"), g("x"), g("x.b"), g("g"), g("o"))
            else:
                assert layer["type"] == "rglru"
                u = causal_conv(linear(h, g("x"), g("x.b")), g("conv"), g("conv.b"))
                S = rg_lru(u, g("ra"), g("ra.b"), g("ri"), g("ri.b"), g("lam"))
                y = linear(S * gelu_tanh(linear(h, g("y"), g("y.b"))), g("o"))
            x = x + rms_norm(y, w[p + "norm1b"], eps)
            if layer["mlp"] is not None:
                h = rms_norm(x, w[p + "norm2"], eps)
                y = linear(gelu_tanh(linear(h, w[p + "mlp.gate"])) * linear(h, w[p + "mlp.up"]), w[p + "mlp.down"])
                x = x + rms_norm(y, w[p + "norm2b"], eps)
            out.append(x)
        return np.array(out)

    def logits(self, tokens, positions=None):
        x = self.layers(tokens, positions)[-1]
        return linear(rms_norm(x, self.w["final.norm"], self.cfg["norm"]["eps"]), self.w["head"])
