"""Kernels of the layer-list architectures through the C ABI, each against a plain fp32 / fp64 computation."""

import ctypes as C

import numpy as np
import pytest
import torch

import fegenex_oracle as fo
from q38_testlib import pkg

pytestmark = pytest.mark.gpu


def up(x, to):
    return (x + to - 1) // to * to


def dev(a, dtype=torch.float32):
    return torch.as_tensor(np.ascontiguousarray(a)).to("cuda", dtype)


def bf16(a):
    return torch.as_tensor(np.asarray(a)).to(torch.bfloat16).to(torch.float64).numpy()


class DenseWeight:
    """W [n][k] and bias on the device in the padded layout the kernels take."""

    def __init__(self, w, bias=None):
        n, k = w.shape
        self.ld = up(k, 64)
        self.w = torch.zeros((up(n, 16), self.ld), dtype=torch.bfloat16, device="cuda")
        self.w[:n, :k] = dev(w, torch.bfloat16)
        self.b = None
        if bias is not None:
            self.b = torch.zeros(up(n, 16), dtype=torch.float32, device="cuda")
            self.b[:n] = dev(bias)
        self.desc = pkg.DenseWeight(pkg.ptr(self.w), pkg.ptr(self.b), n, k, self.ld)


def run_gemm(x, w, kind, out_cols, act, config=-1, ldo=None):
    m, k = x.shape
    tdt = torch.bfloat16 if act == pkg.ACT_BF16 else torch.float32
    ldx, ldo = up(k, 64), ldo or out_cols
    xd = torch.zeros((m, ldx), dtype=tdt, device="cuda")
    xd[:, :k] = dev(x, tdt)
    out = torch.full((m, ldo), 7.0, dtype=torch.float32 if kind == pkg.DENSE_STORE_F32 else tdt, device="cuda")
    ep = pkg.DenseEpilogue(kind, pkg.ptr(out), ldo)
    pkg.check(pkg.kernels().q38_dense_gemm(pkg.ptr(xd), ldx, act, m, C.byref(w.desc), C.byref(ep), None, None, config))
    torch.cuda.synchronize()
    assert pkg.kernels().q38_device_error(1) == 0
    return out.double().cpu().numpy()


@pytest.mark.parametrize("n,k", [(384, 256), (200, 72), (96, 1000), (1042, 520), (16, 8)])
@pytest.mark.parametrize("m", [1, 5, 16, 17, 40, 130, 300])
def test_dense_gemm_every_kernel(n, k, m):
    rng = np.random.default_rng(n + k + m)
    x, wt, b = bf16(rng.standard_normal((m, k))), bf16(rng.standard_normal((n, k)) / np.sqrt(k)), rng.standard_normal(n)
    w = DenseWeight(wt, b)
    want = x @ wt.T + b.astype(np.float32)
    names = [pkg.kernels().q38_dense_gemm_config_name(i).decode() for i in range(pkg.kernels().q38_dense_gemm_num_configs())]
    for i, name in [(-1, "auto")] + list(enumerate(names)):
        if "cluster" in name and (k + 63) // 64 < int(name[-1]):
            continue
        got = run_gemm(x, w, pkg.DENSE_STORE_F32, n, pkg.ACT_BF16, i, ldo=n + 3)
        assert np.all(got[:, n:] == 7.0)
        assert np.abs(got[:, :n] - want).max() < 2e-4, name
        got = run_gemm(x, w, pkg.DENSE_STORE, n, pkg.ACT_BF16, i, ldo=n + 6)
        assert np.all(got[:, n:] == 7.0)
        assert np.all(np.abs(got[:, :n] - want) < 2e-4 + np.abs(want) / 256), name
        again = run_gemm(x, w, pkg.DENSE_STORE_F32, n, pkg.ACT_BF16, i)
        assert np.array_equal(again, run_gemm(x, w, pkg.DENSE_STORE_F32, n, pkg.ACT_BF16, i)), name
        for kind, act in ((pkg.DENSE_GLU_GELU, fo.gelu_tanh), (pkg.DENSE_GLU_SILU, fo.silu)):
            got = run_gemm(x, w, kind, n // 2, pkg.ACT_BF16, i)
            product = act(want[:, 0::2]) * want[:, 1::2]
            assert np.all(np.abs(got - product) < 1e-3 + np.abs(product) / 256), name
    x32 = rng.standard_normal((m, k))
    got = run_gemm(x32, w, pkg.DENSE_STORE, n, pkg.ACT_F32)
    assert np.abs(got - (x32.astype(np.float32).astype(np.float64) @ wt.T + b)).max() < 1e-5


# ---- norms ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("act", [pkg.ACT_BF16, pkg.ACT_F32])
@pytest.mark.parametrize("width,stride", [(64, 0), (333, 0), (1000, 1), (30, 1)])
def test_norm_kernels(act, width, stride):
    rng = np.random.default_rng(width)
    K, tdt, eps, m = pkg.kernels(), torch.bfloat16 if act == pkg.ACT_BF16 else torch.float32, 1e-3, 5
    tol = (0.01 if act == pkg.ACT_BF16 else 1e-5) * 4
    gains = [dev(rng.uniform(0.5, 2.0, width if stride else 1)) for _ in range(2)]
    norms = [pkg.Norm(pkg.ptr(g), stride, eps) for g in gains]
    gn = [g.double().cpu().numpy() for g in gains]
    table, pos = bf16(rng.standard_normal((20, width))), bf16(rng.standard_normal((9, width)))
    tokens, at = np.array([3, 19, 0, 3, 7]), np.array([0, 8, 2, 3, 4])
    td, pd = dev(table, torch.bfloat16), dev(pos, torch.bfloat16)
    tok, atd = dev(tokens, torch.int32), dev(at, torch.int32)
    res, out = torch.empty((m, width), device="cuda"), torch.zeros((m, width + 7), dtype=tdt, device="cuda")
    x = table[tokens] + pos[at]
    pkg.check(K.q38_embed_norm(pkg.ptr(td), pkg.ptr(pd), pkg.ptr(tok), pkg.ptr(atd), m, width, pkg.ptr(res),
                               C.byref(norms[0]), pkg.ptr(out), width + 7, act, None))
    assert np.allclose(res.double().cpu().numpy(), x, atol=1e-6)
    assert np.allclose(out[:, :width].double().cpu().numpy(), fo.rms_norm(x, gn[0], eps), atol=tol)
    y = rng.standard_normal((m, width + 3)).astype(np.float32)
    yd = dev(y)
    pkg.check(K.q38_residual_norm(pkg.ptr(yd), width + 3, m, width, C.byref(norms[0]), pkg.ptr(res), C.byref(norms[1]),
                                  pkg.ptr(out), width + 7, act, None))
    x = x + fo.rms_norm(y[:, :width].astype(np.float64), gn[0], eps)
    assert np.allclose(res.double().cpu().numpy(), x, atol=1e-5)
    assert np.allclose(out[:, :width].double().cpu().numpy(), fo.rms_norm(x, gn[1], eps), atol=tol)
    assert np.all(out[:, width:].double().cpu().numpy() == 0)
    pkg.check(K.q38_residual_norm(pkg.ptr(yd), width + 3, m, width, C.byref(norms[1]), pkg.ptr(res), None, None, 0, act, None))
    x = x + fo.rms_norm(y[:, :width].astype(np.float64), gn[1], eps)
    assert np.allclose(res.double().cpu().numpy(), x, atol=1e-5)
    rows = dev(np.array([4, 1, 1]), torch.int32)
    for r, first, want in ((rows, 0, [4, 1, 1]), (None, 2, [2, 3, 4])):
        pkg.check(K.q38_gather_norm(pkg.ptr(res), pkg.ptr(r), first, 3, width, C.byref(norms[1]), pkg.ptr(out), width + 7, act, None))
        assert np.allclose(out[:3, :width].double().cpu().numpy(), fo.rms_norm(x[want], gn[1], eps), atol=tol)
    torch.cuda.synchronize()


# ---- ragged batches ----------------------------------------------------------------------------------------------------------
class Batch:
    """rows: (slot, pos0, count) per sequence; one-token rows last, as the runner orders them."""

    def __init__(self, rows):
        self.rows = rows
        start = np.concatenate([[0], np.cumsum([r[2] for r in rows])])
        self.m = int(start[-1])
        pos = np.concatenate([np.arange(p, p + n) for _, p, n in rows])
        seq = np.concatenate([np.full(n, i) for i, (_, _, n) in enumerate(rows)])
        self.arr = [dev(a, torch.int32) for a in (start, [r[0] for r in rows], [r[1] for r in rows], pos, seq)]
        self.desc = self.part(0, len(rows))

    def part(self, a, b):
        first = sum(r[2] for r in self.rows[:a])
        start, slot, pos0, pos, seq = [x.data_ptr() for x in self.arr]
        rows = self.rows[a:b]
        return pkg.BatchDesc(len(rows), sum(r[2] for r in rows), max(r[2] for r in rows), start + 4 * a, slot + 4 * a,
                             pos0 + 4 * a, pos + 4 * first, seq + 4 * first)


class Cache:
    def __init__(self, G, dim, vdim, slots, max_pages, act, seed=0):
        self.tdt = torch.bfloat16 if act == pkg.ACT_BF16 else torch.float32
        self.G, self.kd, self.vd = G, up(dim, 32), up(vdim, 8)
        pages = slots * max_pages + 3
        self.elems = G * 64 * (self.kd + self.vd)
        rng = np.random.default_rng(seed)
        # pages that were used before: finite leftovers everywhere
        self.pool = dev(rng.standard_normal((pages, self.elems)) * 3, self.tdt)
        self.table = dev(rng.permutation(pages)[:slots * max_pages].reshape(slots, max_pages), torch.int32)
        es = self.pool.element_size()
        self.desc = pkg.KvLayerDesc(pkg.ptr(self.pool), pkg.KV_BF16 if act == pkg.ACT_BF16 else pkg.KV_F32, G, self.kd,
                                    self.vd, pages, self.elems * es, pkg.ptr(self.table), max_pages)
        self.pages = pages


def rounded(a, act):
    return bf16(a) if act == pkg.ACT_BF16 else np.asarray(a, dtype=np.float32).astype(np.float64)


# heads, kv heads, dim, vdim, rotated dims
SHAPES = [(4, 2, 40, 24, 16), (3, 3, 80, 56, 20), (20, 1, 24, 24, 8), (8, 1, 64, 128, 64), (16, 4, 128, 128, 32), (1, 1, 24, 8, 24),
          (6, 6, 32, 200, 8), (20, 2, 72, 136, 0), (2, 2, 256, 256, 64), (32, 8, 64, 64, 64), (5, 1, 288, 40, 10), (16, 16, 128, 128, 32), (32, 8, 128, 128, 128),
          (9, 3, 16, 300, 6)]


@pytest.mark.parametrize("act", [pkg.ACT_BF16, pkg.ACT_F32])
@pytest.mark.parametrize("shape", SHAPES)
def test_attention_against_the_plain_one(shape, act):
    """Prompts in portions, then decoded tokens, through one shuffled cache: rotation, blending, append, head mixing; keys
    that stand out far away, at a page's first and last token, at the row itself and just behind the causal limit."""
    H, G, dim, vdim, rot = shape
    rng = np.random.default_rng(sum(shape))
    base, scale, lam = 300.0, 0.8 / np.sqrt(dim), 0.4
    lens = [150, 77]
    total = sum(lens)
    K = pkg.kernels()
    cache = Cache(G, dim, vdim, 4, 3, act)
    width = H * dim + G * (dim + vdim)
    proj = rng.standard_normal((total, width))
    first = rounded(rng.standard_normal((total, G * vdim)), act)
    # stand-out pairs: key j of a head looks like the query of row i (the same row's key is made large as well)
    for lo, n in ((0, 150), (150, 77)):
        for i, j in ((n - 1, 0), (n - 1, 63), (n - 2, 64), (70, 3), (64, 63), (65, 66), (n - 5, n - 4), (20, 20)):
            h = (i + j) % H
            kv = H * dim + (h * G // H) * dim
            proj[lo + j, kv:kv + dim] = 3.0 * proj[lo + i, h * dim:(h + 1) * dim]
    proj = rounded(proj, act)
    T = (np.eye(H) + 0.5 * rng.standard_normal((H, H))).astype(np.float32)
    Td, lamd = dev(T), dev(np.array([lam]))
    freq = dev(base ** (-2.0 * np.arange(max(1, rot // 2)) / max(1, rot)), torch.float64)
    ws_stats = torch.zeros(8 * total * H * 2, device="cuda")
    scores = torch.zeros(cache.pages * H * 64, device="cuda")
    partials = torch.zeros(4 * 16 * H * (cache.vd + 2), device="cuda")
    done, outs = [0, 0], [np.zeros((n, H * vdim)) for n in lens]
    v_first_kept = []
    schedule = [[(0, 64), (1, 2)], [(1, 30), (0, 63)], [(0, 2), (1, 44)], [(0, 19), (1, 1)], [(0, 1)], [(0, 1)]]
    for step in schedule:
        rows = [(2 * s + 1, done[s], n) for s, n in step]  # slots 1 and 3
        b = Batch(rows)
        src = np.concatenate([np.arange(done[s], done[s] + n) + (0 if s == 0 else 150) for s, n in step])
        pd, fd = dev(proj[src], cache.tdt), dev(first[src], cache.tdt)
        q = torch.full((b.m, H * cache.kd), 5.0, dtype=cache.tdt, device="cuda")
        keep = torch.zeros((b.m, G * vdim), dtype=cache.tdt, device="cuda")
        rp = pkg.RopeAppendParams(pkg.ptr(pd), width, act, H, G, dim, vdim, rot, pkg.ptr(freq), pkg.ptr(q), pkg.ptr(keep), pkg.ptr(fd),
                                  pkg.ptr(lamd))
        pkg.check(K.q38_rope_append(C.byref(rp), C.byref(b.desc), C.byref(cache.desc), None))
        v_first_kept.append((src, keep))
        out = torch.zeros((b.m, H * vdim + 5), dtype=cache.tdt, device="cuda")
        ap = pkg.MixedAttentionParams(pkg.ptr(q), act, H, vdim, scale, pkg.ptr(Td), pkg.ptr(out), H * vdim + 5, pkg.ptr(ws_stats),
                                      8, pkg.ptr(scores), pkg.ptr(partials), 16)
        multi = sum(n > 1 for _, n in step)
        if multi:
            part = b.part(0, multi)
            pkg.check(K.q38_mixed_attention_prefill(C.byref(ap), C.byref(part), C.byref(cache.desc), None))
        if multi < len(step):
            part = b.part(multi, len(step))
            pkg.check(K.q38_mixed_attention_decode(C.byref(ap), C.byref(part), C.byref(cache.desc), None))
        torch.cuda.synchronize()
        got, at = out.double().cpu().numpy(), 0
        assert np.all(got[:, H * vdim:] == 0)
        for s, n in step:
            outs[s][done[s]:done[s] + n] = got[at:at + n, :H * vdim]
            done[s], at = done[s] + n, at + n
    assert done == lens and K.q38_device_error(1) == 0
    for src, keep in v_first_kept:  # the values before blending, for the layers that blend with them
        assert np.array_equal(keep.double().cpu().numpy(), proj[src][:, H * dim + G * dim:])
    for s, (lo, n) in enumerate(((0, 150), (150, 77))):
        p = proj[lo:lo + n]
        qr = rounded(fo.rope(p[:, :H * dim].reshape(n, H, dim), np.arange(n), rot, base) if rot else p[:, :H * dim].reshape(n, H, dim), act)
        kr = p[:, H * dim:(H + G) * dim].reshape(n, G, dim)
        kr = rounded(fo.rope(kr, np.arange(n), rot, base) if rot else kr, act)
        v = rounded(fo.blend_values(p[:, (H + G) * dim:].reshape(n, G, vdim), first[lo:lo + n], lam), act)
        want = fo.mixed_head_attention(qr, kr, v, scale, T.astype(np.float64)).reshape(n, -1)
        err = np.abs(outs[s] - want).max() / np.abs(want).max()
        assert err < (1.2e-2 if act == pkg.ACT_BF16 else 1e-5), (s, err)


@pytest.mark.parametrize("act", [pkg.ACT_BF16, pkg.ACT_F32])
def test_attention_without_mixing_and_with_many_splits(act):
    """head_mix NULL is plain grouped attention; one long context whose decode is cut over many splits equals few."""
    H, G, dim, vdim, n = 4, 2, 64, 32, 1500
    rng = np.random.default_rng(7)
    K = pkg.kernels()
    cache = Cache(G, dim, vdim, 1, 24, act)
    width = H * dim + G * (dim + vdim)
    proj = rounded(rng.standard_normal((n, width)), act)
    proj[5, H * dim:H * dim + dim] = 2 * proj[-1, :dim]  # a far key that the last query must find
    freq = dev(1e4 ** (-2.0 * np.arange(32) / 64), torch.float64)
    outs = []
    stats = torch.zeros(8 * n * H * 2, device="cuda")
    scores = torch.zeros(cache.pages * H * 64, device="cuda")
    for splits in (1, 3, 24):
        b0, b1 = Batch([(0, 0, n - 1)]), Batch([(0, n - 1, 1)])
        for b, rows in ((b0, proj[:-1]), (b1, proj[-1:])):
            pd = dev(rows, cache.tdt)
            q = torch.zeros((b.m, H * cache.kd), dtype=cache.tdt, device="cuda")
            rp = pkg.RopeAppendParams(pkg.ptr(pd), width, act, H, G, dim, vdim, 64, pkg.ptr(freq), pkg.ptr(q), None, None, None)
            pkg.check(K.q38_rope_append(C.byref(rp), C.byref(b.desc), C.byref(cache.desc), None))
        out = torch.zeros((1, H * vdim), dtype=cache.tdt, device="cuda")
        partials = torch.full((splits * H * (cache.vd + 2),), float("nan"), device="cuda")
        ap = pkg.MixedAttentionParams(pkg.ptr(q), act, H, vdim, 0.125, None, pkg.ptr(out), H * vdim, pkg.ptr(stats), 8,
                                      pkg.ptr(scores), pkg.ptr(partials), splits)
        pkg.check(K.q38_mixed_attention_decode(C.byref(ap), C.byref(b1.desc), C.byref(cache.desc), None))
        torch.cuda.synchronize()
        outs.append(out.double().cpu().numpy().reshape(H, vdim))
    qr = rounded(fo.rope(proj[-1:, :H * dim].reshape(1, H, dim), np.array([n - 1]), 64, 1e4), act)[0]
    kr = rounded(fo.rope(proj[:, H * dim:(H + G) * dim].reshape(n, G, dim), np.arange(n), 64, 1e4), act)
    v = proj[:, (H + G) * dim:].reshape(n, G, vdim)
    for h in range(H):
        s = kr[:, h // 2] @ qr[h] * 0.125
        w = np.exp(s - s.max())
        want = w @ v[:, h // 2] / w.sum()
        for o in outs:
            assert np.abs(o[h] - want).max() < (1.5e-2 if act == pkg.ACT_BF16 else 2e-5)


# ---- recurrences --------------------------------------------------------------------------------------------------------------
class State:
    def __init__(self, width, taps, act, slots=4):
        es = 2 if act == pkg.ACT_BF16 else 4
        self.conv_off = up(width * 4, 256)
        self.slot = self.conv_off + up(max(1, taps * width * es), 256)
        # leftovers of an earlier sequence: a fresh one must not see them
        self.mem = dev(np.random.default_rng(1).standard_normal(slots * self.slot // 4), torch.float32)
        self.desc = pkg.RecurrentStateDesc(self.mem.data_ptr(), self.mem.data_ptr() + self.conv_off, self.slot)


def run_recurrence(call, proj, lens, act, out_width):
    """Two sequences in uneven portions (down to two tokens, and single tokens) -> their outputs."""
    tdt = torch.bfloat16 if act == pkg.ACT_BF16 else torch.float32
    done, outs = [0, 0], [np.zeros((n, out_width)) for n in lens]
    portions = [[(0, 2), (1, 2)], [(0, 3), (1, 1)], [(0, 300), (1, 2)], [(1, 40), (0, 1)], [(0, 1), (1, 1)], [(0, 1)], [(0, lens[0] - 308), (1, lens[1] - 46)]]
    for step in portions:
        b = Batch([(s + 1, done[s], n) for s, n in step])
        src = np.concatenate([np.arange(done[s], done[s] + n) + (0 if s == 0 else lens[0]) for s, n in step])
        pd = dev(proj[src], tdt)
        out = torch.zeros((b.m, out_width), dtype=tdt, device="cuda")
        multi = sum(n > 1 for _, n in step)
        for a, z in ((multi, len(step)), (0, multi)):  # single-token rows first: the parts are independent
            if a < z:
                call(pd, out, b.part(a, z))
        torch.cuda.synchronize()
        got, at = out.double().cpu().numpy(), 0
        for s, n in step:
            outs[s][done[s]:done[s] + n] = got[at:at + n]
            done[s], at = done[s] + n, at + n
    assert done == list(lens)
    return outs


@pytest.mark.parametrize("act", [pkg.ACT_BF16, pkg.ACT_F32])
@pytest.mark.parametrize("width", [8, 72, 200])
def test_mingru_against_the_plain_one(width, act):
    rng = np.random.default_rng(width)
    lens = (700, 90)
    proj = rng.standard_normal((sum(lens), 3 * width)) * 1.5
    proj[:, :width] -= 3.0  # gates that mostly keep the state: long memory
    proj = rounded(proj, act)
    st = State(width, 0, act)

    def call(pd, out, batch):
        p = pkg.MinGruParams(pkg.ptr(pd), 3 * width, act, width, pkg.ptr(out), width)
        pkg.check(pkg.kernels().q38_mingru(C.byref(p), C.byref(batch), C.byref(st.desc), None))
    outs = run_recurrence(call, proj, lens, act, width)
    eye, zero = np.eye(width), np.zeros(width)
    lo = 0
    for o, n in zip(outs, lens):
        z, x, g = np.split(proj[lo:lo + n], 3, axis=1)
        # the projections are already done: identity weights, each role fed its own input
        S = np.zeros(width)
        want = []
        zz, cand = fo.sigmoid(z), np.where(x >= 0, x + 0.5, fo.sigmoid(x))
        for t in range(n):
            S = (1 - zz[t]) * S + zz[t] * cand[t]
            want.append(S * fo.silu(g[t]))
        whole = fo.min_gru(z, eye, zero, eye, zero, eye, eye)
        assert whole.shape == (n, width)
        want = np.array(want)
        assert np.all(np.abs(o - want) < 1e-5 + (np.abs(want) / 200 if act == pkg.ACT_BF16 else 0))
        lo += n


@pytest.mark.parametrize("act", [pkg.ACT_BF16, pkg.ACT_F32])
@pytest.mark.parametrize("width,blocks,taps", [(64, 2, 4), (96, 3, 3), (72, 1, 1), (144, 2, 2), (40, 8, 6), (512, 2, 4)])
def test_rglru_against_the_plain_one(width, blocks, taps, act):
    rng = np.random.default_rng(width + taps)
    lens = (340, 80)
    proj = rounded(rng.standard_normal((sum(lens), 2 * width)), act)
    bs, ld = width // blocks, up(width // blocks, 32)
    gates = bf16(rng.standard_normal((2, blocks, bs, bs)) / np.sqrt(bs))
    gw = np.zeros((blocks, 2, ld, ld))
    gw[:, :, :bs, :bs] = gates.transpose(1, 0, 2, 3)
    gb, conv = rng.standard_normal((2, width)).astype(np.float32), rng.standard_normal((width, taps)).astype(np.float32)
    cb, lam = rng.standard_normal(width).astype(np.float32), rng.uniform(-8, 1, width).astype(np.float32)
    d = [dev(conv.T), dev(cb), dev(gw, torch.bfloat16), dev(gb), dev(lam)]
    scratch = torch.full((2 * sum(lens) * width,), float("nan"), device="cuda")
    st = State(width, taps, act)

    def call(pd, out, batch):
        p = pkg.RgLruParams(pkg.ptr(pd), 2 * width, act, width, blocks, ld, taps, pkg.ptr(d[0]), pkg.ptr(d[1]), pkg.ptr(d[2]),
                            pkg.ptr(d[3]), pkg.ptr(d[4]), -8.0, pkg.ptr(scratch), pkg.ptr(out), width)
        pkg.check(pkg.kernels().q38_rglru(C.byref(p), C.byref(batch), C.byref(st.desc), None))
    outs = run_recurrence(call, proj, lens, act, width)
    lo = 0
    for o, n in zip(outs, lens):
        y, x = np.split(proj[lo:lo + n], 2, axis=1)
        u = fo.causal_conv(x, conv.astype(np.float64), cb.astype(np.float64))
        S = fo.rg_lru(u, gates[0], gb[0].reshape(blocks, bs), gates[1], gb[1].reshape(blocks, bs), lam.astype(np.float64))
        want = S * fo.gelu_tanh(y)
        err = np.abs(o - want).max() / np.abs(want).max()
        assert err < (6e-3 if act == pkg.ACT_BF16 else 1e-5), err
        lo += n


def test_bad_arguments_are_refused():
    K = pkg.kernels()
    x = torch.zeros((4, 64), dtype=torch.bfloat16, device="cuda")
    w = DenseWeight(np.zeros((16, 64)))
    ep = pkg.DenseEpilogue(9, pkg.ptr(x), 64)
    assert K.q38_dense_gemm(pkg.ptr(x), 64, 0, 4, C.byref(w.desc), C.byref(ep), None, None, -1) == -1
    assert b"epilogue 9" in K.q38_last_error()
    ep = pkg.DenseEpilogue(pkg.DENSE_STORE, pkg.ptr(x), 8)
    assert K.q38_dense_gemm(pkg.ptr(x), 64, 0, 4, C.byref(w.desc), C.byref(ep), None, None, -1) == -1
    assert b"ldo 8" in K.q38_last_error()
    assert K.q38_mingru(None, None, None, None) == -1
