"""Kernels of the Nololix design through the C ABI, each against a plain fp64 computation."""

import ctypes as C

import numpy as np
import pytest
import torch

import nololix_oracle as no
from q38_testlib import pkg
from test_layer_list_kernels_gpu import Batch, DenseWeight, bf16, dev, rounded, up

pytestmark = pytest.mark.gpu

ACTS = [pkg.ACT_BF16, pkg.ACT_F32]


def tdt(act):
    return torch.bfloat16 if act == pkg.ACT_BF16 else torch.float32


def clean():
    torch.cuda.synchronize()
    assert pkg.kernels().q38_device_error(1) == 0


# ---- dense products ------------------------------------------------------------------------------------------------------
def gemm_names():
    K = pkg.kernels()
    return [(-1, "auto")] + [(i, K.q38_dense_gemm_config_name(i).decode()) for i in range(K.q38_dense_gemm_num_configs())]


@pytest.mark.parametrize("n,k", [(384, 256), (200, 72), (1042, 520), (17, 8)])
@pytest.mark.parametrize("m", [1, 17, 40, 300])
def test_dense_epilogues_every_kernel(n, k, m):
    """xIELU and the sigmoid gate behind the product, on every kernel and in fp32."""
    rng = np.random.default_rng(n + k + m)
    K = pkg.kernels()
    wt, b = bf16(rng.standard_normal((n, k)) / np.sqrt(k)), rng.standard_normal(n)
    w = DenseWeight(wt, b)
    p, q = 0.4, -0.7
    ap, an = float(no.softplus(p)), float(0.5 + no.softplus(q))
    for act in ACTS:
        x, gate = rounded(rng.standard_normal((m, k)) * 2, act), rounded(rng.standard_normal((m, n)) * 3, act)
        y = x @ wt.T + b.astype(np.float32)
        ldx, ldo, ldg = up(k, 64), n + 6, n + 3
        xd, gd = torch.zeros((m, ldx), dtype=tdt(act), device="cuda"), torch.zeros((m, ldg), dtype=tdt(act), device="cuda")
        xd[:, :k], gd[:, :n] = dev(x, tdt(act)), dev(gate, tdt(act))
        for i, name in gemm_names() if act == pkg.ACT_BF16 else [(-1, "fp32")]:
            if "cluster" in name and (k + 63) // 64 < int(name[-1]):
                continue
            for kind, want in ((pkg.DENSE_XIELU, no.xielu(y, p, q)), (pkg.DENSE_GATE_SIGMOID, y * no.sigmoid(gate))):
                out = torch.full((m, ldo), 7.0, dtype=tdt(act), device="cuda")
                ep = pkg.DenseEpilogue(kind, pkg.ptr(out), ldo, ap, an, pkg.ptr(gd), ldg)
                pkg.check(K.q38_dense_gemm(pkg.ptr(xd), ldx, act, m, C.byref(w.desc), C.byref(ep), None, None, i))
                got = out.double().cpu().numpy()
                assert np.all(got[:, n:] == 7.0)
                tol = 1e-3 + np.abs(want) / 200 if act == pkg.ACT_BF16 else 2e-5 * (1 + np.abs(want))
                assert np.all(np.abs(got[:, :n] - want) < tol), (name, kind)
    clean()


@pytest.mark.parametrize("groups,n,k,x_stride,out_stride", [(3, 64, 24, 24, 64), (5, 200, 64, 72, 203), (1, 40, 100, 0, 0), (20, 96, 16, 16, 96),
                                                            (2, 13, 300, 320, 20), (16, 128, 512, 512, 128)])
@pytest.mark.parametrize("m", [1, 5, 33, 140])
def test_grouped_products_every_kernel(groups, n, k, x_stride, out_stride, m):
    rng = np.random.default_rng(groups + n + m)
    K = pkg.kernels()
    ld, xs, os = up(k, 64), x_stride or k, out_stride or n
    wt = bf16(rng.standard_normal((groups, n, k)) / np.sqrt(k))
    wd = torch.zeros((up(groups * n, 16), ld), dtype=torch.bfloat16, device="cuda")
    wd[:groups * n, :k] = dev(wt.reshape(groups * n, k), torch.bfloat16)
    w = pkg.DenseWeight(pkg.ptr(wd), None, n, k, ld)
    g = pkg.DenseGroups(groups, x_stride, out_stride)
    ldx, ldo = up((groups - 1) * xs + k, 8), (groups - 1) * os + n + 2
    for act in ACTS:
        x, gate = rounded(rng.standard_normal((m, ldx)), act), rounded(rng.standard_normal((m, ldo)), act)
        xd, gd = dev(x, tdt(act)), dev(gate, tdt(act))
        for i, name in gemm_names() if act == pkg.ACT_BF16 else [(-1, "fp32")]:
            if "cluster" in name and (k + 63) // 64 < int(name[-1]):
                continue
            for kind in (pkg.DENSE_STORE, pkg.DENSE_GATE_SIGMOID, pkg.DENSE_STORE_F32):
                f32 = act == pkg.ACT_F32 or kind == pkg.DENSE_STORE_F32
                out = torch.full((m, ldo), 7.0, dtype=torch.float32 if f32 else torch.bfloat16, device="cuda")
                ep = pkg.DenseEpilogue(kind, pkg.ptr(out), ldo, 0, 0, pkg.ptr(gd), ldo)
                pkg.check(K.q38_dense_gemm_grouped(pkg.ptr(xd), ldx, act, m, C.byref(w), C.byref(g), C.byref(ep), None, None, i))
                want = np.full((m, ldo), 7.0)
                for q in range(groups):
                    y = x[:, q * xs:q * xs + k] @ wt[q].T
                    if kind == pkg.DENSE_GATE_SIGMOID:
                        y = y * no.sigmoid(gate[:, q * os:q * os + n])
                    want[:, q * os:q * os + n] = y
                got = out.double().cpu().numpy()
                assert np.all(np.abs(got - want) < 2e-4 + (0 if f32 else np.abs(want) / 250)), (name, kind)
    clean()


# ---- residual streams -------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("act", ACTS)
@pytest.mark.parametrize("m", [5, 200])
@pytest.mark.parametrize("width,groups,streams,stride", [(64, 4, 2, 1), (333, 9, 1, 1), (1000, 1, 3, 0), (30, 15, 16, 1), (96, 1, 4, 1),
                                                         (2560, 40, 2, 1), (4096, 2, 4, 1), (36, 18, 5, 1)])
def test_stream_kernels(width, groups, streams, stride, m, act):
    rng = np.random.default_rng(width + streams)
    K, eps, s = pkg.kernels(), 1e-3, streams
    tol = (0.01 if act == pkg.ACT_BF16 else 1e-5) * 4
    gains = [dev(rng.uniform(0.5, 2.0, width if stride else 1)) for _ in range(2)]
    norms = [pkg.Norm(pkg.ptr(g), stride, eps, groups) for g in gains]
    gn = [g.double().cpu().numpy() for g in gains]
    take, out_w, mix = [rng.standard_normal(n).astype(np.float32) for n in (s, s, (s, s))]
    take2 = rng.standard_normal(s).astype(np.float32)
    d = [dev(a) for a in (take, out_w, mix, take2)]
    table, tokens = bf16(rng.standard_normal((20, width))), rng.integers(0, 20, m)
    td, tok = dev(table, torch.bfloat16), dev(tokens, torch.int32)
    res = torch.full((m, s, width), float("nan"), device="cuda")
    ld = up(width + 7, 8)
    out = torch.zeros((m, ld), dtype=tdt(act), device="cuda")
    pkg.check(K.q38_stream_embed(pkg.ptr(td), pkg.ptr(tok), m, width, 1.5, s, pkg.ptr(res), pkg.ptr(d[0]), C.byref(norms[0]), pkg.ptr(out),
                                 ld, act, None))
    x = np.repeat((table[tokens] * 1.5)[None], s, axis=0)
    as_rows = lambda x: x.transpose(1, 0, 2)
    assert np.allclose(res.double().cpu().numpy(), as_rows(x), atol=1e-6)
    normed = lambda u, i: no.rms_norm(u, gn[i], eps, groups)
    got = lambda n=m: out[:n, :width].double().cpu().numpy()
    assert np.all(np.abs(got() - normed(np.einsum("s,sjw->jw", take, x), 0)) < tol * 2)
    y = rng.standard_normal((m, ld)).astype(np.float32)
    y[:, width:] = np.nan
    yd = dev(y)
    up_ = pkg.StreamUpdate(pkg.ptr(d[2]), pkg.ptr(d[1]), 0.4)
    for turn in range(3):
        last = turn == 2  # the last sublayer is followed by nothing
        pkg.check(K.q38_stream_norm(pkg.ptr(yd), ld, m, width, s, C.byref(up_), pkg.ptr(res), None if last else pkg.ptr(d[3]),
                                    None if last else C.byref(norms[1]), pkg.ptr(out), ld, act, None))
        x = no.hyper_update(x, y[:, :width].astype(np.float64), mix.astype(np.float64), out_w.astype(np.float64), 0.4)
        top = np.abs(x).max()
        assert np.abs(res.double().cpu().numpy() - as_rows(x)).max() < 1e-5 * max(1.0, top)
        if not last:
            want = normed(np.einsum("s,sjw->jw", take2, x), 1)
            assert np.all(np.abs(got() - want) < tol * (1 + np.abs(want)))
    assert np.all(out[:, width:].double().cpu().numpy() == 0)
    rows = np.array([4, 1, 1])
    rd = dev(rows, torch.int32)
    for r, first, pick in ((rd, 0, rows), (None, 2, np.array([2, 3, 4]))):
        pkg.check(K.q38_stream_gather(pkg.ptr(res), pkg.ptr(r), first, 3, width, s, C.byref(norms[1]), pkg.ptr(out), ld, act, None))
        want = normed(x.sum(0)[pick], 1)
        assert np.all(np.abs(got(3) - want) < tol * (1 + np.abs(want)))
    clean()


# ---- retention ------------------------------------------------------------------------------------------------------------------
class RetentionState:
    def __init__(self, floats, slots=4):
        self.floats, self.slot = floats, up(floats * 4, 256) + 256
        # leftovers of an earlier sequence: a fresh one must not see them
        self.mem = dev(np.random.default_rng(1).standard_normal(slots * self.slot // 4), torch.float32)
        self.desc = pkg.RecurrentStateDesc(self.mem.data_ptr(), self.mem.data_ptr(), self.slot)

    def of(self, slot, shape):
        at = slot * self.slot // 4
        return self.mem[at:at + self.floats].double().cpu().numpy().reshape(shape)


class Retention:
    """One layer's constants and scratch, as the kernels take them."""

    def __init__(self, H, dim, vdim, rot, base, decay, act, most, eps=1e-5):
        self.args = (H, dim, vdim, rot)
        self.act, self.eps, self.width, self.most = act, eps, 2 * H * (dim + vdim), most
        self.ld = up(self.width, 64)
        self.freq = dev(base ** (-2.0 * np.arange(max(1, rot // 2)) / max(1, rot)), torch.float64)
        self.pow = dev(np.array(decay)[:, None] ** np.arange(pkg.RETENTION_CHUNK + 1)[None])
        nbytes = pkg.kernels().q38_retention_qk_bytes(most, H, dim, act)
        self.qk = torch.full((max(1, nbytes // 2),), float("nan"), dtype=torch.bfloat16, device="cuda")
        self.o = torch.full((most, H * vdim), float("nan"), device="cuda")
        self.state = RetentionState(H * dim * vdim)

    def __call__(self, pd, out, ld_out, batch):
        H, dim, vdim, rot = self.args
        p = pkg.RetentionParams(pkg.ptr(pd), self.ld, self.act, H, dim, vdim, rot, pkg.ptr(self.freq), pkg.ptr(self.pow), dim ** -0.5,
                                self.eps, pkg.ptr(self.qk), pkg.ptr(self.o), pkg.ptr(out), ld_out)
        pkg.check(pkg.kernels().q38_retention(C.byref(p), C.byref(batch), C.byref(self.state.desc), None))


def retention_reference(proj, H, dim, vdim, rot, base, decay, eps):
    n = len(proj)
    q, k, v, g = np.split(proj, [H * dim, 2 * H * dim, 2 * H * dim + H * vdim], axis=1)
    q, k = q.reshape(n, H, dim), k.reshape(n, H, dim)
    if rot:
        q, k = no.rope(q, np.arange(n), rot, base), no.rope(k, np.arange(n), rot, base)
    o, S = no.retention(q, k * dim ** -0.5, v.reshape(n, H, vdim), decay)
    return no.rms_norm(o, 1.0, eps).reshape(n, -1) * no.silu(g), S


RETENTIONS = [(3, 40, 24, 16), (1, 136, 20, 0), (2, 9, 33, 6), (4, 64, 96, 64), (2, 128, 256, 128), (1, 256, 72, 32), (2, 16, 8, 4),
              (1, 300, 36, 20), (5, 32, 32, 30)]


@pytest.mark.parametrize("act", ACTS)
@pytest.mark.parametrize("shape", RETENTIONS)
def test_retention_against_the_plain_one(shape, act):
    """Two sequences in uneven portions (down to two tokens, around the edges of a chunk, single tokens) over slots that were
    used before; keys that stand out far back, at chunk edges and one before the query, under slow and fast decays."""
    H, dim, vdim, rot = shape
    rng = np.random.default_rng(sum(shape))
    decay = [0.9995, 0.97, 1.0, 0.5, 0.9][:H]
    lens, base = (420, 150), 700.0
    op = Retention(H, dim, vdim, rot, base, decay, act, sum(lens))
    proj = rng.standard_normal((sum(lens), op.width))
    for lo, n in ((0, 420), (420, 150)):
        for i, j in ((n - 1, 0), (n - 1, 63), (n - 2, 64), (70, 3), (64, 63), (65, 64), (n - 5, n - 6), (128, 127), (20, 20)):
            h = (i + j) % H
            proj[lo + j, (H + h) * dim:(H + h + 1) * dim] = 4.0 * proj[lo + i, h * dim:(h + 1) * dim]
    proj = rounded(proj, act)
    done, outs = [0, 0], [np.zeros((n, H * vdim)) for n in lens]
    portions = [[(0, 2), (1, 64)], [(0, 3), (1, 1)], [(0, 300), (1, 2)], [(1, 40), (0, 1)], [(0, 1), (1, 1)], [(0, 63)], [(0, 1)],
                [(0, 49), (1, 42)]]
    ld_out = H * vdim + 5
    for step in portions:
        b = Batch([(s + 1, done[s], n) for s, n in step])
        src = np.concatenate([np.arange(done[s], done[s] + n) + (0 if s == 0 else lens[0]) for s, n in step])
        pd = torch.zeros((b.m, op.ld), dtype=tdt(act), device="cuda")
        pd[:, :op.width] = dev(proj[src], tdt(act))
        out = torch.zeros((b.m, ld_out), dtype=tdt(act), device="cuda")
        multi = sum(n > 1 for _, n in step)
        for a, z in ((multi, len(step)), (0, multi)):
            if a < z:
                op(pd, out, ld_out, b.part(a, z))
        torch.cuda.synchronize()
        got, at = out.double().cpu().numpy(), 0
        assert np.all(got[:, H * vdim:] == 0)
        for s, n in step:
            outs[s][done[s]:done[s] + n] = got[at:at + n, :H * vdim]
            done[s], at = done[s] + n, at + n
    assert done == list(lens)
    clean()
    lo = 0
    for s, n in enumerate(lens):
        want, S = retention_reference(proj[lo:lo + n], H, dim, vdim, rot, base, decay, op.eps)
        # fp32 up to the stored output: what is left is the output's own rounding, and cancellation in small outputs
        tol = 2e-3 + np.abs(want) / 200 if act == pkg.ACT_BF16 else 2e-4 + np.abs(want) * 1e-5
        assert np.all(np.abs(outs[s] - want) < tol), np.abs(outs[s] - want).max()
        state = op.state.of(s + 1, S.shape)
        assert np.abs(state - S).max() < (1e-4 if act == pkg.ACT_BF16 else 1e-5) * np.abs(S).max()
        lo += n


@pytest.mark.parametrize("act", ACTS)
def test_retention_outputs_do_not_depend_on_the_cut(act):
    """One run against every way of cutting it in two around the chunk edges, and against single tokens."""
    H, dim, vdim, rot, n = 2, 32, 64, 32, 140
    op = Retention(H, dim, vdim, rot, 1e4, [0.999, 0.8], act, n)
    rng = np.random.default_rng(3)
    proj = torch.zeros((n, op.ld), dtype=tdt(act), device="cuda")
    proj[:, :op.width] = dev(rng.standard_normal((n, op.width)), tdt(act))

    def run(cuts):
        out = torch.zeros((n, H * vdim), dtype=tdt(act), device="cuda")
        for a, z in zip((0,) + cuts, cuts + (n,)):
            part = out[a:z].clone()
            op(proj[a:z].contiguous(), part, H * vdim, Batch([(2, a, z - a)]).desc)
            out[a:z] = part
        torch.cuda.synchronize()
        return out.double().cpu().numpy(), op.state.of(2, (H * dim, vdim)).copy()
    whole, S = run(())
    for cuts in [(1,), (2,), (62,), (63,), (64,), (65,), (128,), (138,), (139,), (60, 62, 64, 66), tuple(range(1, n))]:
        got, S2 = run(cuts)
        assert np.abs(got - whole).max() < (2e-2 if act == pkg.ACT_BF16 else 1e-4), cuts
        assert np.abs(S2 - S).max() < 1e-4 * np.abs(S).max()
    clean()


# ---- latent attention --------------------------------------------------------------------------------------------------------------
class LatentCache:
    def __init__(self, rank, slots, max_pages, act, seed=0):
        self.kd = up(rank, 32)
        pages = slots * max_pages + 3
        rng = np.random.default_rng(seed)
        # pages that were used before: finite leftovers everywhere
        self.pool = dev(rng.standard_normal((pages, 64 * self.kd)) * 3, tdt(act))
        self.table = dev(rng.permutation(pages)[:slots * max_pages].reshape(slots, max_pages), torch.int32)
        self.desc = pkg.KvLayerDesc(pkg.ptr(self.pool), pkg.KV_BF16 if act == pkg.ACT_BF16 else pkg.KV_F32, 1, self.kd, 0, pages,
                                    64 * self.kd * self.pool.element_size(), pkg.ptr(self.table), max_pages)


# heads, latent size
LATENTS = [(3, 44), (20, 128), (1, 24), (16, 512), (40, 96), (6, 300), (70, 256), (33, 512), (5, 600)]


@pytest.mark.parametrize("act", ACTS)
@pytest.mark.parametrize("heads,rank", LATENTS)
def test_latent_attention_against_the_plain_one(heads, rank, act):
    """Prompts in portions, then decoded tokens, through one shuffled cache; latents that stand out far away, at a page's first
    and last token, at the row itself and just behind the causal limit; with and without scratch for divided key ranges."""
    rng = np.random.default_rng(heads + rank)
    K, q_rank, eps, scale, H = pkg.kernels(), 36, 1e-4, 0.7 / np.sqrt(rank), heads
    lens, slots = [150, 77], (1, 3)
    cache = LatentCache(rank, 4, 3, act)
    width = q_rank + rank + 5
    proj, q = rng.standard_normal((sum(lens), width)), rng.standard_normal((sum(lens), H, rank))
    qg, cg = rng.uniform(0.5, 1.5, q_rank).astype(np.float32), rng.uniform(0.5, 1.5, rank).astype(np.float32)
    proj = rounded(proj, act)
    latent = rounded(no.rms_norm(proj[:, q_rank:q_rank + rank], cg.astype(np.float64), eps), act)
    for lo, n in ((0, 150), (150, 77)):
        for i, j in ((n - 1, 0), (n - 1, 63), (n - 2, 64), (70, 3), (64, 63), (65, 66), (n - 5, n - 4), (20, 20)):
            q[lo + i, (i + j) % H] = 1.5 * latent[lo + j]
    q = rounded(q, act)
    gd, cd = dev(qg), dev(cg)
    partials = torch.full((K.q38_latent_attention_partial_floats(cache.kd),), float("nan"), device="cuda")
    for scratch in (True, False):
        done, outs = [0, 0], [np.zeros((n, H, rank)) for n in lens]
        schedule = [[(0, 64), (1, 2)], [(1, 30), (0, 63)], [(0, 2), (1, 44)], [(0, 19), (1, 1)], [(0, 1)], [(0, 1)]]
        for step in schedule:
            b = Batch([(slots[s], done[s], n) for s, n in step])
            src = np.concatenate([np.arange(done[s], done[s] + n) + (0 if s == 0 else 150) for s, n in step])
            pd = dev(proj[src], tdt(act))
            cq = torch.zeros((b.m, q_rank + 4), dtype=tdt(act), device="cuda")
            lp = pkg.LatentAppendParams(pkg.ptr(pd), width, act, q_rank, rank, pkg.ptr(gd), pkg.ptr(cd), eps, pkg.ptr(cq), q_rank + 4)
            pkg.check(K.q38_latent_append(C.byref(lp), C.byref(b.desc), C.byref(cache.desc), None))
            want = no.rms_norm(proj[src][:, :q_rank], qg.astype(np.float64), eps)
            got = cq.double().cpu().numpy()
            assert np.all(np.abs(got[:, :q_rank] - want) < 1e-5 + (np.abs(want) / 250 if act == pkg.ACT_BF16 else 0)) and np.all(got[:, q_rank:] == 0)
            qd = torch.zeros((b.m, H, cache.kd), dtype=tdt(act), device="cuda")
            qd[:, :, :rank] = dev(q[src], tdt(act))
            out = torch.zeros((b.m, H, cache.kd), dtype=tdt(act), device="cuda")
            ap = pkg.LatentAttentionParams(pkg.ptr(qd), act, H, scale, pkg.ptr(out), pkg.ptr(partials) if scratch else None,
                                           partials.numel() if scratch else 0)
            multi = sum(n > 1 for _, n in step)
            for a, z in ((0, multi), (multi, len(step))):
                if a < z:
                    part = b.part(a, z)
                    pkg.check(K.q38_latent_attention(C.byref(ap), C.byref(part), C.byref(cache.desc), None))
            torch.cuda.synchronize()
            got, at = out.double().cpu().numpy(), 0
            assert np.all(got[:, :, rank:] == 0)
            for s, n in step:
                outs[s][done[s]:done[s] + n] = got[at:at + n, :, :rank]
                done[s], at = done[s] + n, at + n
        assert done == lens
        clean()
        for s, (lo, n) in enumerate(((0, 150), (150, 77))):
            c = np.repeat(latent[lo:lo + n, None], H, 1)
            want = no.softmax_attention(q[lo:lo + n], c, c, scale)
            err = np.abs(outs[s] - want).max() / np.abs(want).max()
            # the cached latents are rounded as stored, the sums are fp32: what is left is the output's rounding, and a latent
            # that a difference in the norm's last bit rounds the other way
            assert err < (8e-3 if act == pkg.ACT_BF16 else 1e-5), (s, err)


@pytest.mark.parametrize("heads,dim,vdim,rank", [(3, 20, 24, 44), (2, 128, 128, 96), (1, 72, 200, 64), (5, 16, 7, 32), (2, 192, 64, 160), (1, 256, 33, 24)])
def test_packed_attention_against_the_plain_one(heads, dim, vdim, rank):
    """Latents of two sequences gathered from shuffled pages, keys and values that stand out at tile borders and far back; a
    run that starts in the middle of a page, one of two tokens, and an output gate."""
    H = heads
    rng = np.random.default_rng(heads + dim)
    K, act = pkg.kernels(), pkg.ACT_BF16
    cache = LatentCache(rank, 4, 4, act)
    rows = [(2, 0, 200), (1, 63, 2), (3, 130, 90)]
    contexts = [200, 65, 220]
    packed = sum(up(c, 64) for c in contexts)
    b = Batch(rows)
    lat = torch.full((packed, cache.kd), float("nan"), dtype=torch.bfloat16, device="cuda")
    pkg.check(K.q38_latent_gather(C.byref(b.desc), C.byref(cache.desc), max(contexts), packed, pkg.ptr(lat), None))
    got, at = lat.double().cpu().numpy(), 0
    pool, table = cache.pool.double().cpu().numpy().reshape(-1, 64, cache.kd), cache.table.cpu().numpy()
    for (slot, _, _), c in zip(rows, contexts):
        want = np.concatenate([pool[p] for p in table[slot][:up(c, 64) // 64]])
        want[c:] = 0
        assert np.array_equal(got[at:at + len(want)], want)
        at += len(want)
    ks, vs = up(dim, 16), up(vdim, 16)
    q, k, v = [rounded(rng.standard_normal(s), act) for s in ((b.m, H, dim), (packed, H, dim), (packed, H, vdim))]
    gate = rounded(rng.standard_normal((b.m, H * vdim)) * 2, act)
    base, first = [0, 256, 384], [0, 200, 202]
    for i, j in ((199, 0), (199, 63), (198, 64), (70, 3), (64, 63), (65, 66), (130, 127), (20, 20)):
        q[i, (i + j) % H] = 2.0 * k[j, (i + j) % H]
    q[201] = k[256]
    q[202 + 89] = k[384 + 5]
    q = rounded(q, act)
    ld_kv, ld_q = H * (ks + vs) + 8, H * ks + 16
    qd, kvd = torch.zeros((b.m, ld_q), dtype=torch.bfloat16, device="cuda"), torch.zeros((packed, ld_kv), dtype=torch.bfloat16, device="cuda")
    for h in range(H):
        qd[:, h * ks:h * ks + dim] = dev(q[:, h], torch.bfloat16)
        kvd[:, h * ks:h * ks + dim] = dev(k[:, h], torch.bfloat16)
        kvd[:, H * ks + h * vs:H * ks + h * vs + vdim] = dev(v[:, h], torch.bfloat16)
    # gates that start at an odd column of their matrix too
    for gated, ld_out, shift in ((True, H * vdim + 2, 0), (True, H * vdim + 2, 1), (False, H * vdim + 3, 0)):
        gd = torch.zeros((b.m, H * vdim + 4), dtype=torch.bfloat16, device="cuda")
        gd[:, shift:shift + H * vdim] = dev(gate, torch.bfloat16)
        out = torch.zeros((b.m, ld_out), dtype=torch.bfloat16, device="cuda")
        p = pkg.PackedAttentionParams(pkg.ptr(qd), ld_q, ks, pkg.ptr(kvd), kvd.data_ptr() + 2 * H * ks, ld_kv, ks, vs, H, dim, vdim, 0.4,
                                      gd.data_ptr() + 2 * shift if gated else None, H * vdim + 4, pkg.ptr(out), ld_out)
        pkg.check(K.q38_packed_attention(C.byref(p), C.byref(b.desc), None))
        torch.cuda.synchronize()
        got = out.double().cpu().numpy()
        assert np.all(got[:, H * vdim:] == 0)
        for (slot, pos0, n), c, k0, m0 in zip(rows, contexts, base, first):
            full = np.zeros((c, H, dim))
            full[pos0:] = q[m0:m0 + n]
            want = no.softmax_attention(full, k[k0:k0 + c], v[k0:k0 + c], 0.4)[pos0:].reshape(n, -1)
            if gated:
                want = want * no.sigmoid(gate[m0:m0 + n])
            assert np.all(np.abs(got[m0:m0 + n, :H * vdim] - want) < 2e-3 + np.abs(want) / 200)
    clean()


@pytest.mark.parametrize("act", ACTS)
@pytest.mark.parametrize("heads", [4, 24])
def test_long_decoding_over_many_pages_with_and_without_divided_ranges(heads, act):
    H, rank, n = heads, 64, 1500
    rng = np.random.default_rng(7)
    K = pkg.kernels()
    cache = LatentCache(rank, 1, 24, act)
    c = rounded(rng.standard_normal((n, rank)), act)
    q = rounded(rng.standard_normal((3, H, rank)), act)
    q[0, 1] = c[5]       # far latents that one query must find, alone at the end of a page, and the newest one
    q[1, 2] = c[1023]
    q[2, 3] = c[n - 1]
    table = cache.table.cpu().numpy()[0]
    pool = cache.pool.view(-1, 64, rank)
    for j0 in range(0, n, 64):
        pool[int(table[j0 // 64]), :min(64, n - j0)] = dev(c[j0:j0 + 64], tdt(act))
    outs = []
    for floats in (0, 3 * 64 * (rank + 2) * 4, K.q38_latent_attention_partial_floats(rank)):
        partials = torch.full((max(1, floats),), float("nan"), device="cuda")
        got = []
        for i, pos in enumerate((n - 3, n - 2, n - 1)):
            qd, out = dev(q[i], tdt(act)), torch.zeros((H, rank), dtype=tdt(act), device="cuda")
            ap = pkg.LatentAttentionParams(pkg.ptr(qd), act, H, 0.5, pkg.ptr(out), pkg.ptr(partials) if floats else None, floats)
            b = Batch([(0, pos, 1)])
            pkg.check(K.q38_latent_attention(C.byref(ap), C.byref(b.desc), C.byref(cache.desc), None))
            torch.cuda.synchronize()
            got.append(out.double().cpu().numpy())
        outs.append(np.array(got))
    for i, pos in enumerate((n - 3, n - 2, n - 1)):
        s = np.einsum("hd,jd->hj", q[i], c[:pos + 1]) * 0.5
        w = np.exp(s - s.max(1, keepdims=True))
        want = (w / w.sum(1, keepdims=True)) @ c[:pos + 1]
        for o in outs:
            assert np.abs(o[i] - want).max() < (8e-3 if act == pkg.ACT_BF16 else 1e-5) * np.abs(want).max()
    clean()


def test_bad_arguments_are_refused():
    K = pkg.kernels()
    x = torch.zeros((4, 512), dtype=torch.bfloat16, device="cuda")
    f = torch.zeros(4096, device="cuda")
    b = Batch([(0, 0, 2)])
    w = DenseWeight(np.zeros((16, 64)))
    ep = pkg.DenseEpilogue(pkg.DENSE_GATE_SIGMOID, pkg.ptr(x), 64)
    assert K.q38_dense_gemm(pkg.ptr(x), 64, 0, 4, C.byref(w.desc), C.byref(ep), None, None, -1) == -1
    assert b"gate" in K.q38_last_error()
    ep = pkg.DenseEpilogue(pkg.DENSE_STORE, pkg.ptr(x), 512)
    g = pkg.DenseGroups(3, 32, 16)
    assert K.q38_dense_gemm_grouped(pkg.ptr(x), 512, 0, 4, C.byref(w.desc), C.byref(g), C.byref(ep), None, None, -1) == -1
    assert b"3 groups" in K.q38_last_error()
    norm = pkg.Norm(pkg.ptr(f), 1, 1e-5, 7)
    up_ = pkg.StreamUpdate(pkg.ptr(f), pkg.ptr(f), 1.0)
    assert K.q38_stream_norm(pkg.ptr(f), 64, 2, 64, 2, C.byref(up_), pkg.ptr(f), pkg.ptr(f), C.byref(norm), pkg.ptr(x), 64, 0, None) == -1
    assert b"7 parts of a row of 64" in K.q38_last_error()
    assert K.q38_stream_norm(pkg.ptr(f), 64, 2, 64, 17, C.byref(up_), pkg.ptr(f), None, None, None, 0, 0, None) == -1
    assert b"17" in K.q38_last_error()
    st = RetentionState(64)
    p = pkg.RetentionParams(pkg.ptr(x), 32, 0, 1, 8, 8, 10, pkg.ptr(f), pkg.ptr(f), 1.0, 1e-5, pkg.ptr(x), pkg.ptr(f), pkg.ptr(x), 64)
    assert K.q38_retention(C.byref(p), C.byref(b.desc), C.byref(st.desc), None) == -1
    assert b"rot_dims 10" in K.q38_last_error()
    cache = LatentCache(32, 1, 1, pkg.ACT_F32)
    ap = pkg.LatentAttentionParams(pkg.ptr(x), pkg.ACT_BF16, 2, 1.0, pkg.ptr(x), None, 0)
    assert K.q38_latent_attention(C.byref(ap), C.byref(b.desc), C.byref(cache.desc), None) == -1
    assert b"cache precision" in K.q38_last_error()
