"""Nololix models through the framework's own runner and scheduler, against the plain oracle."""

import json
import subprocess
import sys

import numpy as np
import pytest

import layer_list_testlib as ll
import nololix_oracle as no
import nololix_testlib as nl
import q38_testlib as tl
from q38b200 import engine as eng
from test_layer_list_gpu import DTYPES, TOL, decode_logits, enter, error

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root, cache = tmp_path_factory.mktemp("models"), {}

    def get(name):
        if name not in cache:
            folder, oracle = nl.make_model(root / name, nl.CONFIGS[name], seed=len(name))
            tokens = np.random.default_rng(3).integers(0, oracle.cfg["vocab"], 250)
            cache[name] = (folder, eng.Model(folder), oracle, tokens, oracle.logits(tokens))
        return cache[name]
    yield get
    for c in cache.values():
        c[1].close()


def runner_of(model, dtype, **kw):
    o = dict(max_batch=4, prefill_chunk=256, kv_tokens=4096, max_context=1024, verbose=0, compute_dtype=dtype)
    o.update(kw)
    return eng.Runner(model, eng.default_runner_options(**o))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(nl.CONFIGS))
def test_prompt_portions_and_decoding_match_the_oracle(models, name, dtype):
    _, model, oracle, tokens, want = models(name)
    n = len(tokens)
    r = runner_of(model, dtype)
    enter(r, 0, n)
    whole = r.prefill_logits(0, 0, tokens)
    assert error(whole, want) < TOL[dtype]
    # portions of several sizes in a slot that was just used, then token by token to the end
    for sizes in ([2, 3, 2, 64, 63, 65], [1, 130, 2, 2], [17] * 8, [2] * 70):
        r.kv_release(0)
        enter(r, 0, n)
        at, got = 0, []
        for s in sizes:
            got.append(r.step_logits([(0, at, tokens[at:at + s], None, 0)], [(0, i) for i in range(s)]))
            at += s
        for p in range(at, n):
            got.append(decode_logits(r, [(0, p, tokens[p])]))
        got = np.concatenate(got)
        assert error(got, want) < TOL[dtype]
        assert error(got, whole) < TOL[dtype]
    r.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "latent"])
def test_token_by_token_from_the_start_equals_the_prompt(models, name, dtype):
    _, model, oracle, tokens, want = models(name)
    r = runner_of(model, dtype)
    enter(r, 2, 140)
    got = np.concatenate([decode_logits(r, [(2, p, tokens[p])]) for p in range(140)])
    assert error(got, want[:140]) < TOL[dtype]
    r.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_unequal_requests_in_one_batch_match_each_alone(models, name, dtype):
    _, model, oracle, _, _ = models(name)
    rng = np.random.default_rng(11)
    seqs = [rng.integers(0, model.vocab, n) for n in (130, 2, 67, 200)]
    wants = [oracle.logits(s) for s in seqs]
    r = runner_of(model, dtype)
    for s in range(4):
        enter(r, s, len(seqs[s]))
    done = [0] * 4
    got = [[] for _ in range(4)]
    # ragged steps that mix chunks, two-token portions and single tokens (slots in changing order)
    for step in ([(3, 100), (0, 64), (1, 1)], [(2, 2), (3, 1), (0, 2)], [(0, 1), (1, 1), (2, 1), (3, 1)],
                 [(2, 63), (0, 1), (3, 90)], [(0, 62), (2, 1), (3, 1)]):
        rows = [(s, done[s], seqs[s][done[s]:done[s] + n], None, 0) for s, n in step]
        out = r.step_logits(rows, [(i, k) for i, (_, n) in enumerate(step) for k in range(n)])
        at = 0
        for s, n in step:
            got[s].append(out[at:at + n])
            done[s] += n
            at += n
    assert done == [130, 2, 67, 193]
    for p in range(7):  # the rest of the longest one, decoded beside nothing
        got[3].append(decode_logits(r, [(3, done[3] + p, seqs[3][done[3] + p])]))
    for s in range(4):
        assert error(np.concatenate(got[s]), wants[s]) < TOL[dtype], s
    r.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_batched_decode_matches_each_alone(models, dtype):
    _, model, oracle, _, _ = models("mixed")
    rng = np.random.default_rng(12)
    seqs = [rng.integers(0, model.vocab, n) for n in (90, 61, 127)]
    wants = [oracle.logits(s) for s in seqs]
    r = runner_of(model, dtype)
    starts = [len(s) - 30 for s in seqs]
    slots = [3, 0, 2]
    for i, s in enumerate(seqs):
        enter(r, slots[i], len(s))
        r.prefill([(slots[i], 0, s[:starts[i]], None, 0)])
    for k in range(30):  # crosses page borders of all three at different steps; padding rows ride in the graph
        order = np.roll(np.arange(3), k)
        got = decode_logits(r, [(slots[i], starts[i] + k, seqs[i][starts[i] + k]) for i in order])
        for row, i in enumerate(order):
            assert error(got[row:row + 1], wants[i][starts[i] + k:starts[i] + k + 1]) < 2 * TOL[dtype]
    r.close()


def test_pages_and_slots_are_freed_and_used_again(models):
    _, model, oracle, tokens, want = models("mixed")
    r = runner_of(model, eng.COMPUTE_F32, max_batch=2, kv_tokens=512)
    free = r.kv_free_pages()
    rng = np.random.default_rng(2)
    for turn in range(6):  # a long sequence leaves its pages and states to a short one and back, in changing slots
        slot = turn % 2
        enter(r, slot, 200)
        r.prefill([(slot, 0, rng.integers(0, model.vocab, 200), None, 0)])
        r.kv_release(slot)
        n = (64, 65, 63, 128, 2, 40)[turn]
        for other in (1 - slot, slot):
            enter(r, other, n)
            assert error(r.prefill_logits(other, 0, tokens[:n]), want[:n]) < 1e-4
            r.kv_release(other)
        assert r.kv_free_pages() == free
    r.close()


def marked_model(kind):
    """One layer whose first head finds the one token whose key matches the last token's query, however far back. Queries
    read one part of the embedding, keys another one."""
    W, V, key, query = 64, 60, 7, 11
    rng = np.random.default_rng(4)
    layer = nl.retention(2, 32, 16, (1.0, 0.9), 8) if kind == "retention" else nl.latent(2, 24, 16, 32, 64, scale=1.0)
    cfg = nl.config(W, V, [layer], streams=2, scale=2.0, mult=2.5)
    t = nl.random_tensors(cfg, 9)
    emb = rng.standard_normal((V, W)) * 0.3
    mark = rng.choice([-1.0, 1.0], 24)
    emb[:, :48] = 0.05 * rng.standard_normal((V, 48))
    emb[key, 24:48] = mark
    emb[query, :24] = mark
    emb[:, 48:] = rng.standard_normal((V, 16))
    t["embed"], t["l0.norm1"] = emb, np.ones(W)
    if kind == "retention":  # the rotated dimensions stay silent
        q, k = np.zeros((64, W)), np.zeros((64, W))
        q[8:32, :24] = k[8:32, 24:48] = np.eye(24) * 3.0
        t.update({"l0.mix.q": q, "l0.mix.k": k, "l0.mix.v": t["l0.mix.v"] * 0.2})
    else:
        dq, dkv, uq, uk, uv = (np.zeros(t["l0.mix." + n].shape) for n in ("dq", "dkv", "uq", "uk", "uv"))
        dq[:24, :24], dq[24:, 48:56] = np.eye(24), np.eye(8)
        dkv[:24, 24:48], dkv[24:40, 48:] = np.eye(24), np.eye(16)
        uq[:24, :24], uk[:24, :24] = np.eye(24) * 2.0, np.eye(24) * 2.0
        uv[:16, 24:40] = uv[16:, 24:40] = np.eye(16)
        uv[:16, :16] = np.eye(16)
        t.update({"l0.mix.dq": dq, "l0.mix.dkv": dkv, "l0.mix.uq": uq, "l0.mix.uk": uk, "l0.mix.uv": uv})
        for n in ("dq.norm", "dkv.norm"):
            t["l0.mix." + n] = np.ones_like(t["l0.mix." + n])
    return cfg, {n: ll.bf16_round(v) for n, v in t.items()}, key, query


@pytest.mark.parametrize("kind", ["retention", "latent"])
def test_a_far_key_decides_the_answer_at_every_distance(tmp_path, kind):
    """The marked token stands at the first positions, around page, chunk and portion borders and one before the query, in a
    prompt, in portions and decoded."""
    cfg, t, key, query = marked_model(kind)
    model, oracle = eng.Model(ll.write_model(tmp_path / "far", cfg, t)), no.Model(cfg, t)
    n = 600
    plain = np.random.default_rng(1).integers(12, cfg["vocab"], n)
    plain[-1] = query
    absent = oracle.logits(plain)[-1]
    places = (0, 1, 63, 64, 127, 128, 319, 320, 575, 576, n - 2)
    wants = {}
    for at in places:
        tokens = plain.copy()
        tokens[at] = key
        wants[at] = (tokens, oracle.logits(tokens)[-1])
        assert error(absent[None], wants[at][1][None]) > 0.15, at  # the key matters
    for dtype in DTYPES:
        r = runner_of(model, dtype, prefill_chunk=640)
        for at, (tokens, want) in wants.items():
            enter(r, 0, n)
            got = r.step_logits([(0, 0, tokens, None, 0)], [(0, n - 1)])
            assert error(got, want[None]) < TOL[dtype], at
            enter(r, 1, n)
            r.prefill([(1, 0, tokens[:n - 1], None, 0)])
            assert error(decode_logits(r, [(1, n - 1, query)]), want[None]) < TOL[dtype], at
            enter(r, 2, n)
            for lo, hi in ((0, 2), (2, 64), (64, 320), (320, 576), (576, n - 2)):
                r.prefill([(2, lo, tokens[lo:hi], None, 0)])
            assert error(r.step_logits([(2, n - 2, tokens[n - 2:], None, 0)], [(0, 1)]), want[None]) < TOL[dtype], at
            for s in range(3):
                r.kv_release(s)
        r.close()
    model.close()


def test_long_decoding(models):
    _, model, oracle, _, _ = models("mixed")
    n = 420
    tokens = np.random.default_rng(8).integers(0, model.vocab, n)
    want = oracle.logits(tokens)
    for dtype in DTYPES:
        r = runner_of(model, dtype)
        enter(r, 0, n)
        r.prefill([(0, 0, tokens[:3], None, 0)])
        got = np.concatenate([decode_logits(r, [(0, p, tokens[p])]) for p in range(3, n)])
        assert error(got, want[3:]) < TOL[dtype]
        r.close()


def test_first_tokens(models):
    for name in sorted(nl.CONFIGS):
        _, model, oracle, tokens, want = models(name)
        r = runner_of(model, eng.COMPUTE_F32)
        for n in (1, 2, 3, 5):
            enter(r, 0, n)
            assert error(r.prefill_logits(0, 0, tokens[:n]), want[:n]) < 1e-4
            r.kv_release(0)
        enter(r, 0, 1)
        assert error(decode_logits(r, [(0, 0, tokens[0])]), want[:1]) < 1e-4
        r.close()


def test_without_optional_entries(tmp_path):
    """No loop, one stream without hyper-connections, scale and factor 1: left out of the configuration altogether."""
    cfg = nl.config(48, 50, [nl.retention(2, 8, 8, (0.9, 0.99), 4, ff=20), nl.latent(2, 8, 8, 8, 8)])
    t = nl.random_tensors(cfg, 2)
    for k in [k for k in t if ".hc" in k]:
        t[k] = np.ones_like(t[k])
    oracle = no.Model(cfg, t)
    tokens = np.random.default_rng(1).integers(0, 50, 90)
    short = {k: v for k, v in cfg.items() if k not in ("loop", "streams", "embedding", "residual_mult")}
    model = eng.Model(ll.write_model(tmp_path / "m", short, {k: v for k, v in t.items() if ".hc" not in k}))
    for dtype in DTYPES:
        r = runner_of(model, dtype)
        enter(r, 0, 90)
        assert error(r.prefill_logits(0, 0, tokens), oracle.logits(tokens)) < TOL[dtype]
        r.close()
    model.close()


@pytest.mark.parametrize("ragged,mixed", [(False, False), (True, False), (True, True)])
def test_greedy_generation_through_the_scheduler(models, ragged, mixed):
    """More requests than slots, 32-bit: every sequence is the oracle's own greedy continuation."""
    _, model, oracle, _, _ = models("mixed")
    rng = np.random.default_rng(21)
    prompts = [rng.integers(0, model.vocab, n) for n in (70, 1, 33, 2, 129, 64)]
    e = eng.Engine(model, eng.default_runner_options(max_batch=3, prefill_chunk=64, kv_tokens=1024, max_context=400, verbose=0,
                                                     compute_dtype=eng.COMPUTE_F32), ragged_prefill=ragged, mixed_steps=mixed)
    ids = [e.submit(p, eng.greedy(), 12, ignore_eos=True) for p in prompts]
    e.run()
    done = {f.id: f for f in e.take_finished()}
    for i, p in zip(ids, prompts):
        f = done[i]
        assert f.finish == "length" and len(f.tokens) == 12
        logits = oracle.logits(np.concatenate([p, f.tokens[:-1]]))[len(p) - 1:]
        for row, tok in zip(logits, f.tokens):  # the oracle's choice, or a tie within rounding
            assert row[tok] > row.max() - 1e-3
    assert e.stats().requests_done == len(prompts)
    e.close()


def test_bf16_generation_sampling_and_scores(models):
    _, model, oracle, tokens, want = models("wide")
    e = eng.Engine(model, eng.default_runner_options(max_batch=2, prefill_chunk=128, verbose=0, max_context=300), ragged_prefill=True,
                   mixed_steps=True)
    a = [e.submit(tokens[:40], eng.Sampling(0.8, 10, 0.9, 0.0, 0.0, 1.0, 77), 20, ignore_eos=True) for _ in range(2)]
    g = e.submit(tokens[:90], eng.greedy(), 8, ignore_eos=True)
    limit = e.submit(tokens[:50], eng.greedy(), 10000, ignore_eos=True)  # runs to the end of the context
    e.run()
    out = {f.id: f for f in e.take_finished()}
    assert np.array_equal(out[a[0]].tokens, out[a[1]].tokens)  # same seed, same draws, whatever the batch
    row = want[89]
    assert row[out[g].tokens[0]] > row.max() - 0.1 * np.sqrt(np.mean(want ** 2))
    assert out[limit].finish == "length" and len(out[limit].tokens) == 300 - 50 + 1
    r = e.runner
    enter(r, 0, 101)
    scores = r.score(0, 0, tokens[:100], tokens[1:101])
    top = want[:100].max(1, keepdims=True)
    ref = want[:100] - np.log(np.exp(want[:100] - top).sum(1, keepdims=True)) - top
    assert np.abs(scores - ref[np.arange(100), tokens[1:101]]).max() < 0.25
    e.close()


def test_trace_replay_program(models, tmp_path):
    """The command-line replay: several live requests, portions, single tokens, a name that comes back after its end."""
    folder, model, oracle, tokens, want = models("mixed")
    t = [int(x) for x in tokens]
    steps = [
        {"step": 0, "entries": [{"id": "a", "tokens": t[:50], "want": [0, 49]}], "end": []},
        {"step": 1, "entries": [{"id": "a", "tokens": t[50:51], "want": [0]}, {"id": "b", "tokens": t[:3], "want": [2]}], "end": []},
        {"step": 2, "entries": [{"id": "b", "tokens": t[3:4], "want": []}], "end": ["a"]},
        {"step": 3, "entries": [{"id": "a", "tokens": t[:1], "want": [0]}, {"id": "b", "tokens": t[4:5], "want": [0]}], "end": ["a", "b"]},
        {"step": 4, "entries": [{"id": "c", "tokens": t[:119], "want": [118]}], "end": ["c"]},
    ]
    places = {0: [0, 49], 1: [50, 2], 3: [0, 4], 4: [118]}
    for dtype, tol in (("float32", 1e-4), ("bfloat16", 2.5e-2)):
        out = tmp_path / dtype
        out.mkdir()
        p = subprocess.run([sys.executable, str(tl.ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out),
                            "--max-tokens", "120"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True,
                           timeout=600)
        assert p.returncode == 0, p.stderr[-2000:]
        assert [x for x in p.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(5)]
        for s, at in places.items():
            got = np.fromfile(out / f"{s}.f32", np.float32).reshape(len(at), -1)
            assert error(got, want[at]) < tol
