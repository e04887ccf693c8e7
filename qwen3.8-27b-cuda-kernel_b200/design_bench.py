"""Throughput of the layer-list designs (Fegenex, Nololix) beside each other and the Qwen3.8 hybrid at equal size.

    python bench.py --designs small,medium [--design-models nololix,qwen38]

All models get the same width, feed-forward, vocabulary, number of layers (two attention layers in six) and attention
width; weights are random, the Qwen3.8 planes in the default recipe. The closest model of Nololix is the Qwen3.8 hybrid: its
Gated DeltaNet keeps the same matrix state per head as the retention layers here. Measured per size: the CUDA-graph decode step at
several batch sizes (device work of the step, replayed), prefill steps of 512 and 2048 tokens, and the per-op device times
of both (eager, CUDA events between the ops) with the fraction of the measured roofline each op reaches: bytes for decode,
FLOPs for the products and the attention of prefill.
"""

from __future__ import annotations

import json
import shutil
import struct
import tempfile
from pathlib import Path

import numpy as np

SIZES = {
    "small": dict(width=2048, ff=5632, heads=16, kv_heads=4, dim=128, vdim=128),
    "medium": dict(width=4096, ff=11008, heads=32, kv_heads=8, dim=128, vdim=128),
}
VOCAB, LAYERS, CONTEXT, CHUNKS, BATCHES = 32768, 6, 2048, (512, 2048), (1, 16, 64)


def fegenex_config(s: dict) -> dict:
    W, mlp = s["width"], {"kind": "dense", "ff": s["ff"]}
    kinds = {
        "attention": {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["vdim"], "v_mix": True,
                      "rot": {"base": 10000.0, "dims": s["dim"] // 2}, "scale": s["dim"] ** -0.5},
        "mingru": {"width": W},
        "rglru": {"width": W, "blocks": W // 256, "conv": 4},
    }
    order = ["mingru", "rglru", "attention"] * (LAYERS // 3)
    return {"architecture": "Fegenex", "width": W, "vocab": VOCAB, "max_positions": 8192, "norm": {"eps": 1e-6},
            "layers": [{"type": t, "mixer": kinds[t], "mlp": mlp} for t in order]}


def nololix_config(s: dict) -> dict:
    W, mlp = s["width"], {"kind": "dense", "ff": s["ff"]}
    H = W // 128
    kinds = {
        "retention": {"heads": H, "dim": 128, "vdim": 128, "decay": [1.0 - 2.0 ** -(5 + 5 * h / H) for h in range(H)],
                      "rot": {"base": 10000.0, "dims": 128}},
        "latent_attention": {"heads": s["heads"], "dim": s["dim"], "vdim": s["vdim"], "q_rank": 3 * W // 8, "kv_rank": 512,
                             "scale": s["dim"] ** -0.5},
    }
    order = ["retention", "retention", "latent_attention"] * (LAYERS // 3)
    return {"architecture": "Nololix", "width": W, "vocab": VOCAB, "embedding": {"scale": 1.0}, "norm": {"eps": 1e-6, "groups": 8},
            "streams": 2, "residual_mult": 0.5, "loop": None,
            "layers": [{"type": t, "mixer": kinds[t], "mlp": mlp} for t in order]}


def nololix_shapes(cfg: dict) -> dict[str, tuple]:
    W, V, S = cfg["width"], cfg["vocab"], cfg["streams"]
    t = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        x, H = p + "mix.", m["heads"]
        for q in "12":
            t[f"{p}norm{q}"] = (W,)
            t[f"{p}hc{q}.in"], t[f"{p}hc{q}.out"], t[f"{p}hc{q}.mix"] = (S,), (S,), (S, S)
        if layer["type"] == "retention":
            for n, d in (("q", m["dim"]), ("k", m["dim"]), ("v", m["vdim"]), ("g", m["vdim"])):
                t[x + n] = (H * d, W)
        else:
            for n, rank in (("dq", m["q_rank"]), ("dkv", m["kv_rank"])):
                t[x + n], t[x + n + ".norm"] = (rank, W), (rank,)
            t[x + "uq"], t[x + "uk"] = (H * m["dim"], m["q_rank"]), (H * m["dim"], m["kv_rank"])
            t[x + "uv"], t[x + "g"] = (H * m["vdim"], m["kv_rank"]), (H * m["vdim"], W)
        t[x + "o"] = (W, H * m["vdim"])
        t[p + "mlp.up"], t[p + "mlp.down"], t[p + "mlp.act"] = (layer["mlp"]["ff"], W), (W, layer["mlp"]["ff"]), (2,)
    return t


def fegenex_shapes(cfg: dict) -> dict[str, tuple]:
    W, V = cfg["width"], cfg["vocab"]
    t = {"embed": (V, W), "pos": (cfg["max_positions"], W), "final.norm": (), "head": (V, W)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        for n in ("norm1", "norm1b", "norm2", "norm2b"):
            t[p + n] = ()
        x = p + "mix."
        if layer["type"] == "attention":
            for n, rows in (("q", m["heads"] * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])):
                t[x + n], t[x + n + ".b"] = (rows, W), (rows,)
            t[x + "o"], t[x + "o.b"] = (W, m["heads"] * m["vdim"]), (W,)
            t[x + "talk"], t[x + "vmix"] = (m["heads"], m["heads"]), ()
        elif layer["type"] == "mingru":
            for n in "zxg":
                t[x + n] = (m["width"], W)
            t[x + "z.b"], t[x + "x.b"], t[x + "o"] = (m["width"],), (m["width"],), (W, m["width"])
        else:
            w, nb = m["width"], m["blocks"]
            for n in "yx":
                t[x + n], t[x + n + ".b"] = (w, W), (w,)
            t[x + "conv"], t[x + "conv.b"], t[x + "lam"], t[x + "o"] = (w, m["conv"]), (w,), (w,), (W, w)
            for n in ("ra", "ri"):
                t[x + n], t[x + n + ".b"] = (nb, w // nb, w // nb), (nb, w // nb)
        t[p + "mlp.gate"] = t[p + "mlp.up"] = (layer["mlp"]["ff"], W)
        t[p + "mlp.down"] = (W, layer["mlp"]["ff"])
    return t


def write_random_folder(folder: Path, cfg: dict, shapes: dict, seed: int = 5) -> Path:
    """Gaussian weights scaled by fan-in, cut from one random block (timing does not depend on their values)."""
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    block = np.random.default_rng(seed).standard_normal(1 << 22, dtype=np.float32)
    head, at = {}, 0
    for name, shape in shapes.items():
        n = int(np.prod(shape)) * 2
        head[name] = {"dtype": "BF16", "shape": list(shape), "data_offsets": [at, at + n]}
        at += n
    text = json.dumps(head).encode()
    with open(folder / "model.safetensors", "wb") as f:
        f.write(struct.pack("<Q", len(text)) + text)
        for name, shape in shapes.items():
            n = int(np.prod(shape))
            scale = 1.0 / np.sqrt(shape[-1]) if len(shape) > 1 and name not in ("embed", "pos") else 1.0 if shape else 0.0
            bits = ((block * scale + (0.0 if shape else 1.0)).view(np.uint32) >> 16).astype(np.uint16)
            for lo in range(0, n, len(bits)):
                f.write(bits[:min(len(bits), n - lo)].tobytes())
    return folder


def _costs():
    """op -> (decode bytes(batch, context), prefill FLOPs(tokens, first position)); None where bytes bound prefill too."""
    cost: dict[str, list] = {}

    def add(op, by, fl=None):
        cost.setdefault(op, []).append((by, fl))

    def gemm(op, n, k, count=1):
        add(op, lambda b, c: count * (2 * n * k + b * (n + k) * 2), lambda m, p: 2.0 * m * n * k * count)
    return cost, add, gemm


def nololix_costs(cfg: dict):
    W, V, S = cfg["width"], cfg["vocab"], cfg["streams"]
    cost, add, gemm = _costs()
    gemm("gemm.lm_head", V, W)
    for layer in cfg["layers"]:
        m, ff = layer["mixer"], layer["mlp"]["ff"]
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        if layer["type"] == "retention":
            gemm("gemm.retention_in", 2 * H * (d + dv), W)
            gemm("gemm.retention_out", W, H * dv)
            row = 2 * H * (2 * d + 3 * dv)
            add("mix.retention", lambda b, c, H=H, d=d, dv=dv, row=row: b * (8 * H * d * dv + row), ("bytes", lambda n, p, row=row: n * row))
        else:
            qr, r = m["q_rank"], m["kv_rank"]
            gemm("gemm.latent_in", qr + r + H * dv, W)
            gemm("gemm.latent_uq", H * d, qr)
            gemm("gemm.latent_uk", r, d, H)
            add("gemm.latent_kv", lambda b, c: 0, lambda n, p, r=r, H=H, d=d, dv=dv: 2.0 * (n + p) * r * H * (d + dv))
            gemm("gemm.latent_uv", dv, r, H)
            gemm("gemm.latent_o", W, H * dv)
            # prefill: the FLOPs of the heads' own dimensions, however the kernel arranges the products
            add("mix.latent", lambda b, c, r=r, H=H: b * (c * r * 2 + 4 * H * r),
                lambda n, p, H=H, d=d, dv=dv: 2.0 * H * (d + dv) * n * (p + (n + 1) / 2))
            add("mix.latent_append", lambda b, c, qr=qr, r=r: b * 4 * (qr + r))
        gemm("gemm.mlp_up", ff, W)
        gemm("gemm.mlp_down", W, ff)
        for _ in range(2):
            add("residual_norm", lambda b, c: b * W * (4 + 8 * S + 2), ("bytes", lambda n, p: n * W * (4 + 8 * S + 2)))
    return cost


def fegenex_costs(cfg: dict):
    W, V = cfg["width"], cfg["vocab"]
    cost, add, gemm = _costs()
    gemm("gemm.lm_head", V, W)
    for layer in cfg["layers"]:
        m, t = layer["mixer"], layer["type"]
        if t == "attention":
            H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            gemm("gemm.attn_qkv", H * d + G * (d + dv), W)
            gemm("gemm.attn_o", W, H * dv)
            add("mix.attn", lambda b, c, G=G, d=d, dv=dv: b * c * G * (d + dv) * 2,
                lambda n, p, H=H, d=d, dv=dv: 2.0 * H * (d + dv + H) * n * (p + (n + 1) / 2))
            add("mix.rope_append", lambda b, c, H=H, G=G, d=d, dv=dv: b * 2 * 2 * (H * d + G * (d + dv)))
        else:
            w = m["width"]
            parts = 3 if t == "mingru" else 2
            gemm(f"gemm.{t}_in", parts * w, W)
            gemm(f"gemm.{t}_out", W, w)
            gates = 0 if t == "mingru" else 2 * w * (w // m["blocks"]) * 2
            taps = 0 if t == "mingru" else m["conv"]
            add(f"mix.{t}", lambda b, c, w=w, parts=parts, gates=gates, taps=taps: gates + b * w * (parts * 2 + 2 * 4 + taps * 2 + 2),
                ("bytes", lambda n, p, w=w, parts=parts, gates=gates: gates + n * w * (parts * 2 + 2)))
        gemm("gemm.mlp_gate_up", 2 * layer["mlp"]["ff"], W)
        gemm("gemm.mlp_down", W, layer["mlp"]["ff"])
        for _ in range(2):
            add("residual_norm", lambda b, c: b * W * (4 + 8 + 2), ("bytes", lambda n, p: n * W * (4 + 8 + 2)))
    return cost


def qwen_costs(cfg: dict, recipe: str, by_role):
    H, I = cfg["hidden_size"], cfg["intermediate_size"]
    nq, nkv, lk, lv = cfg["num_attention_heads"], cfg["num_key_value_heads"], cfg["linear_num_key_heads"], cfg["linear_num_value_heads"]
    n_attn = sum(t == "full_attention" for t in cfg["layer_types"])
    n_gdn = len(cfg["layer_types"]) - n_attn
    conv = 2 * lk * 128 + lv * 128
    flops = {"gemm.attn_qkvg": n_attn * (2 * nq + 2 * nkv) * 256 * H, "gemm.attn_o": n_attn * H * nq * 256,
             "gemm.gdn_qkvz": n_gdn * (conv + lv * 128) * H, "gemm.gdn_out": n_gdn * H * lv * 128,
             "gemm.mlp_gate_up": len(cfg["layer_types"]) * 2 * I * H, "gemm.mlp_down": len(cfg["layer_types"]) * H * I,
             "gemm.lm_head": cfg["vocab_size"] * H}
    cost = {op: [(lambda b, c, n=n: n, lambda m, p, f=flops[op]: 2.0 * m * f)] for op, n in by_role(cfg, recipe).items()}
    cost["attn"] = [(lambda b, c: n_attn * b * c * 2 * nkv * 264, lambda n, p: n_attn * 4.0 * nq * 256 * n * (p + (n + 1) / 2))]
    cost["gdn.recurrence"] = [(lambda b, c: n_gdn * b * (2 * lv * 65536 + conv * 4 + 4 * lv * 128),
                               ("bytes", lambda n, p: n_gdn * n * (conv * 4 + 4 * lv * 128)))]
    cost["gdn.conv"] = [(lambda b, c: n_gdn * b * conv * 18, ("bytes", lambda n, p: n_gdn * n * conv * 6))]
    return cost


def fractions(per_op: dict, cost: dict, peaks: dict, decode, prefill) -> dict:
    """ms per op with the fraction of the roofline: decode = (batch, context), prefill = (tokens, first position)."""
    out = {}
    for op, ms in sorted(per_op.items(), key=lambda kv: -kv[1]):
        key = op.replace("_decode", "").replace("_prefill", "").replace("attn.decode", "attn").replace("attn.prefill", "attn")
        rec = {"ms": round(ms, 4)}
        parts = cost.get(key)
        if parts and ms > 0:
            if decode:
                rec["frac_hbm"] = round(sum(by(*decode) for by, _ in parts) / ms / 1e6 / peaks["hbm_gbs"], 4)
            elif parts[0][1] is not None:
                if isinstance(parts[0][1], tuple):
                    rec["frac_hbm"] = round(sum(f[1](*prefill) for _, f in parts) / ms / 1e6 / peaks["hbm_gbs"], 4)
                else:
                    rec["frac_tensor"] = round(sum(f(*prefill) for _, f in parts) / ms / 1e9 / peaks["bf16_tflops"], 4)
        out[op] = rec
    return out


def measure(eng, path: Path, cost: dict, peaks: dict, seed: int = 3) -> dict:
    model = eng.Model(path)
    chunk = max(CHUNKS)
    runner = eng.Runner(model, eng.default_runner_options(max_batch=max(BATCHES), prefill_chunk=chunk, verbose=0,
                                                          kv_tokens=max(BATCHES) * (CONTEXT + 192), max_context=CONTEXT + 128))
    rng, g = np.random.default_rng(seed), eng.greedy()
    out: dict = {"summary": model.summary(), "decode": {}, "prefill": {}}
    ids = lambda n: rng.integers(0, model.vocab, n).astype(np.int32)
    prompt = ids(CONTEXT)
    for n in CHUNKS:  # one prompt in chunks of n; the second run is timed
        for _ in range(3):
            runner.reset_slot(0)
            assert runner.kv_ensure(0, CONTEXT + 64)
            ms = 0.0
            for at in range(0, CONTEXT, n):
                runner.prefill([(0, at, prompt[at:at + n], None, 0)])
                ms += runner.last_step_ms()
        out["prefill"][n] = {"tok_per_s": CONTEXT / ms * 1000.0, "ms_per_step": ms * n / CONTEXT}
        runner.set_profiling(True)
        runner.profile(clear=True)
        last = CONTEXT - n
        runner.reset_slot(0)
        for at in range(0, CONTEXT, n):
            if at == last:
                runner.profile(clear=True)
            runner.prefill([(0, at, prompt[at:at + n], g if at == last else None, 0)])
        ops = {k: v[0] for k, v in runner.profile(clear=True).items() if k not in ("start", "sample")}
        runner.set_profiling(False)
        head = ops.pop("gemm.lm_head", None)
        del head  # one row only
        out["prefill"][n]["ops"] = fractions(ops, cost, peaks, None, (n, last))
    for s in range(max(BATCHES)):
        runner.reset_slot(s)
        assert runner.kv_ensure(s, CONTEXT + 64)
        runner.prefill([(s, 0, prompt[:CONTEXT - 1], None, 0)])
    for b in BATCHES:
        rows = [(s, CONTEXT - 1, 17, g, 1) for s in range(b)]
        for _ in range(3):
            runner.decode(rows)
        ms = min(runner.replay_decode_core(b, 50) for _ in range(3))
        out["decode"][b] = {"ms_per_step": ms, "tok_per_s": b / ms * 1000.0}
        runner.set_profiling(True)
        runner.decode(rows)
        runner.profile(clear=True)
        for _ in range(5):
            runner.decode(rows)
        ops = {k: v[0] / 5 for k, v in runner.profile(clear=True).items() if k != "start"}
        runner.set_profiling(False)
        out["decode"][b]["ops"] = fractions(ops, cost, peaks, (b, CONTEXT), None)
    runner.close()
    model.close()
    return out


DESIGNS = {"fegenex": (fegenex_config, fegenex_shapes, fegenex_costs), "nololix": (nololix_config, nololix_shapes, nololix_costs)}


def run(eng, synth, sizes: list[str], peaks: dict, by_role, log, recipe: str = "default", models=("fegenex", "nololix", "qwen38")) -> dict:
    result = {}
    for name in sizes:
        s = SIZES[name]
        tmp = Path(tempfile.mkdtemp(prefix="design_bench_"))
        result[name] = {}
        try:
            for model in models:
                log(f"design bench {name}: {model}")
                if model in DESIGNS:
                    config, shapes, costs = DESIGNS[model]
                    cfg = config(s)
                    result[name][model] = measure(eng, write_random_folder(tmp / model, cfg, shapes(cfg)), costs(cfg), peaks)
                    continue
                W = s["width"]
                types = ["linear_attention", "linear_attention", "full_attention"] * (LAYERS // 3)
                qcfg = synth.model_config(hidden=W, vocab=VOCAB, layers=LAYERS, intermediate=s["ff"], nq=s["heads"] * s["dim"] // 256,
                                          nkv=s["kv_heads"] * s["dim"] // 256, lk=W // 256, lv=W // 128, layer_types=types)
                path = tmp / "qwen.q38"
                synth.write_random_planes_q38(path, qcfg, recipe=recipe)
                result[name][model] = measure(eng, path, qwen_costs(qcfg, recipe, by_role), peaks)
        finally:
            shutil.rmtree(tmp, ignore_errors=True)
    return result
