"""Throughput of a design with listed mixers beside a Qwen3-shaped model of equal size (random bf16 weights).

    python bench.py --arch zupudra|rufusun [--arch-size 0.4b,1b,7b-layers] [--steps K] [--warmup W]

Both models of a size have the same width, layer count, feed-forward width, heads of 128, vocabulary and 16-bit
plain weights. Zupudra's layers alternate retention, gated recurrence and latent attention. Rufusun's alternate gated
delta rule and softmax attention, two layers with a dense feed-forward, then two with 16 experts of which a token uses
four beside a shared one: as many feed-forward weights per token as the dense one. Measured
through the session: prefill of a random prompt (host clock around `prefill_argmax`), single-sequence greedy
decode after it (`decode_loop`, CUDA events on the session stream) and batched decode (`step`, host clock,
tokens in and out through host memory). Prints one JSON line per size.
"""
from __future__ import annotations

import json
import os
import statistics
import tempfile
import time

import numpy as np

from . import synth
from .runtime import ModelLoader, SessionConfig

SEED = 20243
VOCAB = 32768
# width, layers, heads of 128, latent rank, recurrence (width, blocks), feed-forward, kv heads of the GQA model
SIZES = {"0.4b": (1024, 12, 8, 256, (1024, 4), 3072, 4),
         "1b": (2048, 12, 16, 512, (2560, 10), 6144, 8),
         "7b-layers": (4096, 6, 32, 512, (4096, 16), 12288, 8)}


def zupudra_doc(size: str) -> dict:
    width, layers, heads, rank, (rw, blocks), ff, _ = SIZES[size]
    mlp = {"kind": "dense", "ff": ff}
    decay = [1.0 - 2.0 ** -(4.5 + 4 * i / heads) for i in range(heads)]
    kinds = [{"type": "retention", "mixer": {"heads": heads, "dim": 128, "vdim": 128, "decay": decay,
                                             "rot": {"dims": 128, "base": 5e5}}, "mlp": mlp},
             {"type": "rglru", "mixer": {"width": rw, "blocks": blocks, "conv": 4}, "mlp": mlp},
             {"type": "latent_attention", "mixer": {"heads": heads, "dim": 128, "vdim": 128, "kv_rank": rank,
                                                    "scale": 128 ** -0.5}, "mlp": mlp}]
    return {"layers": [kinds[i % 3] for i in range(layers)], "width": width, "vocab": VOCAB, "norm": {"eps": 1e-6}}


def rufusun_doc(size: str) -> dict:
    width, layers, heads, _, _, ff, kv = SIZES[size]
    dense = {"kind": "dense", "ff": ff}
    moe = {"kind": "moe", "expert": {"ff": ff // 6, "limit": 7.0}, "router": {"experts": 16, "top": 4},
           "shared": {"ff": ff // 3, "limit": 7.0}}
    delta = {"heads": heads, "kv_heads": heads // 2, "dim": 128, "vdim": 128, "conv": 4}
    attention = {"heads": heads, "kv_heads": kv, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "softcap": 30.0,
                 "rot": {"dims": 128, "base": 5e5}}
    kinds = [{"type": t, "mixer": m, "mlp": f} for f in (dense, moe) for t, m in (("delta", delta), ("attention", attention))]
    return {"layers": [kinds[i % 4] for i in range(layers)], "width": width, "vocab": VOCAB, "norm": {"eps": 1e-6},
            "logit_scale": 1.0}


# architecture -> configuration, shapes, weights, writer, kinds of layers in turn
DESIGNS = {"zupudra": (zupudra_doc, synth.zupudra_shapes, synth.zupudra_tensors, synth.write_zupudra, 3),
           "rufusun": (rufusun_doc, synth.rufusun_shapes, synth.rufusun_tensors, synth.write_rufusun, 4)}


def qwen_config(size: str) -> dict:
    width, layers, heads, _, _, ff, kv = SIZES[size]
    return dict(layers=layers, hidden=width, heads=heads, kv_heads=kv, head_dim=128, intermediate=ff, vocab=VOCAB, eps=1e-6,
                theta=1e6)


def checkpoint(kind: str, size: str) -> str:
    """The seeded checkpoint, written on first use; layers of one kind carry the same random bytes."""
    d = os.environ.get("DYNINFER_BENCH_DIR") or os.path.join(tempfile.gettempdir(), "dyninfer_b200_bench")
    os.makedirs(d, exist_ok=True)
    path = os.path.join(d, f"{kind}_{size}_bf16_seed{SEED}" + (".gguf" if kind == "qwen3" else ""))
    if os.path.exists(path):
        return path
    tmp = path + f".tmp{os.getpid()}"
    if kind == "qwen3":
        synth.write_qwen3_gguf(tmp, qwen_config(size), seed=SEED, default="plain.bf16", embd="plain.bf16", repeat_layers=True)
    else:
        doc_of, shapes, random_tensors, write, kinds = DESIGNS[kind]
        doc = doc_of(size)
        first = random_tensors(dict(doc, layers=doc["layers"][:kinds]), SEED)
        tensors = {}
        for name in shapes(doc):
            p, _, rest = name.partition(".")
            src = f"l{int(p[1:]) % kinds}.{rest}" if p[0] == "l" and p[1:].isdigit() else name
            tensors[name] = first[src]
        write(tmp, doc, tensors=tensors)
    os.replace(tmp, path)
    return path


def measure(path: str, prompt_len: int, steps: int, warmup: int, batches=(8, 32), chunk: int = 512) -> dict:
    import torch
    cap = prompt_len + 2 * (steps + warmup) + 64
    ids = np.random.default_rng(SEED).integers(0, VOCAB, size=prompt_len).tolist()
    out = {}
    model = ModelLoader().load(path, max_kv=cap, kv_dtype="bf16", chunk_size=chunk)
    with model.create_session(SessionConfig(cap)) as s:
        times = []
        for i in range(2 + 5):
            torch.cuda.synchronize()
            t0 = time.perf_counter()
            tok = s.prefill_argmax(ids)
            if i >= 2:
                times.append(time.perf_counter() - t0)
        out["prefill_tokens_per_s"] = round(prompt_len / statistics.median(times))
        toks, _ = s.decode_loop(tok, max(3, warmup))
        n0 = s.launch_count()
        _, ms = s.decode_loop(int(toks[-1]), steps)
        out.update(decode_ms_per_step=round(ms / steps, 4), decode_tokens_per_s=round(1e3 * steps / ms, 1),
                   launches_per_step=round((s.launch_count() - n0) / steps, 1), weight_bytes_per_step=s.decode_weight_bytes(),
                   weight_gbs=round(s.decode_weight_bytes() * steps / ms / 1e6, 1))
    for b in batches:
        with model.create_batched_session(SessionConfig(cap, batch_size=b)) as s:
            feed = {i: s.prefill_slot(i, ids[: prompt_len // 4 + i]) for i in range(b)}
            for _ in range(max(3, warmup)):
                feed = s.step(feed)
            torch.cuda.synchronize()
            t0 = time.perf_counter()
            for _ in range(steps):
                feed = s.step(feed)
            out[f"batch{b}_tokens_per_s"] = round(b * steps / (time.perf_counter() - t0), 1)
    return out


def run(arch: str, sizes, prompt_len: int, steps: int, warmup: int, clocks) -> None:
    for size in sizes:
        line = {"metric": "arch_tokens_per_s", "arch": arch, "size": size, "prompt": prompt_len, "steps": steps,
                "warmup": warmup, "dtype": "bf16 weights and cache", "data": "synthetic", "n_gpus": 1,
                "l2": "each decode step streams more weight bytes than L2 holds"}
        paths = {kind: checkpoint(kind, size) for kind in (arch, "qwen3")}
        with clocks() as c:
            for kind, path in paths.items():
                line[kind] = measure(path, prompt_len, steps, warmup)
        line["clocks"] = c.summary()
        print(json.dumps(line), flush=True)


def profile_case(kind: str, size: str, prompt_len: int, steps: int) -> None:
    """One prefill and a few decode steps, for a launch list."""
    ids = np.random.default_rng(SEED).integers(0, VOCAB, size=prompt_len).tolist()
    model = ModelLoader().load(checkpoint(kind, size), max_kv=prompt_len + steps + 8, kv_dtype="bf16")
    with model.create_session(SessionConfig(prompt_len + steps + 8)) as s:
        tok = s.prefill_argmax(ids)
        for _ in range(steps):
            tok = s.decode_argmax(tok)
