"""Rufusun checkpoints: config.json and tensor names -> the catalog the cuda session is created from.

A Rufusun model is a decoder whose layers are listed one by one; each names its mixer (softmax attention with
capped scores, gated delta rule) with that mixer's sizes, and optionally a feed-forward: dense, or a mixture of
experts with a shared one. Mixer and feed-forward of a layer read the same residual row through a norm each.
Norm weights are stored around zero. A span of layers may run several times in a row with the same tensors;
every run has a cache or state of its own, so the catalog lists runs, and runs after the first borrow tensors.

The catalog carries the runs as generic mixer entries (`config["mixers"]`), which is all the native session
knows: another design made of the same mixers needs only a reader like this one.
"""
from __future__ import annotations

ARCHITECTURE = "Rufusun"

# tensor suffix -> canonical name inside a layer
_NORMS = {"norm1": "attn_norm.weight", "norm2": "ffn_norm.weight"}
_MIXER_TENSORS = {
    "attention": {"mix.q": "attn_q.weight", "mix.q.b": "attn_q.bias", "mix.k": "attn_k.weight", "mix.k.b": "attn_k.bias",
                  "mix.v": "attn_v.weight", "mix.v.b": "attn_v.bias", "mix.o": "attn_output.weight",
                  "mix.o.b": "attn_output.bias"},
    "delta": {"mix.q": "attn_q.weight", "mix.k": "attn_k.weight", "mix.v": "attn_v.weight", "mix.g": "attn_gate.weight",
              "mix.b": "delta_beta.weight", "mix.a": "delta_decay.weight", "mix.q.conv": "conv_q.weight",
              "mix.k.conv": "conv_k.weight", "mix.v.conv": "conv_v.weight", "mix.A_log": "delta_a_log",
              "mix.dt_bias": "delta_dt.bias", "mix.norm": "head_norm.weight", "mix.o": "attn_output.weight"},
}
_GLOBAL = {"embed": "token_embd.weight", "final.norm": "output_norm.weight", "head": "output.weight"}


def run_order(doc: dict) -> list:
    """The layers in the order they run."""
    n = len(doc["layers"])
    loop = doc.get("loop")
    if not loop:
        return list(range(n))
    start, stop, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    if not (0 <= start <= stop <= n and times >= 1):
        raise ValueError(f"loop of layers {start}..{stop} x {times} in a model of {n}")
    return list(range(start)) + list(range(start, stop)) * times + list(range(stop, n))


def first_runs(doc: dict) -> dict:
    """Layer -> the run that owns its tensors."""
    out = {}
    for run, i in enumerate(run_order(doc)):
        out.setdefault(i, run)
    return out


def mixer_entry(layer: dict, i: int, run: int) -> dict:
    """One run of a layer as the native session takes it; its tensors are those of run `run`."""
    kind, m = layer["type"], layer["mixer"]
    if kind not in _MIXER_TENSORS:
        raise ValueError(f"layer {i}: unknown mixer `{kind}`")
    e = {"type": "softmax_attention" if kind == "attention" else "gated_delta", "tensors": run, "ff": 0, "parallel": 1,
         "heads": int(m["heads"]), "kv_heads": int(m["kv_heads"]), "dim": int(m["dim"]), "vdim": int(m["vdim"])}
    if kind == "attention":
        rot = m.get("rot") or {"dims": 0, "base": 0.0}
        e.update(rot_dims=int(rot["dims"]), rot_base=float(rot["base"]), scale=float(m["scale"]),
                 softcap=float(m.get("softcap") or 0.0), bias=1)
    else:
        e.update(taps=int(m["conv"]))
    mlp = layer.get("mlp")
    if not mlp:
        return e
    ff_kind = mlp.get("kind", "dense")
    if ff_kind == "dense":
        e["ff"] = int(mlp["ff"])
    elif ff_kind == "moe":
        shared = mlp.get("shared")
        e.update(experts=int(mlp["router"]["experts"]), top=int(mlp["router"]["top"]), expert_ff=int(mlp["expert"]["ff"]),
                 expert_limit=float(mlp["expert"]["limit"]), shared_ff=int(shared["ff"]) if shared else 0,
                 shared_limit=float(shared["limit"]) if shared else 0.0)
        if not 1 <= e["top"] <= e["experts"]:
            raise ValueError(f"layer {i}: {e['top']} of {e['experts']} experts")
    else:
        raise ValueError(f"layer {i}: unknown feed-forward `{ff_kind}`")
    return e


def state_floats(e: dict) -> int:
    """f32 state of one slot of a run: the delta rule's matrix and the convolution's window."""
    if e["type"] != "gated_delta":
        return 0
    return e["heads"] * e["dim"] * e["vdim"] + e["taps"] * (2 * e["kv_heads"] * e["dim"] + e["heads"] * e["vdim"])


def config(doc: dict) -> dict:
    """Normalised metadata, as for every other architecture, plus the list of mixers."""
    owner = first_runs(doc)
    mixers = [mixer_entry(doc["layers"][i], i, owner[i]) for i in run_order(doc)]
    attn = [e for e in mixers if e["type"] == "softmax_attention"]
    return {
        "model_type": "rufusun", "layers": len(mixers), "hidden": int(doc["width"]),
        "intermediate": max((max(e["ff"], e.get("expert_ff", 0), e.get("shared_ff", 0)) for e in mixers), default=0),
        "heads": max((e["heads"] for e in mixers), default=1), "kv_heads": max((e["kv_heads"] for e in attn), default=1),
        "head_dim": max((max(e["dim"], e["vdim"]) for e in attn), default=1),
        "kv_elements_per_token": sum(e["kv_heads"] * (e["dim"] + e["vdim"]) for e in attn),
        "state_bytes_per_slot": 4 * sum(state_floats(e) for e in mixers),
        "vocab": int(doc["vocab"]), "eps": float(doc["norm"]["eps"]), "context_length": 0,
        "qk_norm": False, "rope": False, "tied": False, "mixers": mixers,
        "norm_offset": 1.0, "logit_scale": float(doc["logit_scale"]),
    }


def _ff_tensors(mlp: dict | None) -> dict:
    if not mlp:
        return {}
    parts = ("gate", "up", "down")
    if mlp.get("kind", "dense") == "dense":
        return {f"mlp.{p}": f"ffn_{p}.weight" for p in parts}
    out = {"mlp.router": "ffn_router.weight"}
    for e in range(int(mlp["router"]["experts"])):
        out.update({f"mlp.e{e}.{p}": f"expert_{e}_{p}.weight" for p in parts})
    if mlp.get("shared"):
        out.update({f"mlp.shared.{p}": f"ffn_{p}.weight" for p in parts})
    return out


def tensor_names(doc: dict) -> dict:
    """Checkpoint tensor name -> canonical parameter name, for every tensor the model has."""
    names = dict(_GLOBAL)
    for i, run in first_runs(doc).items():
        layer = doc["layers"][i]
        own = dict(_NORMS if layer.get("mlp") else {"norm1": _NORMS["norm1"]}, **_MIXER_TENSORS[layer["type"]],
                   **_ff_tensors(layer.get("mlp")))
        names.update({f"l{i}.{suffix}": f"blk.{run}.{canon}" for suffix, canon in own.items()})
    return names
