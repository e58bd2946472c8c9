"""Zupudra checkpoints: config.json and tensor names -> the catalog the cuda session is created from.

A Zupudra model is a decoder whose layers are listed one by one; each names its mixer (retention, a gated
linear recurrence, attention over cached latents) with that mixer's sizes, and optionally a gated
feed-forward. Every size and constant comes from config.json. A layer may run with another layer's
parameters and then has no tensors of its own. The embedding table is also the output matrix.

The catalog carries the layers as generic mixer entries (`config["mixers"]`), which is all the native
session knows: another design made of the same mixers needs only a reader like this one.
"""
from __future__ import annotations

ARCHITECTURE = "Zupudra"

# tensor suffix -> canonical name inside a layer
_COMMON = {"norm1": "attn_norm.weight", "norm2": "ffn_norm.weight", "mlp.gate": "ffn_gate.weight",
           "mlp.up": "ffn_up.weight", "mlp.down": "ffn_down.weight"}
_MIXER_TENSORS = {
    "retention": {"mix.q": "attn_q.weight", "mix.k": "attn_k.weight", "mix.v": "attn_v.weight",
                  "mix.g": "attn_gate.weight", "mix.o": "attn_output.weight"},
    "rglru": {"mix.y": "rec_y.weight", "mix.y.b": "rec_y.bias", "mix.x": "rec_x.weight", "mix.x.b": "rec_x.bias",
              "mix.conv": "rec_conv.weight", "mix.conv.b": "rec_conv.bias", "mix.ra": "rec_a_gate.weight",
              "mix.ra.b": "rec_a_gate.bias", "mix.ri": "rec_i_gate.weight", "mix.ri.b": "rec_i_gate.bias",
              "mix.lam": "rec_lambda", "mix.o": "rec_output.weight"},
    "latent_attention": {"mix.q": "attn_q.weight", "mix.dkv": "attn_kv_down.weight",
                         "mix.dkv.norm": "attn_kv_norm.weight", "mix.uk": "attn_k_up.weight",
                         "mix.uv": "attn_v_up.weight", "mix.g": "attn_gate.weight", "mix.o": "attn_output.weight"},
}
_GLOBAL = {"embed": "token_embd.weight", "final.norm": "output_norm.weight"}


def owner(layers: list, i: int) -> int:
    """The layer whose tensors layer i runs with."""
    seen = set()
    while layers[i].get("weights_of") is not None:
        if i in seen:
            raise ValueError(f"layers share tensors in a circle at layer {i}")
        seen.add(i)
        i = int(layers[i]["weights_of"])
        if not 0 <= i < len(layers):
            raise ValueError(f"weights_of names layer {i} of {len(layers)}")
    return i


def mixer_entry(layers: list, i: int) -> dict:
    """One layer as the native session takes it."""
    layer = layers[i]
    kind, m = layer["type"], layer["mixer"]
    if kind not in _MIXER_TENSORS:
        raise ValueError(f"layer {i}: unknown mixer `{kind}`")
    mlp = layer.get("mlp")
    if mlp and mlp.get("kind", "dense") != "dense":
        raise ValueError(f"layer {i}: unknown feed-forward `{mlp['kind']}`")
    e = {"type": kind, "tensors": owner(layers, i), "ff": int(mlp["ff"]) if mlp else 0}
    if kind == "retention":
        rot = m.get("rot") or {"dims": 0, "base": 0.0}
        e.update(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), rot_dims=int(rot["dims"]),
                 rot_base=float(rot["base"]), decay=[float(d) for d in m["decay"]])
    elif kind == "rglru":
        e.update(width=int(m["width"]), blocks=int(m["blocks"]), taps=int(m["conv"]))
    else:
        e.update(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), rank=int(m["kv_rank"]),
                 scale=float(m["scale"]))
    return e


def state_floats(e: dict) -> int:
    """f32 state of one slot of a layer: what it carries from token to token besides cached latents."""
    if e["type"] == "retention":
        return e["heads"] * e["dim"] * e["vdim"]
    return e["width"] * (1 + e["taps"]) if e["type"] == "rglru" else 0


def config(doc: dict) -> dict:
    """Normalised metadata, as for every other architecture, plus the list of mixers."""
    layers = doc["layers"]
    mixers = [mixer_entry(layers, i) for i in range(len(layers))]
    attn = [e for e in mixers if "heads" in e]
    ranks = [e["rank"] for e in mixers if "rank" in e]
    return {
        "model_type": "zupudra", "layers": len(layers), "hidden": int(doc["width"]),
        "intermediate": max((e["ff"] for e in mixers), default=0),
        "heads": max((e["heads"] for e in attn), default=1),
        # the cache holds one latent vector per token and latent-attention layer
        "kv_heads": 1, "head_dim": max(ranks, default=1), "kv_elements_per_token": sum(ranks),
        "state_bytes_per_slot": 4 * sum(state_floats(e) for e in mixers),
        "vocab": int(doc["vocab"]), "eps": float(doc["norm"]["eps"]), "context_length": 0,
        "qk_norm": False, "rope": False, "tied": True, "mixers": mixers,
    }


def tensor_names(doc: dict) -> dict:
    """Checkpoint tensor name -> canonical parameter name, for every tensor the model has."""
    names = dict(_GLOBAL)
    for i, layer in enumerate(doc["layers"]):
        if owner(doc["layers"], i) != i:
            continue
        own = dict(_COMMON, **_MIXER_TENSORS[layer["type"]])
        for suffix, canon in own.items():
            if not layer.get("mlp") and (suffix == "norm2" or suffix.startswith("mlp.")):
                continue
            names[f"l{i}.{suffix}"] = f"blk.{i}.{canon}"
    return names
