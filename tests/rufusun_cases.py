"""Small Rufusun configurations for the tests: sizes that differ from each other in every model, odd ones that
no fast kernel takes, and ones that reach the tensor-core, grouped and fused paths."""
import numpy as np

from dyninfer_b200 import synth


def attention(heads=6, kv_heads=2, dim=20, vdim=12, dims=14, base=3000.0, scale=0.3, softcap=7.0, mlp=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                                           "softcap": softcap, "rot": {"dims": dims, "base": base}}, "mlp": mlp}


def delta(heads=4, kv_heads=2, dim=12, vdim=20, conv=3, mlp=None):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts=5, top=2, ff=28, limit=0.8, shared=36, shared_limit=1.7):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top},
            "shared": {"ff": shared, "limit": shared_limit} if shared else None}


def model(layers, width=44, vocab=101, eps=1e-5, loop=None, logit_scale=0.7):
    doc = {"layers": layers, "width": width, "vocab": vocab, "norm": {"eps": eps}, "logit_scale": logit_scale}
    return dict(doc, loop=loop) if loop else doc


def span(start, stop, times):
    return {"start": start, "stop": stop, "times": times}


def mixed():
    """Every mixer with every feed-forward, a loop in the middle, no size a multiple of the others."""
    return model([attention(mlp=dense(52)), delta(mlp=moe()), attention(heads=5, kv_heads=5, dim=8, vdim=28, dims=8, mlp=moe(7, 3, 20)),
                  delta(heads=3, kv_heads=1, dim=28, vdim=8, conv=5), delta(heads=2, kv_heads=2, dim=16, vdim=24, conv=1, mlp=dense(40)),
                  attention(heads=4, kv_heads=1, dim=12, vdim=16, dims=4, softcap=30.0)], loop=span(1, 4, 2))


def fast():
    """Widths that the tensor-core GEMM, the streaming GEMV, the chunked delta rule, grouped products and the
    tensor-core attention take."""
    return model([delta(heads=4, kv_heads=2, dim=64, vdim=64, conv=4, mlp=moe(8, 3, 64, 1.5, 128, 2.5)),
                  attention(heads=8, kv_heads=2, dim=64, vdim=128, dims=32, scale=0.15, softcap=20.0, mlp=dense(256)),
                  delta(heads=2, kv_heads=1, dim=128, vdim=96, conv=4, mlp=dense(192)),
                  attention(heads=4, kv_heads=4, dim=128, vdim=64, dims=128, scale=0.1, softcap=12.0, mlp=moe(4, 1, 128, 0.9, 64, 1.2))],
                 width=256, vocab=320, eps=1e-6, loop=span(0, 2, 2))


MECHANISMS = {
    "attention": model([attention()]),
    "attention_one_kv_head": model([attention(heads=7, kv_heads=1, dim=16, vdim=40, dims=16)]),
    "attention_no_groups": model([attention(heads=3, kv_heads=3, dim=24, vdim=24, dims=2, scale=1.0, softcap=3.0)]),
    "attention_fast": model([attention(heads=12, kv_heads=2, dim=64, vdim=64, dims=64, scale=0.2)], width=64),
    "attention_fast_uneven": model([attention(heads=4, kv_heads=2, dim=40, vdim=104, dims=24)], width=72),
    "attention_wide_heads": model([attention(heads=4, kv_heads=2, dim=200, vdim=136, dims=100)], width=64),
    "attention_very_wide_heads": model([attention(heads=2, kv_heads=1, dim=300, vdim=290, dims=70)], width=64),
    "attention_dense": model([attention(mlp=dense(60))]),
    "attention_moe": model([attention(mlp=moe())]),
    "delta": model([delta()]),
    "delta_one_tap": model([delta(heads=3, kv_heads=3, dim=8, vdim=36, conv=1)]),
    "delta_many_taps": model([delta(heads=5, kv_heads=1, dim=20, vdim=12, conv=7)]),
    "delta_chunks": model([delta(heads=6, kv_heads=2, dim=48, vdim=40, conv=4)], width=64),
    "delta_chunks_uneven": model([delta(heads=2, kv_heads=2, dim=40, vdim=72, conv=2)], width=64),
    "delta_chunks_wide": model([delta(heads=2, kv_heads=1, dim=128, vdim=136, conv=6)], width=64),
    "delta_wide_keys": model([delta(heads=2, kv_heads=1, dim=200, vdim=48, conv=4)], width=64),
    "delta_wide_values": model([delta(heads=1, kv_heads=1, dim=24, vdim=300, conv=2)]),
    "delta_dense": model([delta(mlp=dense(36))]),
    "moe": model([delta(heads=2, kv_heads=1, mlp=moe(9, 4, 20, 0.5, 12, 3.0))]),
    "moe_one_of_one": model([attention(heads=2, kv_heads=1, mlp=moe(1, 1, 24))]),
    "moe_all_chosen": model([delta(mlp=moe(4, 4, 16))]),
    "moe_many_experts": model([delta(mlp=moe(70, 2, 8))]),
    "moe_nothing_shared": model([delta(mlp=moe(6, 2, 20, shared=0))]),
    "moe_grouped": model([delta(heads=2, kv_heads=1, dim=16, vdim=16, mlp=moe(6, 2, 64, 1.1, 192))], width=128),
    "moe_grouped_wide_limit": model([delta(heads=2, kv_heads=1, dim=16, vdim=16, mlp=moe(6, 2, 64, 900.0, 192, 1e6))], width=128),
    "moe_grouped_narrow_limit": model([delta(heads=2, kv_heads=1, dim=16, vdim=16, mlp=moe(6, 2, 64, 0.03, 192, 0.01))], width=128),
    "moe_grouped_uneven": model([delta(heads=2, kv_heads=1, dim=16, vdim=16, mlp=moe(40, 7, 128, 1.1, 72))], width=256),
    "odd_widths": model([delta(heads=3, kv_heads=1, dim=7, vdim=9, conv=4, mlp=moe(5, 2, 11, 1.0, 13)),
                         attention(heads=3, kv_heads=3, dim=9, vdim=5, dims=6, mlp=dense(17))], width=33, vocab=67),
    "loop_of_one": model([delta(), attention(), delta(heads=2)], loop=span(1, 2, 3)),
    "loop_of_all": model([delta(mlp=dense(20)), attention()], loop=span(0, 2, 2)),
}


def stored(tensors):
    """Weights as a checkpoint holds them (bf16 values), in float32."""
    return {k: synth.bf16_bits_to_f32(synth.f32_to_bf16_bits(np.ascontiguousarray(v, np.float32))) for k, v in tensors.items()}


CHANNELS = 8


def clear_choices(doc, t, seed=0):
    """Makes every router read a few channels that no layer writes, and the embedding there such that no token's choice
    is a close call: 16-bit operands then never change which experts run, only what they give."""
    routers = [(i, layer["mlp"]["router"]["top"]) for i, layer in enumerate(doc["layers"]) if (layer["mlp"] or {}).get("kind") == "moe"]
    if not routers:
        return t
    rng = np.random.default_rng(seed + 77)
    n = CHANNELS
    for name in t:
        if name.endswith((".o", ".down")):
            t[name][:n] = 0.0
        elif name.endswith(".o.b"):
            t[name][:n] = 0.0
    for i, _ in routers:
        t[f"l{i}.norm2"][:n] = 0.0
        r = t[f"l{i}.mlp.router"]
        r[:] = 0.0
        r[:, :n] = rng.normal(0.0, 1.0, size=(len(r), n))
    t.update(stored({k: v for k, v in t.items() if k.endswith("router")}))
    for tok in range(doc["vocab"]):
        while True:
            x = stored({"x": rng.normal(0.0, 1.0, size=n)})["x"]
            gaps = []
            for i, top in routers:
                z = np.sort(t[f"l{i}.mlp.router"][:, :n] @ x)[::-1]
                gaps.append((z[top - 1] - z[top]) / np.abs(z).max() if top < len(z) else 1.0)
            if min(gaps) > 0.02:
                break
        t["embed"][tok, :n] = x
    return t


def weights(doc, seed=0):
    return stored(clear_choices(doc, synth.rufusun_tensors(doc, seed), seed))


def tokens(n, vocab, seed=0):
    return np.random.default_rng(seed).integers(0, vocab, size=n).tolist()


def error(got, want):
    """Root mean square difference over the vocabulary, mean taken off, per row, relative to the logits."""
    d = np.asarray(got, np.float64) - want
    d = d - d.mean(-1, keepdims=True)
    w = want - want.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / np.sqrt((w * w).mean())
