"""Small Zupudra configurations for the tests: sizes that differ from each other in every model, odd ones that
no fast kernel takes, and ones that reach the tensor-core and fused paths."""
import numpy as np

from dyninfer_b200 import synth


def retention(heads=3, dim=20, vdim=28, dims=12, base=5000.0, decay=None, mlp=None):
    decay = decay or [float(1.0 - 0.3 * 0.31 ** i) for i in range(heads)]
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay,
                                           "rot": {"dims": dims, "base": base}}, "mlp": mlp}


def rglru(width=60, blocks=5, conv=3, mlp=None):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}, "mlp": mlp}


def latent(heads=3, dim=20, vdim=12, kv_rank=36, scale=0.9, mlp=None):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank,
                                                  "scale": scale}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def shared(layers, j):
    return dict(layers[j], weights_of=j)


def model(layers, width=44, vocab=101, eps=1e-5):
    return {"layers": layers, "width": width, "vocab": vocab, "norm": {"eps": eps}}


def mixed():
    """Every mixer with and without a feed-forward, shared tensors, no size a multiple of the others."""
    ls = [latent(heads=5, dim=12, vdim=20, kv_rank=28, mlp=dense(52)), retention(mlp=dense(36)), rglru(),
          retention(heads=2, dim=36, vdim=8, dims=36, base=300.0), rglru(width=48, blocks=3, conv=5, mlp=dense(40)), latent()]
    return model(ls + [shared(ls, 1), shared(ls, 4), shared(ls, 0)])


def fast():
    """Widths that the tensor-core GEMM, the streaming GEMV and the 128-wide prefill attention take."""
    ls = [retention(heads=2, dim=64, vdim=128, dims=32, base=10000.0), rglru(width=320, blocks=2, conv=4, mlp=dense(192)),
          latent(heads=3, dim=128, vdim=64, kv_rank=192, scale=0.6, mlp=dense(256))]
    return model(ls + [shared(ls, 0), shared(ls, 2)], width=512, vocab=384, eps=1e-6)


MECHANISMS = {
    "retention": model([retention()]),
    "retention_full_rotation": model([retention(heads=1, dim=96, vdim=144, dims=96, base=1e5, decay=[0.9997])]),
    "retention_no_memory_and_no_decay": model([retention(heads=2, dim=8, vdim=36, dims=4, decay=[1.0, 0.0])]),
    "retention_wide_values": model([retention(heads=1, dim=16, vdim=300, dims=8, decay=[0.97])]),
    "retention_feed_forward": model([retention(heads=4, dim=16, vdim=16, dims=16, mlp=dense(60))], width=64),
    "rglru": model([rglru()]),
    "rglru_one_block": model([rglru(width=40, blocks=1, conv=7)]),
    "rglru_one_tap": model([rglru(width=36, blocks=4, conv=1)]),
    "rglru_single_channel_blocks": model([rglru(width=18, blocks=18, conv=2, mlp=dense(20))]),
    "latent": model([latent()]),
    "latent_wide_rank": model([latent(heads=9, dim=40, vdim=24, kv_rank=140, scale=0.4)]),
    "latent_rank_one": model([latent(heads=2, dim=4, vdim=8, kv_rank=1, scale=2.0, mlp=dense(24))]),
    "latent_wide_heads": model([latent(heads=2, dim=132, vdim=136, kv_rank=64, scale=0.5)], width=64),
    "odd_widths": model([retention(heads=1, dim=7, vdim=9, dims=6), rglru(width=15, blocks=3, conv=4), latent(1, 5, 11, 13, mlp=dense(17))],
                        width=33, vocab=67),
}


def stored(tensors):
    """Weights as a checkpoint holds them (bf16 values), in float32."""
    return {k: synth.bf16_bits_to_f32(synth.f32_to_bf16_bits(v)) for k, v in tensors.items()}


def weights(doc, seed=0):
    return stored(synth.zupudra_tensors(doc, seed))


def tokens(n, vocab, seed=0):
    return np.random.default_rng(seed).integers(0, vocab, size=n).tolist()


def error(got, want):
    """Root mean square difference over the vocabulary, mean taken off, per row, relative to the logits."""
    d = np.asarray(got, np.float64) - want
    d = d - d.mean(-1, keepdims=True)
    w = want - want.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / np.sqrt((w * w).mean())
