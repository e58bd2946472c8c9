"""Zupudra on CPU: configuration and tensor names, coverage, and that the plain evaluation the GPU tests compare
with would show the faults they look for."""
import json

import numpy as np
import pytest

from dyninfer_b200 import checkpoint as ck, registry as reg, synth, zupudra
from dyninfer_b200.runtime import ModelLoader, DynInferError
import zupudra_cases as cases
import zupudra_ref as ref


def test_catalog_reads_every_size_and_name(tmp_path):
    doc = cases.mixed()
    cat = ck.open_catalog(synth.write_zupudra(str(tmp_path / "m"), doc, seed=1))
    c = cat.config
    assert (c["layers"], c["hidden"], c["vocab"], c["tied"]) == (9, 44, 101, True) and c["eps"] == 1e-5
    assert [m["tensors"] for m in c["mixers"]] == [0, 1, 2, 3, 4, 5, 1, 4, 0]
    assert c["mixers"][3] == {"type": "retention", "tensors": 3, "ff": 0, "heads": 2, "dim": 36, "vdim": 8, "rot_dims": 36,
                              "rot_base": 300.0, "decay": doc["layers"][3]["mixer"]["decay"]}
    assert c["mixers"][7]["taps"] == 5 and c["mixers"][5]["rank"] == 36 and c["mixers"][5]["ff"] == 0
    assert c["kv_elements_per_token"] == 28 + 36 + 28                      # one latent per latent-attention layer
    assert c["state_bytes_per_slot"] == 4 * (2 * 3 * 20 * 28 + 60 * 4 + 2 * 36 * 8 + 2 * 48 * 6)
    assert set(cat.parameters) == set(zupudra.tensor_names(doc).values())
    assert cat.parameters["blk.2.rec_a_gate.weight"].shape == (5, 12, 12)
    assert not any(p.startswith(("blk.6.", "blk.7.", "blk.8.")) for p in cat.parameters)
    plan = ck.build_runtime_provider_plan(cat)
    assert len(plan.parameters) == len(synth.zupudra_shapes(doc))


def test_shared_layers_resolve_through_chains_and_refuse_circles():
    layers = [cases.rglru(), dict(cases.rglru(), weights_of=0), dict(cases.rglru(), weights_of=1)]
    assert [zupudra.owner(layers, i) for i in range(3)] == [0, 0, 0]
    with pytest.raises(ValueError, match="circle"):
        zupudra.owner([dict(cases.rglru(), weights_of=1), dict(cases.rglru(), weights_of=0)], 0)
    with pytest.raises(ValueError, match="names layer"):
        zupudra.owner([dict(cases.rglru(), weights_of=5)], 0)


def test_bad_checkpoints_are_refused(tmp_path):
    doc = cases.model([cases.retention()])
    path = synth.write_zupudra(str(tmp_path / "m"), doc)
    t = cases.weights(doc)
    del t["l0.mix.g"]
    with pytest.raises(ck.CheckpointError, match="lacks tensor l0.mix.g"):
        ck.open_catalog(synth.write_zupudra(str(tmp_path / "missing"), doc, tensors=t))
    for change, match in ((("layers", [dict(doc["layers"][0], type="conv")]), "unknown mixer"), (("width", None), "config.json")):
        with open(f"{path}/config.json", "w") as f:
            json.dump(dict(doc, architecture="Zupudra", **{change[0]: change[1]}), f)
        with pytest.raises(ck.CheckpointError, match=match):
            ck.open_catalog(path)
    with open(f"{path}/config.json", "w") as f:
        json.dump(dict(doc, architecture="Other"), f)
    with pytest.raises(ck.CheckpointError, match="unknown architecture `Other`"):
        ck.open_catalog(path)


def test_every_operation_is_covered_in_both_modes(tmp_path):
    loader = ModelLoader()
    cat = loader.bind(synth.write_zupudra(str(tmp_path / "m"), cases.mixed()))
    rep = loader.kernel_coverage(cat, loader.resolve_target("cuda")[0])
    assert not rep.missing
    ids = {k for _, _, k in rep.selected}
    assert {"retention.cuda_sm100.f32", "rglru.cuda_sm100.f32", "attention.latent.cuda_sm100", "short_conv.cuda_sm100.f32",
            "plain.bf16.matmul.cuda_sm100", "plain.bf16.lm_head.cuda_sm100"} <= ids
    other = loader.kernel_coverage(cat, reg.TargetProfile.llvm_cpu_host())       # never another target's kernels
    assert {op for op, _, _ in other.missing} >= {"blk.1.retention", "blk.2.recurrence", "blk.0.attention"}


def test_tensor_parallel_is_refused(tmp_path):
    path = synth.write_zupudra(str(tmp_path / "m"), cases.mixed())
    with pytest.raises(DynInferError, match="tensor parallelism"):
        ModelLoader().load(path, tp=(0, 2))


# ---- the plain evaluation ------------------------------------------------------------------------

def test_retention_state_is_the_decayed_sum():
    rng = np.random.default_rng(0)
    k, v, q = rng.normal(size=(7, 4)), rng.normal(size=(7, 5)), rng.normal(size=4)
    S = np.zeros((4, 5))
    for t in range(7):
        S = ref.retention_state(S, k[t], v[t], 0.9)
    want = sum(0.9 ** (6 - t) * (q @ k[t]) * v[t] for t in range(7))
    assert np.allclose(S.T @ q, want)


def test_rotation_keeps_relative_positions_and_passes_the_rest():
    rng = np.random.default_rng(1)
    a, b = rng.normal(size=10), rng.normal(size=10)
    at = lambda p, r: ref.rotate_half(a, p, 6, 50.0) @ ref.rotate_half(b, r, 6, 50.0)   # noqa: E731
    assert np.isclose(at(3, 1), at(12, 10)) and not np.isclose(at(3, 1), at(3, 2))
    assert np.array_equal(ref.rotate_half(a, 9, 6, 50.0)[6:], a[6:])


def test_convolution_is_causal_with_the_last_tap_on_the_current_token():
    x = np.arange(12.0).reshape(6, 2)
    w = np.array([[1.0, 10.0, 100.0], [2.0, 20.0, 200.0]])
    tail, out = np.zeros((2, 2)), []
    for row in x:
        out.append(ref.causal_conv(row, tail, w, np.array([0.5, 0.25])))
    assert np.allclose(out[0], x[0] * w[:, 2] + [0.5, 0.25])
    assert np.allclose(out[4], x[2] * w[:, 0] + x[3] * w[:, 1] + x[4] * w[:, 2] + [0.5, 0.25])


def test_latent_scores_equal_the_absorbed_form():
    rng = np.random.default_rng(2)
    uk, q, c = rng.normal(size=(6, 9)), rng.normal(size=6), rng.normal(size=(4, 9))
    assert np.allclose((c @ uk.T) @ q, c @ (uk.T @ q))


FAULTS = {
    "some tokens missing in the state": ("retention_state", lambda S, k, v, decay: decay * S + np.outer(k, v) * (k[0] > 0)),
    "decay of two tokens": ("retention_state", lambda S, k, v, decay: decay * decay * S + np.outer(k, v)),
    "rotation one position off": ("rotate_half", lambda v, p, d, b, f=ref.rotate_half: f(v, p + (p > 3), d, b)),
    "convolution tail dropped": ("causal_conv", lambda x, tail, w, b, f=ref.causal_conv: f(x, np.zeros_like(tail), w, b)),
    "no input scaling": ("rglru_state", lambda S, u, r, i, lam: np.exp(-8 * r * ref.softplus(lam)) * S + i * u),
    "newest key hidden": ("softmax", lambda s, f=ref.softmax: f(np.append(s[:-1], -1e30)) if len(s) > 1 else f(s)),
    "oldest key hidden": ("softmax", lambda s, f=ref.softmax: f(np.append(-1e30, s[1:])) if len(s) > 1 else f(s)),
    "norm by the mean magnitude": ("rms", lambda x, eps: x / (np.abs(x).mean() + eps)),
}


@pytest.mark.parametrize("fault", FAULTS)
def test_faults_show_in_the_logits(fault, monkeypatch):
    """Each planted fault moves the logits by far more than the tolerances of the GPU tests."""
    doc = cases.mixed()
    ids = cases.tokens(12, doc["vocab"])
    want = ref.Model(doc, cases.weights(doc)).forward(ids)
    name, wrong = FAULTS[fault]
    monkeypatch.setattr(ref, name, wrong)
    assert cases.error(ref.Model(doc, cases.weights(doc)).forward(ids), want)[4:].max() > 0.1
