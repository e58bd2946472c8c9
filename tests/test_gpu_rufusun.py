"""Rufusun on the GPU against the plain evaluation in rufusun_ref.py: every mechanism alone, prompts, portions,
token-by-token decoding, batches, slots and pages used again, far keys, and generation."""
import io
import json

import numpy as np
import pytest

from dyninfer_b200 import synth
from dyninfer_b200.runtime import (DynInferError, GenerateConfig, ModelLoader, PerfConfig, SessionConfig, generate_greedy,
                                   run_perf)
import rufusun_cases as cases
import rufusun_ref as ref

pytestmark = pytest.mark.gpu

# relative to the logits: f32 sessions differ by rounding, serving ones by 16-bit operands and cache
LIMIT = {"f32": 1e-5, "serve": 1.5e-2}
KV = {"f32": "f32", "serve": "bf16"}


def load(tmp_path, doc, compute, seed=0, tensors=None, chunk=512, max_kv=512, kv=None):
    path = synth.write_rufusun(str(tmp_path / f"m{seed}{compute}"), doc, tensors=tensors or cases.weights(doc, seed))
    return ModelLoader().load(path, max_kv=max_kv, kv_dtype=kv or KV[compute], compute=compute, chunk_size=chunk)


def evaluate(doc, ids, seed=0, tensors=None):
    return ref.Model(doc, tensors or cases.weights(doc, seed)).forward(ids)


def assert_close(got, want, compute):
    e = cases.error(got, want)
    assert np.isfinite(got).all() and e.max() <= LIMIT[compute], (float(e.max()), int(e.argmax()))


def portions(n, sizes):
    out, i = [], 0
    while sum(out) < n:
        out.append(min(sizes[i % len(sizes)], n - sum(out)))
        i += 1
    return out


def run_portions(session, ids, cuts):
    session.reset()
    got, at = [], 0
    for n in cuts:
        got.append(session.extend(ids[at:at + n], range(n)))
        at += n
    return np.concatenate(got)


@pytest.mark.parametrize("compute", ["f32", "serve"])
@pytest.mark.parametrize("name", cases.MECHANISMS)
def test_each_mechanism_alone(native_lib, tmp_path, name, compute):
    """Whole prompt, one token at a time, and portions that end inside and across chunks of 64."""
    doc = cases.MECHANISMS[name]
    ids = cases.tokens(141, doc["vocab"], seed=5)
    want = evaluate(doc, ids)
    with load(tmp_path, doc, compute).create_session(SessionConfig(512)) as s:
        assert_close(run_portions(s, ids, [141]), want, compute)
        assert_close(run_portions(s, ids, [1] * 141), want, compute)
        assert_close(run_portions(s, ids, portions(141, [2, 3, 63, 1, 65, 2])), want, compute)
        assert_close(run_portions(s, ids, portions(141, [17, 4, 33])), want, compute)


@pytest.mark.parametrize("compute", ["f32", "serve"])
@pytest.mark.parametrize("doc", [cases.mixed(), cases.fast()], ids=["odd_sizes", "fast_paths"])
def test_whole_models_in_any_portions(native_lib, tmp_path, doc, compute):
    """Pages end at 256 tokens: the prompt passes the border in one piece, in pieces and token by token."""
    ids = cases.tokens(300, doc["vocab"], seed=6)
    want = evaluate(doc, ids)
    with load(tmp_path, doc, compute).create_session(SessionConfig(512)) as s:
        for cuts in ([300], [250] + [1] * 10 + [2] * 20, portions(300, [2]), portions(300, [64, 2, 65, 3]), [255, 2, 43],
                     [64, 64, 128, 44], [31, 33, 32, 70, 134]):
            assert_close(run_portions(s, ids, cuts), want, compute)


def test_chunk_size_smaller_than_the_prompt(native_lib, tmp_path):
    doc = cases.mixed()
    ids = cases.tokens(75, doc["vocab"], seed=7)
    want = evaluate(doc, ids)
    with load(tmp_path, doc, "f32", chunk=16).create_session(SessionConfig(512)) as s:
        assert_close(s.extend(ids, [0, 15, 16, 17, 74, 40]), want[[0, 15, 16, 17, 74, 40]], "f32")
        assert_close(s.prefill(ids).values[None], want[-1:], "f32")
        assert s.position() == 75 and s.prefill_argmax(ids) == int(want[-1].argmax())


@pytest.mark.parametrize("slots", [3, 7])
@pytest.mark.parametrize("compute", ["f32", "serve"])
@pytest.mark.parametrize("doc", [cases.mixed(), cases.fast()], ids=["odd_sizes", "fast_paths"])
def test_batches_of_unequal_requests_and_reused_slots(native_lib, tmp_path, doc, compute, slots):
    """Requests of different lengths decode together, in steps of a few rows and of more; a finished one's slot goes to
    another, and every one reads as if it were alone."""
    model = load(tmp_path, doc, compute)
    lengths = [1, 2, 70, 33, 129, 5, 18, 64, 3]
    seqs = [cases.tokens(n + 12, doc["vocab"], seed=20 + n) for n in lengths]
    want = [evaluate(doc, q) for q in seqs]
    with model.create_batched_session(SessionConfig(512, batch_size=slots)) as s:
        slot_of, at, waiting, order = {}, {}, list(range(len(lengths))), []
        while waiting or slot_of:
            for slot in range(slots):
                if slot not in slot_of.values() and waiting:
                    i = waiting.pop(0)
                    slot_of[i], at[i] = slot, lengths[i]
                    order.append((i, slot))
                    assert_close(s.extend_slot(slot, seqs[i][:lengths[i]], range(lengths[i]), restart=True),
                                 want[i][:lengths[i]], compute)
            _, lg = s.step({slot_of[i]: seqs[i][at[i]] for i in slot_of}, want_logits=True)
            for i in list(slot_of):
                assert_close(lg[slot_of[i]][None], want[i][at[i]:at[i] + 1], compute)
                at[i] += 1
                if at[i] == len(seqs[i]) or (i == 1 and at[i] == lengths[i] + 5):
                    del slot_of[i]
        assert len({slot for _, slot in order}) == slots and len(order) == len(lengths)


@pytest.mark.parametrize("slots", [20, 70])
@pytest.mark.parametrize("doc", [cases.mixed(), cases.fast()], ids=["odd_sizes", "fast_paths"])
def test_wide_decode_steps(native_lib, tmp_path, doc, slots):
    """Steps of as many rows as the many-row products take: every slot at a position of its own."""
    seqs = [cases.tokens(4 + i % 5, doc["vocab"], seed=60 + i) for i in range(slots)]
    want = [evaluate(doc, q) for q in seqs]
    with load(tmp_path, doc, "serve", chunk=128).create_batched_session(SessionConfig(256, batch_size=slots)) as s:
        for i, q in enumerate(seqs):
            s.extend_slot(i, q[:-3], restart=True)
        for back in (3, 2, 1):
            _, lg = s.step({i: q[len(q) - back] for i, q in enumerate(seqs)}, want_logits=True)
            for i, q in enumerate(seqs):
                assert_close(lg[i][None], want[i][len(q) - back][None], "serve")


def test_prompt_between_other_slots_decoding(native_lib, tmp_path):
    """A prompt's portions alternate with decode steps of other slots: neither disturbs the other."""
    doc = cases.fast()
    a, b = cases.tokens(80, doc["vocab"], 1), cases.tokens(150, doc["vocab"], 2)
    want_a, want_b = evaluate(doc, a), evaluate(doc, b)
    for compute in ("f32", "serve"):
        with load(tmp_path, doc, compute).create_batched_session(SessionConfig(512, batch_size=2)) as s:
            s.extend_slot(1, a[:70], restart=True)
            at = 0
            for n, i in ((64, 70), (2, 71), (3, 72), (81, 73)):
                assert_close(s.extend_slot(0, b[at:at + n], range(n), restart=at == 0), want_b[at:at + n], compute)
                at += n
                _, lg = s.step({1: a[i]}, want_logits=True)
                assert_close(lg[1][None], want_a[i:i + 1], compute)


@pytest.mark.parametrize("compute", ["f32", "serve"])
@pytest.mark.parametrize("name", ["moe_grouped", "moe_grouped_uneven", "moe"])
def test_all_tokens_at_the_same_experts(native_lib, tmp_path, name, compute):
    """The longest lists an expert can have, beside experts without any token; then one odd token among them."""
    doc = cases.MECHANISMS[name]
    ids = [7] * 300
    ids[150] = 8
    want = evaluate(doc, ids)
    with load(tmp_path, doc, compute).create_session(SessionConfig(512)) as s:
        for cuts in ([300], [140, 20] + portions(140, [5, 9, 70])):
            assert_close(run_portions(s, ids, cuts), want, compute)


@pytest.mark.parametrize("scale", [2.0 ** -14, 1.0])
def test_experts_of_any_range(native_lib, tmp_path, scale):
    """Experts whose weights would lose bits in f16 keep their own type; what they give is scaled back by the down matrix."""
    doc = cases.MECHANISMS["moe_grouped"]
    t = cases.weights(doc)
    for name in t:
        if ".mlp.e" in name or ".mlp.shared" in name:
            t[name] = t[name] * (scale if name.endswith(("gate", "up")) else 1.0 / scale ** 0.5)
    t = cases.stored(t)
    ids = cases.tokens(150, doc["vocab"], 16)
    want = evaluate(doc, ids, tensors=t)
    with load(tmp_path, doc, "serve", tensors=t).create_session(SessionConfig(256)) as s:
        assert_close(run_portions(s, ids, [100, 20, 7] + [1] * 23), want, "serve")


def far_key_model(dim, vdim, heads, kv_heads):
    """One attention layer whose queries of token 1 match the key of token 2 alone, by a wide margin, in the dims that
    are not rotated."""
    doc = cases.model([cases.attention(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, dims=8, scale=0.02, softcap=45.0)], width=64,
                      vocab=40, logit_scale=1.0)
    t = cases.weights(doc, 3)
    for name in ("l0.norm1", "final.norm"):
        t[name][:] = 0.0
    e = t["embed"] * 0.3
    e[:, :2] = 0.0
    e[1, 0] = e[2, 1] = 9.0
    e[1, 2:] *= 0.1
    q, k = t["l0.mix.q"] * 0.1, t["l0.mix.k"] * 0.1
    q[:, :2] = k[:, :2] = 0.0
    q[10::dim, 0] = 6.0
    k[10::dim, 1] = 6.0
    t.update({"embed": e, "l0.mix.q": q, "l0.mix.k": k, "l0.mix.q.b": t["l0.mix.q.b"] * 0.1, "l0.mix.k.b": t["l0.mix.k.b"] * 0.1})
    return doc, cases.stored(t)


@pytest.mark.parametrize("compute", ["f32", "serve"])
@pytest.mark.parametrize("shape", [(32, 16, 4, 2), (64, 128, 8, 1), (36, 20, 2, 2)], ids=["narrow", "wide", "odd"])
@pytest.mark.parametrize("at", [0, 1, 63, 64, 127, 255, 256, 257])
def test_far_key_is_found_from_everywhere(native_lib, tmp_path, at, shape, compute):
    """The key stands at the first tokens and around the borders of chunks and pages, and is asked for from a prompt, a
    portion and decoded tokens."""
    doc, t = far_key_model(*shape)
    rng = np.random.default_rng(at)
    ids = rng.integers(3, 40, size=420).tolist()
    ids[at] = 2
    for p in (at + 1, 300, 350, 399, 400, 419):
        ids[p] = 1
    want = evaluate(doc, ids, tensors=t)
    gone = list(ids)
    gone[at] = 3
    assert cases.error(evaluate(doc, gone, tensors=t), want)[[at + 1, 300, 399, 419]].min() > 0.1      # the key matters
    with load(tmp_path, doc, compute, tensors=t).create_session(SessionConfig(512)) as s:
        for cuts in ([420], [at + 1, 419 - at], [260, 40, 50] + [1] * 70):
            assert_close(run_portions(s, ids, cuts), want, compute)


@pytest.mark.parametrize("compute", ["f32", "serve"])
def test_state_reaches_far_back(native_lib, tmp_path, compute):
    """Slow decays: the first token still shows hundreds of tokens later, and must not be lost between portions; fast
    ones beside them leave nothing."""
    doc = cases.model([cases.delta(heads=4, kv_heads=2, dim=128, vdim=16, conv=2)], width=64, logit_scale=1.0)
    t = cases.weights(doc, 4)
    t["l0.mix.A_log"][:] = [-9.0, -11.0, 4.0, 2.0]
    t["l0.mix.b"] *= 0.1
    t["embed"][7] *= 3.0
    t = cases.stored(t)
    ids = [7] + [i if i != 7 else 8 for i in cases.tokens(399, doc["vocab"], 9)]
    want = evaluate(doc, ids, tensors=t)
    shown = cases.error(evaluate(doc, [9] + ids[1:], tensors=t), want)[399]
    assert shown > (2e-4 if compute == "f32" else 1e-5)
    with load(tmp_path, doc, compute, tensors=t).create_session(SessionConfig(512)) as s:
        for cuts in ([400], [1, 399], [2] * 10 + [380], [64] * 5 + [1] * 80):
            assert_close(run_portions(s, ids, cuts), want, compute)


def test_chunked_delta_rule_with_exact_inputs(native_lib, tmp_path):
    """Embeddings of +-1 are exact in every operand type, so a portion's rows differ from the evaluation by the chunks'
    arithmetic and the rounding of the output rows alone. Decays from none to complete, runs of one key, other keys between."""
    doc = dict(cases.MECHANISMS["delta_chunks"], logit_scale=1.0)
    t = cases.weights(doc, 5)
    t["embed"] = np.where(t["embed"] > 0, 1.0, -1.0)
    t["l0.norm1"][:] = 0.0
    t["l0.mix.A_log"][:] = [-8.0, -6.0, -4.0, 0.0, 2.0, 4.0]
    t = cases.stored(t)
    ids = [3] * 40 + cases.tokens(200, doc["vocab"], 10) + [5] * 60
    want = evaluate(doc, ids, tensors=t)
    with load(tmp_path, doc, "serve", tensors=t).create_session(SessionConfig(512)) as s:
        for cuts, limit in (([300], 8e-4), ([63, 65, 172], 8e-4), ([1] * 300, 1e-5)):
            e = cases.error(run_portions(s, ids, cuts), want)
            assert e.max() <= limit, (cuts[:3], float(e.max()))


def test_runs_of_a_loop_have_states_of_their_own(native_lib, tmp_path):
    ls = [cases.delta(mlp=cases.moe()), cases.attention(mlp=cases.dense(24)), cases.delta(heads=2)]
    doc = cases.model(ls, loop=cases.span(0, 2, 3))
    plain = cases.model(ls[:2] * 3 + ls[2:])
    t = cases.weights(doc, 8)
    full = {k: v for k, v in t.items() if not k.startswith("l2.")}
    for k, v in t.items():
        for i in (0, 1):
            for run in range(3):
                if k.startswith(f"l{i}."):
                    full[k.replace(f"l{i}.", f"l{i + 2 * run}.", 1)] = v
        if k.startswith("l2."):
            full["l6." + k[3:]] = v
    ids = cases.tokens(40, doc["vocab"], 3)
    got = []
    for i, (d, w) in enumerate(((doc, t), (plain, full))):
        with load(tmp_path, d, "f32", seed=i, tensors=w).create_session(SessionConfig(256)) as s:
            got.append(run_portions(s, ids, [30] + [1] * 10))
    assert np.array_equal(got[0], got[1])


def test_growing_the_cache_keeps_keys_values_and_states(native_lib, tmp_path):
    doc = cases.mixed()
    ids = cases.tokens(400, doc["vocab"], 11)
    want = evaluate(doc, ids)
    model = load(tmp_path, doc, "f32", max_kv=1024)
    with model.create_batched_session(SessionConfig(256, batch_size=2)) as s:
        for slot in (0, 1):
            assert_close(s.extend_slot(slot, ids[:200 + slot], range(200 + slot), restart=True), want[:200 + slot], "f32")
        assert s.kv_cache_metrics().page_count == 1
        s.config.max_sequence_length = 768
        for slot in (0, 1):
            assert_close(s.extend_slot(slot, ids[200 + slot:], range(200 - slot)), want[200 + slot:], "f32")
        m, c = s.kv_cache_metrics(), model.catalog.config
        assert m.page_count == 3 and m.allocated_bytes >= 2 * (768 * c["kv_elements_per_token"] * 4 + c["state_bytes_per_slot"])


@pytest.mark.parametrize("compute", ["f32", "serve"])
@pytest.mark.parametrize("doc", [cases.mixed(), cases.fast()], ids=["odd_sizes", "fast_paths"])
def test_long_decoding_on_the_device(native_lib, tmp_path, doc, compute):
    """Hundreds of greedy steps without the host: the logits after them are those of the whole sequence."""
    prompt = cases.tokens(9, doc["vocab"], 12)
    with load(tmp_path, doc, compute).create_session(SessionConfig(512)) as s:
        first = s.prefill_argmax(prompt)
        loop, ms = s.decode_loop(first, 330)
        ids = prompt + [first] + loop.tolist()
        assert ms > 0 and s.position() == 339
        got = s.extend(ids[-1:], [0])
        want = evaluate(doc, ids)
        assert_close(got, want[-1:], compute)
        assert s.prefill_argmax(prompt) == first and s.decode_loop(first, 330)[0].tolist() == loop.tolist()
        s.prefill_argmax(prompt)
        step = [first]
        for _ in range(20):
            step.append(s.decode_argmax(step[-1]))
        assert step[1:] == loop[:20].tolist()


def greedy(doc, prompt, n, penalty=1.0):
    m = ref.Model(doc, cases.weights(doc))
    lg, ids, margin = m.forward(prompt)[-1], list(prompt), []
    for _ in range(n):
        lg = lg.copy()
        for t in set(ids) if penalty != 1.0 else ():
            lg[t] = lg[t] * penalty if lg[t] < 0 else lg[t] / penalty
        top = np.sort(lg)[-2:]
        margin.append(top[1] - top[0])
        ids.append(int(lg.argmax()))
        lg = m.forward(ids[-1:])[0]
    return ids, min(margin)


@pytest.mark.parametrize("penalty", [1.0, 1.3])
def test_greedy_generation_through_the_entry_point(native_lib, tmp_path, penalty):
    doc = cases.mixed()
    prompt = cases.tokens(17, doc["vocab"], 13)
    want, margin = greedy(doc, prompt, 24, penalty)
    assert margin > 1e-3
    ids, stats = generate_greedy(load(tmp_path, doc, "f32"), prompt, GenerateConfig(max_new_tokens=24, repetition_penalty=penalty),
                                 SessionConfig(256))
    assert ids == want and stats.generated_tokens == 24
    rep = run_perf(load(tmp_path, doc, "serve", seed=1), PerfConfig(prefill_tokens=20, tg=4), SessionConfig(256))
    assert rep["decode"]["tps"] > 0 and rep["prefill"]["tps"] > 0


@pytest.mark.parametrize("count", [3, 6])
def test_batched_greedy_generation(native_lib, tmp_path, count):
    """Prompts generate together as they do alone, also past the row counts at which other kernels take over."""
    doc = cases.mixed()
    model = load(tmp_path, doc, "f32")
    prompts = [cases.tokens(n, doc["vocab"], 40 + n) for n in (3, 50, 18, 1, 33, 7)[:count]]
    alone = [generate_greedy(model, p, GenerateConfig(max_new_tokens=12), SessionConfig(256))[0] for p in prompts]
    with model.create_batched_session(SessionConfig(256, batch_size=count)) as s:
        feed = {i: s.prefill_slot(i, p) for i, p in enumerate(prompts)}
        ids = [list(p) for p in prompts]
        for _ in range(12):
            for i, t in feed.items():
                ids[i].append(t)
            feed = s.step(feed)
    assert ids == alone


def test_positions_cannot_be_rewound(native_lib, tmp_path):
    doc = cases.mixed()
    with load(tmp_path, doc, "f32").create_batched_session(SessionConfig(256, batch_size=2)) as s:
        s.extend_slot(0, [1, 2, 3], restart=True)
        s.positions[0] = 2
        with pytest.raises(DynInferError, match="slot 0 is at position 3"):
            s.extend_slot(0, [4])
        with pytest.raises(DynInferError, match="slot 0 is at position 3"):
            s.step({0: 4})
        s.positions[0] = 3
        s.extend_slot(0, [4, 5])
        with pytest.raises(DynInferError, match="exceeds session"):
            s.extend_slot(1, [1] * 257, restart=True)


@pytest.mark.parametrize("kv", ["f16", "f32"])
def test_other_caches(native_lib, tmp_path, kv):
    doc = cases.fast()
    ids = cases.tokens(130, doc["vocab"], 14)
    with load(tmp_path, doc, "serve", kv=kv).create_session(SessionConfig(256)) as s:
        assert_close(run_portions(s, ids, [100, 2] + [1] * 28), evaluate(doc, ids), "serve")


def test_trace_replay(native_lib, tmp_path, monkeypatch, capsys):
    from dyninfer_b200 import trace_run
    doc = cases.mixed()
    path = synth.write_rufusun(str(tmp_path / "m"), doc, tensors=cases.weights(doc))
    seqs = {n: cases.tokens(n, doc["vocab"], n) for n in (40, 23, 9)}
    steps, want = [], []
    for n, q in seqs.items():
        for lo, hi in ((0, n - 3), (n - 3, n - 1), (n - 1, n)):
            rows = list(range(0, hi - lo, 2))[::-1] if hi < n or n != 9 else []
            steps.append({"step": len(steps), "entries": [{"id": f"r{n}", "tokens": q[lo:hi], "want": rows}],
                          "end": [f"r{n}"] if hi == n else []})
            want.append(evaluate(doc, q)[[lo + r for r in rows]])
    out = tmp_path / "out"
    out.mkdir()
    monkeypatch.setattr("sys.stdin", io.StringIO("".join(json.dumps(s) + "\n" for s in steps)))
    assert trace_run.main(["--model", path, "--dtype", "float32", "--out", str(out), "--max-tokens", "40"]) == 0
    assert [ln for ln in capsys.readouterr().out.split("\n") if ln] == [f"done {i}" for i in range(9)]
    for i, w in enumerate(want):
        f = out / f"{i}.f32"
        assert f.exists() == bool(len(w))
        if len(w):
            assert_close(np.fromfile(f, "<f4").reshape(len(w), -1), w, "f32")
