"""The Vosotar design on the engine against the plain numpy statement of it (oracle/vosotar_oracle.py)."""
import io
import json
import os

import numpy as np
import pytest

from juno_b200 import synth
from vosotarutil import CONFIGS, L, Pair, check, decode_all, row_err

pytestmark = pytest.mark.gpu
DTYPES = ["f32", "default"]
NAMES = sorted(CONFIGS)


# ── whole prompts, decoding, portions ────────────────────────────────────────────────────────────
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_prompt_and_decoding_match_the_oracle(tmp_path, name, dtype):
    p = Pair(tmp_path, CONFIGS[name])
    toks = p.tokens(150)
    ref = p.oracle(toks)
    h = p.open(dtype)
    check(h.prefill_logits("a", toks, 0, range(len(toks))), ref, dtype, "prompt")
    check(decode_all(h, "b", toks), ref, dtype, "token by token")
    # a prompt, then decoding from its cache and state
    check(h.prefill_logits("c", toks[:101], 0, [0, 50, 100]), ref[[0, 50, 100]], dtype, "first part")
    check(decode_all(h, "c", toks[101:], 101), ref[101:], dtype, "decoded after a prompt")
    # the last position's logits of plain prefill, and the order of the wanted places
    check(h.prefill("d", toks, 0, want_logits=True), ref[-1], dtype, "last position")
    check(h.prefill_logits("e", toks, 0, [149, 3, 3, 60]), ref[[149, 3, 3, 60]], dtype, "places out of order")
    assert h.arch.architecture == "Vosotar" and h.arch.n_layers == len(p.cfg["layers"])
    h.release_gpu_resources()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["odd", "groups", "real", "wide"])
def test_portions_of_any_size(tmp_path, name, dtype):
    p = Pair(tmp_path, CONFIGS[name], seed=2)
    toks = p.tokens(230, 1)
    ref = p.oracle(toks)
    h = p.open(dtype, max_seqs=8)
    for k, sizes in enumerate([[2, 3, 2, 49, 50, 16, 17, 1, 1, 2, 64, 23], [230], [48, 49, 47, 2, 2, 2, 80], [1, 2, 1, 3, 100, 123], [2] * 115]):
        rid, pos = f"r{k}", 0
        for n in sizes:
            got = h.feed(rid, toks[pos:pos + n], range(n))
            check(got, ref[pos:pos + n], dtype, f"schedule {k}, portion at {pos}")
            pos += n
        assert pos == 230 and h.length(rid) == 230
    h.release_gpu_resources()
    # the engine's own cut of a long prompt
    h = p.open(dtype, max_rows=64)
    check(h.prefill_logits("a", toks, 0, range(230)), ref, dtype, "passes of 64 rows")
    h.release_gpu_resources()


def test_portions_do_not_change_the_result(tmp_path):
    """32-bit: any cut of a prompt gives the same logits up to rounding, also against the engine itself."""
    p = Pair(tmp_path, CONFIGS["odd"], seed=3)
    toks = p.tokens(97, 5)
    h = p.open("f32")
    whole = h.prefill_logits("a", toks, 0, range(97))
    parts = np.concatenate([h.feed("b", toks[i:i + 2], range(len(toks[i:i + 2]))) for i in range(0, 97, 2)])
    assert row_err(parts, whole).max() <= 1e-5
    h.release_gpu_resources()


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 9])
def test_first_tokens_of_a_sequence(tmp_path, taps):
    p = Pair(tmp_path, synth.vosotar_config(80, 77, [L(2, 16, 32, 24, 40, 48)], taps=taps), seed=taps)
    for dtype in DTYPES:
        h = p.open(dtype, max_seqs=40)
        for n in (1, 2, 3, 4, 5, 11):
            toks = p.tokens(n, 9)
            ref = p.oracle(toks)
            check(h.prefill_logits(f"p{n}", toks, 0, range(n)), ref, dtype, f"{n} tokens")
            check(decode_all(h, f"d{n}", toks), ref, dtype, f"{n} tokens, decoded")
        h.release_gpu_resources()


# ── batches, slots and pages ─────────────────────────────────────────────────────────────────────
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n", [2, 3, 8, 13])
def test_batches_of_unequal_requests(tmp_path, n, dtype):
    p = Pair(tmp_path, CONFIGS["groups"], seed=4)
    h = p.open(dtype, max_batch=16, max_seqs=16)
    lens = [(7 + 29 * i * i) % 171 + 1 for i in range(n)]
    seqs = [p.tokens(k + 6, 20 + i) for i, k in enumerate(lens)]
    refs = [p.oracle(s) for s in seqs]
    names = [f"r{i}" for i in range(n)]
    for r, s, k in zip(names, seqs, lens):
        h.feed(r, s[:k])
    for step in range(6):
        got = h.forward_batch(names, [[s[k + step]] for s, k in zip(seqs, lens)], [k + step for k in lens])
        for i in range(n):
            check(got[i], refs[i][lens[i] + step], dtype, f"request {i} of {n}, step {step}")
    h.release_gpu_resources()


@pytest.mark.parametrize("dtype", DTYPES)
def test_slots_and_pages_are_used_again(tmp_path, dtype):
    p = Pair(tmp_path, CONFIGS["odd"], seed=5)
    h = p.open(dtype, max_seqs=2, max_ctx=64)  # room for exactly two requests
    rng = np.random.default_rng(0)
    for k in range(7):
        n = int(rng.integers(3, 60))
        toks = p.tokens(n, 100 + k)
        ref = p.oracle(toks)
        rid = f"r{k}"
        cut = int(rng.integers(1, n))
        check(h.feed(rid, toks[:cut], range(cut)), ref[:cut], dtype, f"request {k}")
        check(decode_all(h, rid, toks[cut:], cut), ref[cut:], dtype, f"request {k}, decoded")
        if k:
            h.evict(f"r{k - 1}")
    # a request starts over at position 0 in its own slot
    toks = p.tokens(20, 999)
    check(h.prefill_logits("r6", toks, 0, range(20)), p.oracle(toks), dtype, "start over")
    h.release_gpu_resources()


def test_shared_prefix_has_its_own_state(tmp_path):
    p = Pair(tmp_path, CONFIGS["real"], seed=6)
    a, b = p.tokens(75, 1), p.tokens(75, 2)
    b[:50] = a[:50]
    ra, rb = p.oracle(a), p.oracle(b)
    for dtype in DTYPES:
        h = p.open(dtype, max_seqs=3)
        h.prefill("a", a[:50], 0)
        h.fork("a", "b", 50)
        for i in range(50, 75):  # both write into what was the shared page
            got = np.stack([h.forward_batch(["a"], [[a[i]]], [i])[0], h.forward_batch(["b"], [[b[i]]], [i])[0]])
            check(got, np.stack([ra[i], rb[i]]), dtype, f"position {i}")
        h.release_gpu_resources()


def test_rewind_within_and_beyond_the_state(tmp_path):
    p = Pair(tmp_path, CONFIGS["real"], seed=7)
    toks = p.tokens(60, 3)
    h = p.open("f32")
    h.prefill("a", toks, 0)
    new = toks[:50] + p.tokens(8, 4)
    check(decode_all(h, "a", new[50:], 50), p.oracle(new)[50:], "f32", "ten positions back")
    for pos in (5, 40):
        with pytest.raises(ValueError, match="start over at 0"):
            h.forward_batch(["a"], [[1]], [pos])
        with pytest.raises(ValueError, match="start over at 0"):
            h.prefill("a", [1, 2], pos)
        with pytest.raises(ValueError, match="start over at 0"):
            h.fork("a", f"f{pos}", pos)
    with pytest.raises(ValueError, match="gap"):
        h.forward_batch(["a"], [[1]], [61])
    h.release_gpu_resources()


# ── far keys, peaked scores ──────────────────────────────────────────────────────────────────────
def _peaked(tmp_path, taps=1, scale=6.0, **kw):
    """One layer whose scores are large: a key that matches the last query outweighs hundreds that do not."""
    def edit(t):
        t["l0.mix.uk"] *= 2.0
        t["l0.norm1b"] = np.float32(1.5)
        if taps > 1:
            t["l0.canon1"] *= 0.1
    return Pair(tmp_path, synth.vosotar_config(128, 64, [dict(L(4, 32, 32, 64, 64, 0), scale=scale / 32 ** 0.5)], taps=taps), edit=edit, **kw)


@pytest.mark.parametrize("dtype", DTYPES)
def test_one_far_key_among_hundreds(tmp_path, dtype):
    p = _peaked(tmp_path, seed=11)
    T = 300
    # the token that the query token's heads look at hardest, by the oracle: try each as the only different one
    fill, query = 1, 2
    base = [fill] * (T - 1) + [query]
    ref0 = p.oracle(base)[-1]
    effect = {}
    for tok in range(3, 24):
        s = list(base)
        s[100] = tok
        effect[tok] = row_err(p.oracle(s)[-1], ref0)[0]
    tok = max(effect, key=effect.get)
    assert effect[tok] > 0.2, "the test's weights hide the key"
    h = p.open(dtype, max_seqs=64)
    for k, pos in enumerate([0, 1, 15, 16, 17, 31, 32, 47, 48, 63, 64, 127, 128, 255, 256, 297, 298]):
        s = list(base)
        s[pos] = tok
        ref = p.oracle(s)[-1]
        assert row_err(ref, ref0)[0] > 0.15
        check(h.prefill_logits(f"p{k}", s, 0, [T - 1]), ref, dtype, f"key at {pos}, prompt")
        h.prefill(f"d{k}", s[:-1], 0)
        check(h.forward_batch([f"d{k}"], [[query]], [T - 1])[0], ref, dtype, f"key at {pos}, decoded")
        h.prefill(f"s{k}", s[:-3], 0)
        check(h.feed(f"s{k}", s[-3:], [2]), ref, dtype, f"key at {pos}, short portion")
        for r in "pds":
            h.evict(f"{r}{k}")
    h.release_gpu_resources()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(tmp_path, dtype):
    p = _peaked(tmp_path, taps=4, scale=2.0, seed=12)
    toks = p.tokens(420, 8)
    ref = p.oracle(toks)
    h = p.open(dtype)
    h.prefill("a", toks[:20], 0)
    check(decode_all(h, "a", toks[20:], 20), ref[20:], dtype, "four hundred decoded positions")
    h.release_gpu_resources()


def test_lengths_around_the_split_boundaries(tmp_path):
    """Every length near the tiles and splits of the decode attention, one step each."""
    p = _peaked(tmp_path, scale=3.0, seed=13)
    toks = p.tokens(200, 9)
    ref = p.oracle(toks)
    h = p.open("default", max_seqs=2)
    h.feed("a", toks[:2])
    for i in range(2, 200):
        check(h.forward_batch(["a"], [[toks[i]]], [i])[0], ref[i], "default", f"length {i + 1}")
    h.release_gpu_resources()


# ── each mechanism alone ─────────────────────────────────────────────────────────────────────────
def _neutral(t):
    """Everything round the named mechanism does as little as it can: gates open, no convolution, uniform attention."""
    for k in t:
        if k.endswith((".rg1", ".rg2", ".mix.g", ".canon1", ".mix.uq")):
            t[k] = np.zeros_like(t[k])
        elif k.endswith((".rg1.b", ".rg2.b")):
            t[k] = np.full_like(t[k], 8.0)
        elif "norm" in k:
            t[k] = np.ones_like(t[k])


def _mechanism(name):
    def edit(t):
        keep = {k: v.copy() for k, v in t.items()}
        _neutral(t)
        for k in t:
            back = {"convolution": k.endswith("canon1"), "mixer gate": ".rg1" in k, "feed-forward gate": ".rg2" in k,
                    "head gate": k.endswith("mix.g"), "scores": k.endswith("mix.uq"), "scalar norms": k.endswith(("norm1", "norm1b", "norm2", "norm2b", "embed.norm", "final.norm")),
                    "query latent norm": k.endswith(("dq.norm", "mix.uq")), "key/value latent norm": k.endswith("dkv.norm")}[name]
            if back:
                t[k] = keep[k] * (3.0 if name in ("scores", "head gate") else 1.0)
        if name == "query latent norm":
            t["l0.mix.dq.norm"] = t["l0.mix.dq.norm"] * 3.0
    return edit


@pytest.mark.parametrize("name", ["convolution", "mixer gate", "feed-forward gate", "head gate", "scores", "scalar norms", "query latent norm",
                                  "key/value latent norm"])
def test_each_mechanism_alone(tmp_path, name):
    cfg = synth.vosotar_config(112, 101, [L(3, 16, 24, 40, 48, 72)], taps=4, eps=1e-3)
    p, plain = Pair(tmp_path, cfg, 21, _mechanism(name)), Pair(tmp_path, cfg, 21, _neutral)
    toks = p.tokens(60, 3)
    ref = p.oracle(toks)
    assert row_err(ref, plain.oracle(toks)).max() > 0.1, "the mechanism does not show"
    for dtype in DTYPES:
        h = p.open(dtype)
        check(h.prefill_logits("a", toks, 0, range(60)), ref, dtype, f"{name}, prompt")
        check(decode_all(h, "b", toks), ref, dtype, f"{name}, decoded")
        h.release_gpu_resources()


def test_shared_weights_keep_their_own_cache(tmp_path):
    one = L(2, 16, 16, 32, 32, 48)
    p = Pair(tmp_path, synth.vosotar_config(64, 70, [one, L(3, 16, 32, 16, 48, 0), dict(one, weights_of=0), dict(L(3, 16, 32, 16, 48, 0), weights_of=1), dict(one, weights_of=2)]), 31)
    toks = p.tokens(70, 1)
    ref = p.oracle(toks)
    for dtype in DTYPES:
        h = p.open(dtype)
        check(h.prefill_logits("a", toks, 0, range(70)), ref, dtype)
        check(decode_all(h, "b", toks), ref, dtype)
        h.release_gpu_resources()


def test_residual_stream_after_the_last_layer(tmp_path):
    from oracle import vosotar_oracle as vo
    p = Pair(tmp_path, CONFIGS["odd"], 32)
    toks, streams = p.tokens(64, 1), []
    vo.forward(toks, p.cfg, p.w, streams)
    h = p.open("f32")
    h.prefill("a", toks, 0)
    assert np.abs(h.last_hidden(64) - streams[-1]).max() <= 1e-4
    h.release_gpu_resources()
    h = p.open("default")  # the decode step's residual rows alternate between two buffers
    h.prefill("a", toks[:-1], 0)
    for _ in range(3):  # eager, captured, replayed
        h.forward_batch(["a"], [[toks[-1]]], [63])
        assert np.abs(h.last_hidden(1)[0] - streams[-1][-1]).max() <= 0.05 * np.abs(streams[-1][-1]).max()
    h.release_gpu_resources()


# ── generation, the trace command, refusals ──────────────────────────────────────────────────────
@pytest.mark.parametrize("chunked", [False, True])
def test_greedy_generation(tmp_path, chunked):
    from juno_b200.handler import B200InferencePipeline, generate_greedy
    from oracle import vosotar_oracle as vo
    p = Pair(tmp_path, CONFIGS["real"], 41)
    prompt = p.tokens(30, 1)
    for dtype in DTYPES:
        h = p.open(dtype)
        got = generate_greedy(B200InferencePipeline(h), "g", prompt, 24, chunked_prefill=chunked)
        ref, margins = vo.generate_greedy(prompt, 24, p.cfg, p.w)
        scale = np.abs(p.oracle(prompt)).max()
        for i, (x, y) in enumerate(zip(got, ref)):
            if margins[i] < (1e-4 if dtype == "f32" else 0.1) * scale:
                break  # the two best are too close to call: from here the continuations may differ
            assert x == y, f"token {i}"
        # every generated token is the argmax of the step that produced it
        logits = h.prefill_logits("v", prompt + got[:-1], 0, range(29, 29 + 24))
        best = logits.max(-1)
        assert all(best[i] - logits[i, t] <= (1e-4 if dtype == "f32" else 0.1) * scale for i, t in enumerate(got))
        h.release_gpu_resources()


def test_generation_in_batches_equals_generation_alone(tmp_path):
    p = Pair(tmp_path, CONFIGS["real"], 42)
    h = p.open("f32", max_batch=4, max_seqs=8)
    prompts = [p.tokens(5 + 9 * i, i) for i in range(4)]
    alone = []
    for i, s in enumerate(prompts):
        h.prefill(f"a{i}", s[:-1], 0)
        alone.append(h.decode_greedy([f"a{i}"], [s[-1]], [len(s) - 1], 12)[:, 0].tolist())
        h.evict(f"a{i}")
        h.prefill(f"b{i}", s[:-1], 0)
    got = h.decode_greedy([f"b{i}" for i in range(4)], [s[-1] for s in prompts], [len(s) - 1 for s in prompts], 12)
    assert got.T.tolist() == alone
    h.release_gpu_resources()


def test_generation_from_the_command_line(tmp_path, capsys):
    from juno_b200 import generate
    p = Pair(tmp_path, CONFIGS["odd"], 43)
    prompts = [p.tokens(12, 1), p.tokens(3, 2)]
    arg = [",".join(map(str, s)) for s in prompts]
    lines = []
    for args in (["--ids", arg[0]], ["--ids", arg[0], "--token-by-token"], ["--ids", arg[1]], ["--ids", arg[0], "--ids", arg[1]]):
        assert generate.main([p.dir, "--steps", "9", "--dtype", "f32", *args]) == 0
        lines.append(capsys.readouterr().out.split())
    assert lines[0] == lines[1] and lines[3] == lines[0] + lines[2] and len(lines[0][0].split(",")) == 9


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay(tmp_path, dtype):
    from juno_b200 import trace
    p = Pair(tmp_path, CONFIGS["odd"], 51)
    a, b = p.tokens(40, 1), p.tokens(9, 2)
    steps = [([("a", a[:30], [0, 29])], []), ([("a", a[30:31], [0])], []), ([("a", a[31:33], [])], []), ([("a", a[33:], [6, 1])], ["a"]),
             ([("b", b[:1], [0])], []), ([("b", b[1:], list(range(8)))], ["b"])]
    lines = [json.dumps({"step": i, "entries": [{"id": r, "tokens": t, "want": w} for r, t, w in e], "end": end}) + "\n" for i, (e, end) in enumerate(steps)]
    h, said = p.open(dtype, max_seqs=1), []
    trace.run(h, io.StringIO("".join(lines)), str(tmp_path), said.append)
    h.release_gpu_resources()
    assert said == [f"done {i}" for i in range(6)]
    ra, rb = p.oracle(a), p.oracle(b)
    want = {0: ra[[0, 29]], 1: ra[[30]], 3: ra[[39, 34]], 4: rb[[0]], 5: rb[1:]}
    for i in range(6):
        f = tmp_path / f"{i}.f32"
        assert f.exists() == (i in want)
        if i in want:
            check(np.fromfile(f, "<f4").reshape(want[i].shape), want[i], dtype, f"step {i}")


def test_what_the_registry_refuses(tmp_path):
    from juno_b200._lib import JunoError
    from juno_b200.safetensors_file import write_model_folder
    from vosotarutil import build
    cfg = synth.vosotar_config(64, 70, [L(2, 16, 16, 32, 32, 48)])
    t, _ = build(cfg)

    def opened(c, tensors):
        from juno_b200.handler import B200TransformerHandler
        d = write_model_folder(str(tmp_path / f"x{len(os.listdir(tmp_path))}"), c, tensors)
        B200TransformerHandler.open(d).release_gpu_resources()

    opened(cfg, t)
    with pytest.raises(JunoError, match="not in the model registry"):
        opened(dict(cfg, architecture="Nothing"), t)
    with pytest.raises(ValueError, match="l0.mix.uk is missing"):
        opened(cfg, {k: v for k, v in t.items() if k != "l0.mix.uk"})
    with pytest.raises(ValueError, match="has shape"):
        opened(cfg, dict(t, head=t["head"][:, :32]))
    bad = json.loads(json.dumps(cfg))
    bad["layers"][0]["type"] = "window_attention"
    with pytest.raises(JunoError, match="not part of this design"):
        opened(bad, t)
    bad = json.loads(json.dumps(cfg))
    bad["layers"][0]["weights_of"] = 0
    with pytest.raises(ValueError, match="never reaches"):
        opened(bad, t)
    bad = json.loads(json.dumps(cfg))
    del bad["layers"][0]["mixer"]["q_rank"]
    with pytest.raises(ValueError, match="q_rank"):
        opened(bad, t)
    with pytest.raises(ValueError, match="cannot open"):
        from juno_b200.handler import B200TransformerHandler
        B200TransformerHandler.open(str(tmp_path / "missing"))


def test_gguf_files_open_through_the_registry(tmp_path):
    from juno_b200.gguf_file import write_model
    from juno_b200.handler import B200TransformerHandler
    from modelutil import TINY
    tensors = list(synth.random_model(TINY, 3, norm="random"))
    write_model(tmp_path / "m.gguf", TINY, tensors)
    h = B200TransformerHandler.open(str(tmp_path / "m.gguf"), max_batch=8, max_ctx=64)
    g = B200TransformerHandler(TINY, h.ctx, max_batch=8, max_seqs=8, max_ctx=64).load(tensors)
    toks = np.random.default_rng(0).integers(0, TINY.vocab, 12).tolist()
    assert h.arch.architecture == "llama" and h.arch.vocab == TINY.vocab
    assert np.array_equal(h.prefill("a", toks, 0, want_logits=True), g.prefill("a", toks, 0, want_logits=True))
    got = h.prefill_logits("b", toks, 0, [11, 0, 5])
    assert np.array_equal(got[0], h.prefill("c", toks, 0, want_logits=True)) and np.isfinite(got).all()
    h.release_gpu_resources()
    g.release_gpu_resources()
