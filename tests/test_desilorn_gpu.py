"""The Desilorn design on the engine against the plain numpy statement of it (oracle/desilorn_oracle.py)."""
import io
import json
import os

import numpy as np
import pytest

from desilornutil import CONFIGS, C, Pair, W, build, check, decode_all, row_err
from juno_b200 import synth
from oracle import desilorn_oracle as do

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
    # a prompt, then decoding from its cache
    check(h.prefill_logits("c", toks[:101], 0, [0, 50, 100]), ref[[0, 50, 100]], dtype, "first part")
    check(decode_all(h, "c", toks[101:], 101), ref[101:], dtype, "decoded after a prompt")
    # the last position's logits of plain prefill, and the order of the wanted places
    check(h.prefill("d", toks, 0, want_logits=True), ref[-1], dtype, "last position")
    check(h.prefill_logits("e", toks, 0, [149, 3, 3, 60]), ref[[149, 3, 3, 60]], dtype, "places out of order")
    assert h.arch.architecture == "Desilorn" and h.arch.n_layers == len(do.layer_runs(p.cfg))
    h.release_gpu_resources()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["odd", "groups", "long", "wide", "d256", "real"])
def test_portions_of_any_size(tmp_path, name, dtype):
    p = Pair(tmp_path, CONFIGS[name], seed=2)
    toks = p.tokens(400, 1)
    ref = p.oracle(toks)
    h = p.open(dtype, max_seqs=8)
    for k, sizes in enumerate([[2, 3, 2, 49, 50, 16, 17, 1, 1, 2, 64, 23, 170], [400], [48, 49, 47, 2, 2, 2, 80, 15, 155], [1, 2, 1, 3, 100, 123, 170], [2] * 60 + [18, 17] * 8]):
        rid, pos = f"r{k}", 0
        for n in sizes:
            got = h.feed(rid, toks[pos:pos + n], range(n))
            check(got, ref[pos:pos + n], dtype, f"schedule {k}, portion at {pos}")
            pos += n
        assert pos == 400 and h.length(rid) == 400
    h.release_gpu_resources()
    # the engine's own cut of a long prompt
    h = p.open(dtype, max_rows=64)
    check(h.prefill_logits("a", toks, 0, range(400)), ref, dtype, "passes of 64 rows")
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


@pytest.mark.parametrize("streams", [1, 2, 4, 7])
def test_first_tokens_of_a_sequence(tmp_path, streams):
    cfg = synth.desilorn_config(80, 77, [W(2, 1, 16, 32, 3, 48, (0.5, 2)), C(2, 2, 24, 16, 4, 40, (30.0, 8))], streams=streams)
    p = Pair(tmp_path, cfg, seed=streams)
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
@pytest.mark.parametrize("name", ["groups", "real"])
def test_batches_of_unequal_requests(tmp_path, name, n, dtype):
    p = Pair(tmp_path, CONFIGS[name], seed=4)
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
    # a request starts over at position 0 in its own slot, and is rewound
    toks = p.tokens(20, 999)
    ref = p.oracle(toks)
    check(h.prefill_logits("r6", toks, 0, range(20)), ref, dtype, "start over")
    check(decode_all(h, "r6", toks[3:], 3), ref[3:], dtype, "rewound")
    h.release_gpu_resources()


def test_shared_prefix(tmp_path):
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


# ── one key that stands out: edges of windows and chunks, far keys, page borders ─────────────────
FILL, QUERY = 1, 2


def _one_layer(tmp_path, layer, seed):
    """One layer whose scores are large: a key that matches the last query outweighs those that do not."""
    def edit(t):
        t["l0.mix.v"] *= 2.0
        t["l0.mix.v.b"] *= 0.0
        t["l0.hc1.out"] = np.full_like(t["l0.hc1.out"], 2.0)
        if "l0.mix.sink" in t:
            t["l0.mix.sink"] = np.full_like(t["l0.mix.sink"], -2.0)
    return Pair(tmp_path, synth.desilorn_config(128, 64, [layer], streams=2), seed, edit)


def _sequence(p, pos, tok, last):
    s = [FILL] * last + [QUERY]
    s[pos] = tok
    return s


def _strongest(p, pos, last):
    """The token that changes the last position's logits most when it stands at `pos`, and by how much."""
    base = p.oracle(_sequence(p, last, QUERY, last))[-1]
    effect = {tok: row_err(p.oracle(_sequence(p, pos, tok, last))[-1], base)[0] for tok in range(3, 30)}
    tok = max(effect, key=effect.get)
    return tok, effect[tok], base


def _last_logits(h, s, k):
    """The last position's logits by every route that reads the cache in another way."""
    T = len(s)
    out = {"prompt": h.prefill_logits(f"p{k}", s, 0, [T - 1])[0]}
    if T > 1:
        h.feed(f"d{k}", s[:-1])
        out["decoded"] = h.feed(f"d{k}", s[-1:], [0])[0]
    if T > 3:
        h.feed(f"s{k}", s[:-3])
        out["short portion"] = h.feed(f"s{k}", s[-3:], [2])[0]
    if T > 24:
        h.feed(f"l{k}", s[:-23])
        out["long portion"] = h.feed(f"l{k}", s[-23:], [22])[0]
    for r in "pdsl":
        h.evict(f"{r}{k}")
    return out


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size", [2, 16, 17, 37, 64, 100])
def test_edges_of_the_window(tmp_path, size, dtype):
    p = _one_layer(tmp_path, W(4, 2, 32, 32, size, 0, (0.3, 40), scale=0.8), seed=size)
    h = p.open(dtype, max_seqs=8)
    for k, last in enumerate(sorted({size - 1, size, size + 1, size + 14, size + 15, 2 * size + 3, 127, 128, 150})):
        first = last - size + 1  # the first position the last one sees
        if first < 0:
            continue
        tok, effect, base = _strongest(p, first, last)
        assert effect > 0.1, "the test's weights hide the key"
        cases = [(first, "just inside")] + ([(first - 1, "just outside")] if first > 0 else [])
        for pos, what in cases:
            s = _sequence(p, pos, tok, last)
            ref = p.oracle(s)[-1]
            assert (row_err(ref, base)[0] > 0.1) == (what == "just inside")
            for route, got in _last_logits(h, s, k).items():
                check(got, ref, dtype, f"window {size}, query {last}, key {what}, {route}")
    h.release_gpu_resources()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size", [2, 16, 31, 64, 75])
def test_edges_of_the_chunk(tmp_path, size, dtype):
    p = _one_layer(tmp_path, C(4, 2, 32, 32, size, 0, (1e6, 8), scale=1.0), seed=100 + size)
    h = p.open(dtype, max_seqs=8)
    for k, last in enumerate(sorted({size, size + 1, 2 * size - 1, 2 * size, 2 * size + 1, 3 * size - 1, 3 * size, 3 * size + 1})):
        first = last // size * size
        if first < last:
            tok, effect, base = _strongest(p, first, last)
            assert effect > 0.1, "the test's weights hide the key"
        else:
            tok, _, base = _strongest(p, last - 1, last)
        for pos, what in [(first, "first of the chunk"), (first - 1, "last of the chunk before")]:
            if pos == last:
                continue
            s = _sequence(p, pos, tok, last)
            ref = p.oracle(s)[-1]
            assert (row_err(ref, base)[0] > 0.1) == (pos >= first)
            for route, got in _last_logits(h, s, k).items():
                check(got, ref, dtype, f"chunk {size}, query {last}, key {what}, {route}")
    h.release_gpu_resources()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["window", "chunk"])
def test_one_far_key_among_hundreds(tmp_path, kind, dtype):
    """Spans of hundreds of positions (several splits of the decode attention); the key stands at page borders."""
    T = 300
    layer = W(2, 1, 64, 32, 400, 0, (0.2, 100), scale=0.7) if kind == "window" else C(2, 1, 64, 32, 512, 0, (1e7, 8), scale=1.3)
    p = _one_layer(tmp_path, layer, seed=11)
    tok, effect, base = _strongest(p, 100, T - 1)
    assert effect > 0.1, "the test's weights hide the key"
    h = p.open(dtype, max_seqs=8)
    for k, pos in enumerate([0, 1, 15, 16, 17, 31, 32, 47, 48, 63, 64, 127, 128, 255, 256, 297, 298]):
        s = _sequence(p, pos, tok, T - 1)
        ref = p.oracle(s)[-1]
        assert row_err(ref, base)[0] > 0.05
        for route, got in _last_logits(h, s, k).items():
            check(got, ref, dtype, f"key at {pos}, {route}")
    h.release_gpu_resources()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["long", "odd"])
def test_long_decoding(tmp_path, name, dtype):
    p = Pair(tmp_path, CONFIGS[name], seed=12)
    toks = p.tokens(420, 8)
    ref = p.oracle(toks)
    h = p.open(dtype)
    h.prefill("a", toks[:20], 0)
    check(decode_all(h, "a", toks[20:], 20), ref[20:], dtype, "four hundred decoded positions")
    h.release_gpu_resources()


def test_steps_repeat_exactly(tmp_path):
    """The merge of the splits does not depend on the order in which they finish."""
    p = Pair(tmp_path, CONFIGS["long"], seed=13)
    toks = p.tokens(300, 8)
    h = p.open("default")
    h.prefill("a", toks[:-1], 0)
    first = h.forward_batch(["a"], [[toks[-1]]], [299])
    for _ in range(20):
        assert np.array_equal(h.forward_batch(["a"], [[toks[-1]]], [299]), first)
    h.release_gpu_resources()


# ── each mechanism alone ─────────────────────────────────────────────────────────────────────────
def _plain_layer(kind):
    return W(4, 2, 24, 16, 1000, 64, (0.0, 10)) if kind == "window" else C(4, 2, 24, 16, 1000, 64, (100.0, 12))


# name -> (kind of layer, changes of the layer, edit of the tensors, what the oracle without the mechanism is patched to)
def _times(k, *suffixes):
    def edit(t):
        for name in t:
            if name.endswith(suffixes):
                t[name] = t[name] * np.float32(k)
    return edit


def _norms_wide(t):
    for name in t:
        if name.endswith((".norm1", ".norm2", "final.norm")):
            t[name] = t[name] * np.float32(2.0)


MECHANISMS = {
    "window": ("window", dict(size=9), None, "window_mask", lambda T, size: np.tril(np.ones((T, T), bool))),
    "chunk": ("chunk", dict(size=11), None, "chunk_mask", lambda T, size: np.tril(np.ones((T, T), bool))),
    "distance bias": ("window", {}, None, "distance_slopes", lambda H: np.zeros(H)),
    "query temperature": ("window", dict(q_temp=(1.5, 6)), _times(2, ".mix.q"), "query_temperature", lambda T, c, e: np.ones(T)),
    "learned sink": ("window", {}, _times(3, ".sink"), "sink_softmax", lambda s, m, k: RIGHT_SOFTMAX(s, m, np.full_like(k, -1e9))),
    "fixed sink": ("chunk", {}, None, "sink_softmax", lambda s, m, k: RIGHT_SOFTMAX(s, m, np.full_like(k, -1e9))),
    "rotation": ("chunk", {}, _times(2, ".q.norm"), "rotate_half", lambda x, b, d: x),
    "query and key norms": ("chunk", dict(scale=1.0), _times(2, ".mix.q", ".mix.k"), "rms_unit", lambda x, eps: x if x.ndim == 3 else x / np.sqrt(np.mean(x * x, -1, keepdims=True) + eps)),
    "biases": ("window", {}, _times(5, ".q.b", ".k.b", ".v.b"), "heads_of", lambda h, w, name, n: (h @ w[name].T).reshape(h.shape[0], n, -1)),
    "norm weights": ("window", {}, _norms_wide, "offset_norm", lambda x, w, eps: x / np.sqrt(np.mean(x * x, -1, keepdims=True) + eps)),
    "feed-forward": ("window", {}, None, "gated_gelu_mlp", lambda h, w, p: 0.0 * h),
    "hyper-connections": ("chunk", {}, _times(2, "hc1.out", "hc2.out"), "hyper_connection",
                          lambda xs, w, p, f: xs + f(xs.mean(0))[None]),
}
RIGHT_SOFTMAX = do.sink_softmax


@pytest.mark.parametrize("name", sorted(MECHANISMS))
def test_each_mechanism_alone(tmp_path, name, monkeypatch):
    kind, change, edit, attr, without = MECHANISMS[name]
    p = Pair(tmp_path, synth.desilorn_config(112, 101, [dict(_plain_layer(kind), **change)], streams=3, eps=1e-3), 21, edit)
    toks = p.tokens(60, 3)
    ref = p.oracle(toks)
    with monkeypatch.context() as m:
        m.setattr(do, attr, without)
        assert row_err(p.oracle(toks), ref).max() > 0.1, "the mechanism does not show"
    for dtype in DTYPES:
        h = p.open(dtype)
        check(h.prefill_logits("a", toks, 0, range(60)), ref, dtype, f"{name}, prompt")
        check(decode_all(h, "b", toks), ref, dtype, f"{name}, decoded")
        h.release_gpu_resources()


def test_every_pass_of_a_loop_has_its_own_cache(tmp_path):
    layers = [W(2, 1, 16, 16, 12, 48), C(3, 1, 16, 32, 20, 0, (50.0, 6)), W(2, 2, 16, 16, 30, 32)]
    for k, loop in enumerate([(0, 2, 4), (2, 3, 3), (0, 3, 2), (1, 1, 7)]):
        p = Pair(tmp_path, synth.desilorn_config(64, 70, layers, streams=2, loop=loop), 31)
        toks = p.tokens(70, 1)
        ref = p.oracle(toks)
        for dtype in DTYPES:
            h = p.open(dtype)
            check(h.prefill_logits("a", toks, 0, range(70)), ref, dtype)
            check(decode_all(h, "b", toks), ref, dtype)
            h.release_gpu_resources()


def test_residual_stream_after_the_last_layer(tmp_path):
    p = Pair(tmp_path, CONFIGS["odd"], 32)
    toks, streams = p.tokens(64, 1), []
    do.forward(toks, p.cfg, p.w, streams)
    top = np.abs(streams[-1]).max()
    h = p.open("f32")
    h.prefill("a", toks, 0)
    assert np.abs(h.last_hidden(64) - streams[-1]).max() <= 2e-5 * top
    h.release_gpu_resources()
    h = p.open("default")  # the decode step's residual rows alternate between two buffers
    h.prefill("a", toks[:-1], 0)
    for _ in range(3):  # eager, captured, replayed
        h.forward_batch(["a"], [[toks[-1]]], [63])
        assert np.abs(h.last_hidden(1)[0] - streams[-1][-1]).max() <= 0.05 * top
    h.release_gpu_resources()


# ── generation, the trace command, refusals ──────────────────────────────────────────────────────
@pytest.mark.parametrize("chunked", [False, True])
def test_greedy_generation(tmp_path, chunked):
    from juno_b200.handler import B200InferencePipeline, generate_greedy
    p = Pair(tmp_path, CONFIGS["real"], 41)
    prompt = p.tokens(30, 1)
    for dtype in DTYPES:
        h = p.open(dtype)
        got = generate_greedy(B200InferencePipeline(h), "g", prompt, 24, chunked_prefill=chunked)
        ref, margins = do.generate_greedy(prompt, 24, p.cfg, p.w)
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
    from juno_b200.handler import B200TransformerHandler
    from juno_b200.safetensors_file import write_model_folder
    cfg = synth.desilorn_config(64, 70, [W(2, 1, 16, 16, 8, 48), C(2, 1, 16, 16, 8, 48)], loop=(0, 1, 2))
    t, _ = build(cfg)

    def opened(c, tensors):
        d = write_model_folder(str(tmp_path / f"x{len(os.listdir(tmp_path))}"), c, tensors)
        B200TransformerHandler.open(d).release_gpu_resources()

    def changed(f):
        c = json.loads(json.dumps(cfg))
        f(c)
        return c

    opened(cfg, t)
    opened(changed(lambda c: c.pop("loop")), t)
    with pytest.raises(ValueError, match="l1.mix.k.norm is missing"):
        opened(cfg, {k: v for k, v in t.items() if k != "l1.mix.k.norm"})
    with pytest.raises(ValueError, match="has shape"):
        opened(cfg, dict(t, **{"l0.hc2.mix": t["l0.hc2.mix"][:1]}))
    for error, text, f in [
        (JunoError, "not part of this design", lambda c: c["layers"][0].update(type="latent_attention")),
        (JunoError, "not part of this design", lambda c: c["layers"][1]["mlp"].update(kind="experts")),
        (ValueError, "cannot share", lambda c: c["layers"][0]["mixer"].update(heads=3, kv_heads=2)),
        (ValueError, "mask.size", lambda c: c["layers"][1]["mixer"].pop("mask")),
        (ValueError, "rot.dims", lambda c: c["layers"][1]["mixer"]["rot"].update(dims=18)),
        (ValueError, "rot.dims", lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7)),
        (ValueError, "streams", lambda c: c.update(streams=0)),
        (ValueError, "loop.stop", lambda c: c["loop"].update(stop=3)),
    ]:
        with pytest.raises(error, match=text):
            opened(changed(f), t)
