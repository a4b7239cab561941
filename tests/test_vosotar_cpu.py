"""CPU checks: the numpy statement of the Vosotar design against independent formulas, and the model-folder reader."""
import ctypes as C
import json
import struct

import numpy as np
import pytest

from juno_b200 import _lib, synth
from juno_b200.safetensors_file import SafetensorsFile, from_bf16, to_bf16, write_safetensors
from oracle import vosotar_oracle as vo
from vosotarutil import CONFIGS, L, build, row_err


def test_norms():
    x = np.random.default_rng(0).standard_normal((5, 12))
    assert np.allclose(np.mean(vo.scalar_norm(x, 2.0, 0.0) ** 2, -1), 4.0)
    w = np.arange(12.0)
    assert np.allclose(vo.vector_norm(x, w, 1e-2), x * w / np.sqrt((x ** 2).sum(-1, keepdims=True) / 12 + 1e-2))


@pytest.mark.parametrize("taps", [1, 2, 4, 7])
def test_convolution_is_causal_and_ends_at_the_last_tap(taps):
    rng = np.random.default_rng(taps)
    h, w = rng.standard_normal((20, 3)), rng.standard_normal((3, taps))
    ref = np.stack([np.convolve(h[:, c], w[c, ::-1])[:20] for c in range(3)], 1)
    assert np.allclose(vo.causal_conv(h, w), ref)


def test_attention_of_one_position_is_its_own_value():
    mix = dict(heads=2, dim=4, vdim=3, q_rank=5, kv_rank=6, scale=0.3)
    rng = np.random.default_rng(1)
    shapes = {"dq": (5, 8), "dq.norm": (5,), "uq": (8, 5), "dkv": (6, 8), "dkv.norm": (6,), "uk": (8, 6), "uv": (6, 6), "g": (2, 8), "o": (8, 6)}
    w = {"m." + k: rng.standard_normal(s) for k, s in shapes.items()}
    h = rng.standard_normal((1, 8))
    c = vo.vector_norm(h @ w["m.dkv"].T, w["m.dkv.norm"], 1e-6)
    v = (c @ w["m.uv"].T)[0] * np.repeat(vo.sigmoid(h @ w["m.g"].T)[0], 3)
    assert np.allclose(vo.latent_attention(h, mix, w, "m.", 1e-6)[0], w["m.o"] @ v)


def test_absorbed_queries_give_the_same_scores():
    rng = np.random.default_rng(2)
    q, uk, c = rng.standard_normal(4), rng.standard_normal((4, 6)), rng.standard_normal((9, 6))
    assert np.allclose((c @ uk.T) @ q, c @ (uk.T @ q))


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_a_position_does_not_see_the_future(name):
    cfg = CONFIGS[name]
    _, w = build(cfg, 3)
    a = np.random.default_rng(0).integers(0, cfg["vocab"], 20).tolist()
    b = a[:12] + [(t + 1) % cfg["vocab"] for t in a[12:]]
    x, y = vo.forward(a, cfg, w), vo.forward(b, cfg, w)
    assert np.allclose(x[:12], y[:12]) and not np.allclose(x[12], y[12])


def test_a_layer_without_a_feed_forward_and_shared_weights():
    one = L(2, 8, 8, 12, 12, 16)
    cfg = synth.vosotar_config(24, 30, [dict(one, ff=0), one, dict(one, weights_of=1)])
    names = synth.vosotar_shapes(cfg)
    assert "l0.mlp.up" not in names and "l0.rg2" not in names and "l1.mlp.up" in names and not any(n.startswith("l2.") for n in names)
    _, w = build(cfg)
    twice = synth.vosotar_config(24, 30, [dict(one, ff=0), one, one])
    w2 = dict(w, **{"l2" + k[2:]: v for k, v in w.items() if k.startswith("l1.")})
    toks = list(range(11))
    assert np.allclose(vo.forward(toks, cfg, w), vo.forward(toks, twice, w2))


def test_a_planted_mistake_shows():
    """Faults of the kinds a cache or a kernel could make, planted in the oracle: each moves the logits far beyond the tolerances."""
    cfg = CONFIGS["real"]
    _, w = build(cfg, 5)
    toks = np.random.default_rng(4).integers(0, cfg["vocab"], 40).tolist()
    ref = vo.forward(toks, cfg, w)
    for name, broken in {"no convolution": {"l0.canon1": 0.0}, "flipped taps": {"l0.canon1": "flip"}, "no head gate": {"l0.mix.g": 0.0},
                         "no gate bias": {"l0.rg1.b": 0.0}, "no latent norm weight": {"l0.mix.dkv.norm": 1.0}}.items():
        v = dict(w)
        for k, how in broken.items():
            v[k] = w[k][:, ::-1] if how == "flip" else np.full_like(w[k], how)
        assert np.median(row_err(vo.forward(toks, cfg, v), ref)) > 0.05, name


# ── the container ────────────────────────────────────────────────────────────────────────────────
def test_bf16_rounding():
    v = np.array([1.0, 1.00390625, 1.01171875, -3.14159, 0.0, 1e-30, 65504.0], np.float32)
    b = from_bf16(to_bf16(v))
    assert np.all(np.abs(b - v) <= np.abs(v) * 2.0 ** -8)
    assert from_bf16(to_bf16(np.float32([1.00390625])))[0] == 1.0  # half way: to even


def test_safetensors_round_trip(tmp_path):
    t = {"a": to_bf16(np.arange(12.0)).reshape(3, 4), "b.norm": to_bf16(np.float32([2.5])).reshape(()), "c": np.arange(5, dtype=np.int32),
         "d": np.linspace(0, 1, 6, dtype=np.float32)}
    write_safetensors(tmp_path / "m.safetensors", t)
    with SafetensorsFile(tmp_path / "m.safetensors") as f:
        assert f.names() == list(t)
        for k, v in t.items():
            dt, shape, raw = f.tensor(k)
            assert dt == {"uint16": "BF16", "int32": "I32", "float32": "F32"}[v.dtype.name] and shape == v.shape
            assert raw.tobytes() == v.tobytes()
        with pytest.raises(ValueError, match="not found"):
            f.tensor("nothing")


@pytest.mark.parametrize("damage", ["short", "header length", "not json", "offset", "size", "dtype shape", "deep"])
def test_damaged_safetensors_are_refused(tmp_path, damage):
    entry = {"dtype": "BF16", "shape": [2, 3], "data_offsets": [0, 12]}
    head, data = {"a": entry}, b"\0" * 12
    if damage == "offset":
        entry["data_offsets"] = [4, 16]
    if damage == "size":
        entry["shape"] = [2, 4]
    if damage == "dtype shape":
        entry["shape"] = [-1, 3]
    raw = json.dumps(head).encode()
    if damage == "not json":
        raw = raw[:-1]
    if damage == "deep":
        raw = b'{"a":' + b"[" * 200 + b"]" * 200 + b"}"
    blob = struct.pack("<Q", len(raw) + (1000 if damage == "header length" else 0)) + raw + data
    p = tmp_path / "m.safetensors"
    p.write_bytes(blob[:5] if damage == "short" else blob)
    with pytest.raises(ValueError):
        SafetensorsFile(p)


def test_structs_match_the_header():
    assert C.sizeof(_lib.OpenOpts) == 24 and C.sizeof(_lib.ModelInfo) == 32 + 8 * 4 + 3 * 8
    assert len(_lib.PROF_NAMES) == 10


def test_model_open_needs_a_context():
    h = C.c_void_p()
    o = _lib.OpenOpts(C.sizeof(_lib.OpenOpts), 1, 1, 16, 0, 0)
    assert _lib.load().juno_model_open(None, b"/nowhere", C.byref(o), C.byref(h)) != _lib.OK
