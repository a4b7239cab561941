"""CPU checks: the numpy statement of the Desilorn design against independent formulas, and mistakes planted in it."""
import math

import numpy as np
import pytest

from desilornutil import CONFIGS, C, W, build, row_err
from juno_b200 import synth
from oracle import desilorn_oracle as do


def test_norm_weights_are_distances_from_one():
    x = np.random.default_rng(0).standard_normal((5, 12))
    w = np.arange(12.0)
    assert np.allclose(do.offset_norm(x, w, 1e-2), x * (w + 1) / np.sqrt((x ** 2).sum(-1, keepdims=True) / 12 + 1e-2))


def test_gelu_tanh_is_close_to_the_exact_gelu():
    z = np.linspace(-6, 6, 101)
    exact = z * np.array([0.5 * (1 + math.erf(v / math.sqrt(2))) for v in z])
    assert np.abs(do.gelu_tanh(z) - exact).max() < 2e-3 and do.gelu_tanh(np.array([0.0]))[0] == 0.0


def test_rotation_makes_products_depend_on_the_distance():
    rng = np.random.default_rng(1)
    q, k = rng.standard_normal(8), rng.standard_normal(8)
    Q, K = (do.rotate_half(np.tile(v, (20, 1, 1)), 100.0, 6)[:, 0] for v in (q, k))
    assert np.allclose(Q[0], q) and np.allclose(Q[:, 6:], q[6:])
    d = Q[:, :6] @ K[:, :6].T
    for s in range(1, 20):
        assert np.allclose(np.diag(d, -s), d[s, 0])
    # pair (i, i + 3) turns by p * base^(-2 i / 6), as a complex number
    z = (q[:3] + 1j * q[3:6]) * np.exp(1j * 7 * 100.0 ** (-np.arange(3) / 3.0))
    assert np.allclose(Q[7, :6], np.concatenate([z.real, z.imag]))


def test_query_temperature_steps():
    f = do.query_temperature(25, 0.5, 10)
    assert np.allclose(f[:9], 1.0) and np.allclose(f[9:19], 1 + 0.5 * math.log(2)) and np.allclose(f[19:], 1 + 0.5 * math.log(3))


def test_slopes():
    assert np.allclose(do.distance_slopes(8), [0.5 ** (h + 1) for h in range(8)]) and np.allclose(do.distance_slopes(3)[2], 2.0 ** -8)


@pytest.mark.parametrize("size", [1, 2, 5, 30])
def test_masks(size):
    w, c = do.window_mask(17, size), do.chunk_mask(17, size)
    for i in range(17):
        assert np.flatnonzero(w[i]).tolist() == list(range(max(0, i - size + 1), i + 1))
        assert np.flatnonzero(c[i]).tolist() == list(range(i // size * size, i + 1))


def test_the_sink_takes_weight_and_gives_nothing():
    rng = np.random.default_rng(2)
    s, sink = rng.standard_normal((2, 4, 4)), np.array([0.0, 2.5])
    mask = np.tril(np.ones((4, 4), bool))
    p = do.sink_softmax(s, mask, sink)
    for h in range(2):
        for i in range(4):
            e = np.exp(s[h, i, :i + 1])
            assert np.allclose(p[h, i, :i + 1], e / (e.sum() + np.exp(sink[h]))) and (p[h, i, i + 1:] == 0).all()
    assert np.allclose(do.sink_softmax(s + 1000.0, mask, sink).sum(-1), 1.0)  # no overflow


def test_one_stream_with_unit_connections_is_the_plain_residual_sum():
    w = {"h.in": np.ones(1), "h.out": np.ones(1), "h.mix": np.ones((1, 1))}
    x = np.random.default_rng(3).standard_normal((1, 5, 7))
    assert np.allclose(do.hyper_connection(x, w, "h.", lambda u: 2 * u), 3 * x)


def test_streams_mix_from_to():
    w = {"h.in": np.array([1.0, 0.0]), "h.out": np.array([0.0, 3.0]), "h.mix": np.array([[0.0, 1.0], [0.0, 0.0]])}
    x = np.arange(8.0).reshape(2, 2, 2)
    y = do.hyper_connection(x, w, "h.", lambda u: u + 1)
    assert np.allclose(y[0], 0.0) and np.allclose(y[1], x[0] + 3 * (x[0] + 1))


def test_grouped_heads_share_keys():
    rng = np.random.default_rng(4)
    q, k, v = rng.standard_normal((5, 6, 3)), rng.standard_normal((5, 2, 3)), rng.standard_normal((5, 2, 4))
    s = do.grouped_scores(q, k, 0.5)
    p = rng.random((6, 5, 5))
    o = do.grouped_average(p, v, 6).reshape(5, 6, 4)
    for h in range(6):
        assert np.allclose(s[h], 0.5 * q[:, h] @ k[:, h // 3].T) and np.allclose(o[:, h], p[h] @ v[:, h // 3])


def test_order_of_runs():
    def runs(loop):
        return do.layer_runs(synth.desilorn_config(16, 10, [W(2, 1, 8, 8, 4, 8)] * 4, loop=loop))
    assert runs((1, 3, 3)) == [0, 1, 2, 1, 2, 1, 2, 3] and runs((0, 4, 2)) == [0, 1, 2, 3] * 2
    assert runs(None) == runs((2, 3, 1)) == runs((2, 2, 5)) == [0, 1, 2, 3]


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_a_position_does_not_see_the_future(name):
    cfg = CONFIGS[name]
    _, w = build(cfg, 3)
    a = np.random.default_rng(0).integers(0, cfg["vocab"], 20).tolist()
    b = a[:12] + [(t + 1) % cfg["vocab"] for t in a[12:]]
    x, y = do.forward(a, cfg, w), do.forward(b, cfg, w)
    assert np.allclose(x[:12], y[:12]) and not np.allclose(x[12], y[12])


def test_tensor_names_follow_the_layers():
    names = synth.desilorn_shapes(CONFIGS["odd"])
    assert "l1.mix.q.norm" in names and "l0.mix.sink" in names and "l1.mix.sink" not in names
    assert "l1.hc1.mix" in names and "l1.hc2.mix" not in names and "l1.norm2" not in names and not any(n.startswith("l3.") for n in names)


# ── mistakes that the tests of the engine have to be able to see, planted in the oracle ──────────
RIGHT = {k: getattr(do, k) for k in ("window_mask", "chunk_mask", "query_temperature", "sink_softmax", "rotate_half", "hyper_connection", "layer_runs")}


def _mix_with(change):
    return lambda xs, w, p, f: RIGHT["hyper_connection"](xs, dict(w, **{p + "mix": change(w[p + "mix"])}), p, f)


def _neighbours_rotated(x, base, dims):
    order = np.concatenate([np.arange(0, dims, 2), np.arange(1, dims, 2)])
    y = RIGHT["rotate_half"](np.concatenate([x[..., order], x[..., dims:]], -1), base, dims)
    out = y.copy()
    out[..., order] = y[..., :dims]
    return out


MISTAKES = {
    "window one longer": ("window_mask", lambda T, n: RIGHT["window_mask"](T, n + 1)),
    "window one shorter": ("window_mask", lambda T, n: RIGHT["window_mask"](T, n - 1)),
    "chunk one longer": ("chunk_mask", lambda T, n: RIGHT["chunk_mask"](T, n + 1)),
    "no distance bias": ("distance_slopes", lambda H: np.zeros(H)),
    "slopes from head 0": ("distance_slopes", lambda H: 2.0 ** (-8.0 * np.arange(H) / H)),
    "no temperature": ("query_temperature", lambda T, c, e: np.ones(T)),
    "temperature a position late": ("query_temperature", lambda T, c, e: np.concatenate([[1.0], RIGHT["query_temperature"](T, c, e)[:-1]])),
    "no sink": ("sink_softmax", lambda s, m, k: RIGHT["sink_softmax"](s, m, np.full_like(k, -1e9))),
    "sink twice": ("sink_softmax", lambda s, m, k: RIGHT["sink_softmax"](s, m, k + math.log(2))),
    "no rotation": ("rotate_half", lambda x, b, d: x),
    "neighbours rotated together": ("rotate_half", _neighbours_rotated),
    "streams not mixed": ("hyper_connection", _mix_with(lambda m: np.eye(len(m)))),
    "mixture transposed": ("hyper_connection", _mix_with(lambda m: m.T)),
    "gate and value exchanged": ("gated_gelu_mlp", lambda h, w, p: (do.gelu_tanh(h @ w[p + "up"].T) * (h @ w[p + "gate"].T)) @ w[p + "down"].T),
    "one loop less": ("layer_runs", lambda cfg: RIGHT["layer_runs"](dict(cfg, loop=dict(cfg["loop"], times=cfg["loop"]["times"] - 1)))),
}


def test_planted_mistakes_show(monkeypatch):
    cfg = synth.desilorn_config(96, 120, [W(4, 2, 24, 16, 19, 64, (0.6, 12)), C(4, 2, 24, 16, 23, 64, (100.0, 12))], streams=3, loop=(0, 2, 2))

    def edit(t):
        for k in t:
            if k.endswith((".mix.q", ".mix.k")):
                t[k] *= 1.5
    _, w = build(cfg, 5, edit)
    toks = np.random.default_rng(0).integers(0, 120, 60).tolist()
    ref = do.forward(toks, cfg, w)
    for what, (name, wrong) in MISTAKES.items():
        with monkeypatch.context() as m:
            m.setattr(do, name, wrong)
            assert row_err(do.forward(toks, cfg, w), ref).max() > 0.1, what
    assert np.allclose(do.forward(toks, cfg, w), ref)
