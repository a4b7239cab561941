"""Plain restatement of the Desilorn design in numpy: one function per mechanism, whole sequences, no cache.

Test infrastructure, like the rest of this folder: only tests use it.  Everything is computed in the dtype of the weights it
is given (float64 by default), so it says what the design computes, not how the engine rounds.

`cfg` is the parsed config.json, `w` maps tensor names to arrays.
"""
from __future__ import annotations

import math

import numpy as np

from .vosotar_oracle import rms_unit


def offset_norm(x, w, eps):
    """RMS norm whose weight is stored as its distance from one."""
    return rms_unit(x, eps) * (1.0 + w)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rotate_half(x, base, dims):
    """x [T, H, d], row t at position t: dimension i < dims/2 turns together with dimension i + dims/2."""
    T, half = x.shape[0], dims // 2
    freq = float(base) ** (-2.0 * np.arange(half) / dims)
    a = np.arange(T)[:, None] * freq
    cos, sin = np.cos(a)[:, None, :].astype(x.dtype), np.sin(a)[:, None, :].astype(x.dtype)
    u, v = x[..., :half], x[..., half:dims]
    return np.concatenate([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], axis=-1)


def query_temperature(T, coef, every):
    """Factor of the query at each position."""
    return np.array([1.0 + coef * math.log(math.floor((p + 1) / every) + 1.0) for p in range(T)])


def distance_slopes(heads):
    return np.array([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)])


def window_mask(T, size):
    """[T, T] True where position i sees j: itself and the size - 1 positions before it."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (i - j >= 0) & (i - j < size)


def chunk_mask(T, size):
    """[T, T] True where j <= i lies in the same chunk of `size` positions, chunks counted from position 0."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & (i // size == j // size)


def sink_softmax(scores, mask, sink):
    """scores [H, T, T]; the denominator has one more term exp(sink[h])."""
    s = np.where(mask, scores, -np.inf)
    m = np.maximum(s.max(axis=-1, keepdims=True), sink[:, None, None])
    e = np.exp(s - m)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(sink[:, None, None] - m))


def heads_of(h, w, name, n):
    """Biased projection, [T, n, size]."""
    y = h @ w[name].T + w[name + ".b"]
    return y.reshape(h.shape[0], n, -1)


def grouped_scores(q, k, scale):
    """q [T, H, d], k [T, G, d] -> [H, T, T]; query head h meets key head h // (H / G)."""
    k = np.repeat(k, q.shape[1] // k.shape[1], axis=1)
    return np.einsum("ihd,jhd->hij", q, k) * scale


def grouped_average(p, v, H):
    """p [H, T, T], v [T, G, dv] -> [T, H * dv]."""
    v = np.repeat(v, H // v.shape[1], axis=1)
    return np.einsum("hij,jhd->ihd", p, v).reshape(v.shape[0], -1)


def window_attention(h, mix, w, p, eps):
    """Sliding window, distance bias, query temperature, one learned sink per head."""
    H, G, T = mix["heads"], mix["kv_heads"], h.shape[0]
    q, k, v = heads_of(h, w, p + "q", H), heads_of(h, w, p + "k", G), heads_of(h, w, p + "v", G)
    if mix.get("q_temp"):
        q = q * query_temperature(T, mix["q_temp"]["coef"], mix["q_temp"]["every"])[:, None, None].astype(h.dtype)
    s = grouped_scores(q, k, mix["scale"])
    s = s - distance_slopes(H)[:, None, None].astype(h.dtype) * (np.arange(T)[:, None] - np.arange(T)[None, :])
    return grouped_average(sink_softmax(s, window_mask(T, mix["mask"]["size"]), w[p + "sink"]), v, H) @ w[p + "o"].T


def chunk_attention(h, mix, w, p, eps):
    """Chunked, normed and rotated queries and keys, a fixed sink of score 0."""
    H, G, T = mix["heads"], mix["kv_heads"], h.shape[0]
    q = rms_unit(heads_of(h, w, p + "q", H), eps) * w[p + "q.norm"]
    k = rms_unit(heads_of(h, w, p + "k", G), eps) * w[p + "k.norm"]
    v = heads_of(h, w, p + "v", G)
    q, k = (rotate_half(x, mix["rot"]["base"], mix["rot"]["dims"]) for x in (q, k))
    s = grouped_scores(q, k, mix["scale"])
    return grouped_average(sink_softmax(s, chunk_mask(T, mix["mask"]["size"]), np.zeros(H, h.dtype)), v, H) @ w[p + "o"].T


MIXERS = {"attention": window_attention, "attention_2": chunk_attention}


def gated_gelu_mlp(h, w, p):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def hyper_connection(xs, w, p, sublayer):
    """xs [S, T, width]: the sublayer reads a weighted sum of the streams; every stream then becomes its own mixture of the old
    streams (mix[from, to]) plus its share of the result."""
    y = sublayer(np.tensordot(w[p + "in"], xs, axes=(0, 0)))
    return np.stack([np.tensordot(w[p + "mix"][:, t], xs, axes=(0, 0)) + w[p + "out"][t] * y for t in range(xs.shape[0])])


def layer(xs, cfg, i, w):
    spec, L, eps = cfg["layers"][i], f"l{i}.", cfg["norm"]["eps"]
    mixer = MIXERS[spec["type"]]
    xs = hyper_connection(xs, w, L + "hc1.", lambda u: mixer(offset_norm(u, w[L + "norm1"], eps), spec["mixer"], w, L + "mix.", eps))
    if spec["mlp"] is not None:
        xs = hyper_connection(xs, w, L + "hc2.", lambda u: gated_gelu_mlp(offset_norm(u, w[L + "norm2"], eps), w, L + "mlp."))
    return xs


def layer_runs(cfg):
    """Indices of the layers in the order they run: a span of them runs several times in a row."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


def forward(tokens, cfg, w, streams=None):
    """Logits [T, vocab] of one sequence; `streams` (a list) collects the sum of the streams after every layer run."""
    e = w["embed"][np.asarray(tokens)]
    xs = np.repeat(e[None], cfg["streams"], axis=0)
    for i in layer_runs(cfg):
        xs = layer(xs, cfg, i, w)
        if streams is not None:
            streams.append(xs.sum(axis=0))
    return offset_norm(xs.sum(axis=0), w["final.norm"], cfg["norm"]["eps"]) @ w["embed"].T


def generate_greedy(prompt, steps, cfg, w):
    """Greedy continuation by running the whole sequence again for every token.  Returns (ids, top-2 margins)."""
    seq, ids, margins = list(prompt), [], []
    for _ in range(steps):
        row = forward(seq, cfg, w)[-1]
        top = np.sort(row)[-2:]
        ids.append(int(np.argmax(row)))
        margins.append(float(top[1] - top[0]))
        seq.append(ids[-1])
    return ids, margins
