"""Plain restatement of the Vosotar design in numpy: one function per mechanism, whole sequences, no cache.

Test infrastructure, like the rest of this folder: only tests use it.  Everything is computed in the dtype of the weights it
is given (float64 by default), so it says what the design computes, not how the engine rounds.

`cfg` is the parsed config.json, `w` maps tensor names to arrays.
"""
from __future__ import annotations

import numpy as np


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def rms_unit(x, eps):
    """x divided by its root mean square, eps inside the root."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def scalar_norm(x, g, eps):
    """RMS norm whose weight is one number."""
    return rms_unit(x, eps) * g


def vector_norm(x, w, eps):
    return rms_unit(x, eps) * w


def causal_conv(h, w):
    """Depthwise causal convolution over time: tap taps-1 meets the current input, zeros before the first position."""
    T, taps = h.shape[0], w.shape[1]
    out = np.zeros_like(h)
    for t in range(T):
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                out[t] += w[:, j] * h[s]
    return out


def causal_softmax(scores):
    """scores [H, T, T] -> weights, position i over j <= i."""
    T = scores.shape[-1]
    s = np.where(np.tril(np.ones((T, T), dtype=bool)), scores, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def latent_attention(h, mix, w, p, eps):
    """h [T, width] -> [T, width].  Keys and values are linear in a normed latent of kv_rank numbers per position."""
    H, d, dv = mix["heads"], mix["dim"], mix["vdim"]
    T = h.shape[0]
    q = vector_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps) @ w[p + "uq"].T
    c = vector_norm(h @ w[p + "dkv"].T, w[p + "dkv.norm"], eps)
    k, v = c @ w[p + "uk"].T, c @ w[p + "uv"].T
    q = q.reshape(T, H, d).transpose(1, 0, 2)
    k = k.reshape(T, H, d).transpose(1, 0, 2)
    v = v.reshape(T, H, dv).transpose(1, 0, 2)
    o = causal_softmax(q @ k.transpose(0, 2, 1) * mix["scale"]) @ v
    o = o * sigmoid(h @ w[p + "g"].T).T[:, :, None]  # one gate per head
    return o.transpose(1, 0, 2).reshape(T, H * dv) @ w[p + "o"].T


def squared_relu_mlp(h, w, p):
    a = np.maximum(h @ w[p + "up"].T, 0.0)
    return (a * a) @ w[p + "down"].T


def residual_gate(h, w, name):
    """Element-wise gate of a sublayer's result, read from what the sublayer was handed."""
    return sigmoid(h @ w[name].T + w[name + ".b"])


def layer(x, cfg, i, w):
    spec, src = cfg["layers"][i], i
    while cfg["layers"][src].get("weights_of") is not None:  # this layer runs with another layer's tensors
        src = cfg["layers"][src]["weights_of"]
    L, eps = f"l{src}.", cfg["norm"]["eps"]
    h = scalar_norm(x, w[L + "norm1"], eps)
    y = latent_attention(h + causal_conv(h, w[L + "canon1"]), spec["mixer"], w, L + "mix.", eps)
    x = x + scalar_norm(y * residual_gate(h, w, L + "rg1"), w[L + "norm1b"], eps)
    if spec["mlp"] is not None:
        h = scalar_norm(x, w[L + "norm2"], eps)
        y = squared_relu_mlp(h, w, L + "mlp.")
        x = x + scalar_norm(y * residual_gate(h, w, L + "rg2"), w[L + "norm2b"], eps)
    return x


def forward(tokens, cfg, w, streams=None):
    """Logits [T, vocab] of one sequence; `streams` (a list) collects the residual stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = scalar_norm(w["embed"][np.asarray(tokens)], w["embed.norm"], eps)
    for i in range(len(cfg["layers"])):
        x = layer(x, cfg, i, w)
        if streams is not None:
            streams.append(x.copy())
    return scalar_norm(x, w["final.norm"], eps) @ w["head"].T


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
