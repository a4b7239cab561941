"""Small random Vosotar models for the tests: the same weights for the numpy oracle and, as a folder, for the engine."""
import numpy as np

from juno_b200 import synth
from juno_b200.safetensors_file import from_bf16, to_bf16, write_model_folder
from oracle import vosotar_oracle as vo


def L(heads, dim, vdim, q_rank, kv_rank, ff, scale=None, weights_of=None):
    return dict(heads=heads, dim=dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, ff=ff, scale=scale or dim ** -0.5, weights_of=weights_of)


# sizes that are no multiples of the kernels' tiles, and the corners the kernels split at
CONFIGS = {
    # nothing is a multiple of 16; three taps; layers of different sizes; a layer without a feed-forward
    "odd": synth.vosotar_config(150, 333, [L(3, 24, 40, 56, 72, 200), L(5, 20, 12, 30, 50, 0), L(1, 33, 17, 9, 5, 77)], taps=3, eps=1e-5),
    # more than one group of heads, a wide latent, shared weights
    "groups": synth.vosotar_config(192, 257, [L(20, 32, 16, 64, 272, 96), L(4, 16, 16, 16, 32, 64), L(20, 32, 16, 64, 272, 96, weights_of=0)], taps=5),
    # latent wider than 512 (one head tile per block), one tap (no state)
    "wide": synth.vosotar_config(96, 130, [L(18, 16, 24, 48, 600, 40)], taps=1),
    # heads wider than the prompt attention takes: the general kernel
    "bighead": synth.vosotar_config(64, 90, [L(2, 272, 300, 40, 48, 50)], taps=2),
    # head sizes of real models
    "real": synth.vosotar_config(256, 300, [L(2, 128, 192, 96, 512, 128), L(2, 128, 192, 96, 512, 128, weights_of=0)], taps=4, eps=1e-6),
}


def build(cfg, seed=1, edit=None):
    """(bf16 tensors, float64 weights); edit(name -> float32 array) may change values before they are rounded."""
    t = synth.random_vosotar(cfg, seed)
    if edit:
        f = {k: from_bf16(v) for k, v in t.items()}
        edit(f)
        t = {k: to_bf16(np.asarray(v, np.float32)) for k, v in f.items()}
    return t, {k: from_bf16(v).astype(np.float64) for k, v in t.items()}


class Pair:
    def __init__(self, tmp_path, cfg, seed=1, edit=None):
        self.cfg = cfg
        t, self.w = build(cfg, seed, edit)
        self.dir = write_model_folder(str(tmp_path / f"m{seed}_{len(list(tmp_path.iterdir()))}"), cfg, t)

    def open(self, dtype="default", **kw):
        from juno_b200.handler import B200TransformerHandler
        kw.setdefault("max_ctx", 512)
        return B200TransformerHandler.open(self.dir, dtype=dtype, **kw)

    def oracle(self, tokens):
        return vo.forward(tokens, self.cfg, self.w)

    def tokens(self, n, seed=0):
        return np.random.default_rng(seed).integers(0, self.cfg["vocab"], n).tolist()


def row_err(got, ref):
    """Per position: rms over the vocabulary of the difference (means taken off), relative to the reference's rms."""
    got, ref = np.atleast_2d(np.asarray(got, np.float64)), np.atleast_2d(np.asarray(ref, np.float64))
    d = got - ref
    d = d - d.mean(-1, keepdims=True)
    scale = np.sqrt(((ref - ref.mean(-1, keepdims=True)) ** 2).mean())
    return np.sqrt((d ** 2).mean(-1)) / scale


# 32-bit arithmetic against float64; 16-bit operands with 32-bit sums, norms, scores and state
TOL = {"f32": 2e-5, "default": 3e-2}


def check(got, ref, dtype, what=""):
    e = row_err(got, ref)
    assert np.isfinite(e).all() and e.max() <= TOL[dtype], f"{what}: position {int(np.argmax(e))} of {len(e)} is off by {e.max():.2e}"
