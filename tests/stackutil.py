"""Small random models of the layer-stack designs for the tests: the same weights for a numpy oracle and, as a folder, for the
engine, and the comparison of their logits."""
import numpy as np

from juno_b200.safetensors_file import from_bf16, to_bf16, write_model_folder


def build(random_model, cfg, seed=1, edit=None):
    """(bf16 tensors, float64 weights); edit(name -> float32 array) may change values before they are rounded."""
    t = random_model(cfg, seed)
    if edit:
        f = {k: from_bf16(v) for k, v in t.items()}
        edit(f)
        t = {k: to_bf16(np.asarray(v, np.float32)) for k, v in f.items()}
    return t, {k: from_bf16(v).astype(np.float64) for k, v in t.items()}


class Pair:
    oracle_module = None  # the design's numpy statement
    random_model = None   # (cfg, seed) -> tensors

    def __init__(self, tmp_path, cfg, seed=1, edit=None):
        self.cfg = cfg
        t, self.w = build(type(self).random_model, cfg, seed, edit)
        self.dir = write_model_folder(str(tmp_path / f"m{seed}_{len(list(tmp_path.iterdir()))}"), cfg, t)

    def open(self, dtype="default", **kw):
        from juno_b200.handler import B200TransformerHandler
        kw.setdefault("max_ctx", 512)
        return B200TransformerHandler.open(self.dir, dtype=dtype, **kw)

    def oracle(self, tokens):
        return self.oracle_module.forward(tokens, self.cfg, self.w)

    def tokens(self, n, seed=0):
        return np.random.default_rng(seed).integers(0, self.cfg["vocab"], n).tolist()


def decode_all(h, rid, tokens, start=0):
    return np.stack([h.forward_batch([rid], [[t]], [start + i])[0] for i, t in enumerate(tokens)])


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
