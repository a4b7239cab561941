"""Small random Vosotar models for the tests (see stackutil)."""
import stackutil
from juno_b200 import synth
from oracle import vosotar_oracle as vo
from stackutil import check, decode_all, row_err  # noqa: F401


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
    return stackutil.build(synth.random_vosotar, cfg, seed, edit)


class Pair(stackutil.Pair):
    oracle_module = vo
    random_model = staticmethod(synth.random_vosotar)
