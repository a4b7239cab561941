"""Small random Desilorn models for the tests (see stackutil)."""
import stackutil
from juno_b200 import synth
from oracle import desilorn_oracle as do
from stackutil import check, decode_all, row_err  # noqa: F401


def W(heads, kv_heads, dim, vdim, size, ff, q_temp=(0.4, 50), scale=None):
    """A window layer: positions through a distance bias."""
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, size=size, ff=ff, q_temp=q_temp, scale=scale or dim ** -0.5)


def C(heads, kv_heads, dim, vdim, size, ff, rot=(10000.0, 16), scale=None):
    """A chunk layer: positions through a rotation."""
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, size=size, ff=ff, rot=rot, scale=scale or dim ** -0.5)


# sizes that are no multiples of the kernels' tiles, and the corners the kernels split at
CONFIGS = {
    # nothing is a multiple of 16; half the rotated dimensions an odd number; a layer without a feed-forward; a looped pair
    "odd": synth.desilorn_config(150, 333, [W(6, 3, 20, 28, 21, 200, (0.7, 10)), C(4, 1, 36, 18, 33, 0, (500.0, 10)), W(3, 3, 17, 33, 50, 77, (-0.2, 7))],
                                 streams=3, loop=(1, 3, 2), eps=1e-5),
    # more query heads per key/value head than a tile of the decode attention; a window of one position, a chunk of one
    "groups": synth.desilorn_config(192, 257, [W(40, 2, 32, 16, 100, 96), C(20, 1, 16, 32, 70, 64, (10000.0, 16)), W(2, 1, 16, 16, 1, 0), C(2, 2, 16, 16, 1, 40, (10.0, 4))],
                                    streams=2, loop=(0, 2, 2)),
    # spans longer than what one split takes; one stream; every dimension rotated
    "long": synth.desilorn_config(128, 200, [W(4, 1, 64, 64, 333, 128, (0.3, 100)), C(8, 4, 48, 64, 200, 96, (1e6, 48))], streams=1, loop=(0, 1, 1)),
    # heads of two hundred dimensions; five streams; the whole stack three times
    "wide": synth.desilorn_config(96, 130, [C(3, 1, 200, 144, 90, 40, (50000.0, 120)), W(2, 1, 144, 256, 64, 56)], streams=5, loop=(0, 2, 3)),
    # heads wider than the tensor-core kernels take: the general kernel
    "bighead": synth.desilorn_config(64, 90, [W(2, 1, 272, 300, 40, 50), C(2, 2, 280, 16, 48, 0, (100.0, 280))], streams=2),
    # heads of two hundred and fifty-six
    "d256": synth.desilorn_config(80, 110, [W(3, 1, 256, 256, 130, 64), C(2, 2, 256, 256, 210, 0, (1e4, 64))], streams=3),
    # head sizes of real models
    "real": synth.desilorn_config(256, 300, [C(8, 2, 128, 128, 256, 256, (500000.0, 64)), W(8, 2, 128, 128, 128, 256, (0.1, 32))], streams=4, loop=(1, 2, 2)),
}


def build(cfg, seed=1, edit=None):
    return stackutil.build(synth.random_desilorn, cfg, seed, edit)


class Pair(stackutil.Pair):
    oracle_module = do
    random_model = staticmethod(synth.random_desilorn)
