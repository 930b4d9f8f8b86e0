"""Small random Ganupel models for the tests."""
import numpy as np

from tests.bolonex_util import bf16_exact, row_errors, tokens_for  # noqa: F401
from tnsr_b200.ganupel import Ganupel, GanupelConfig


def parallel(left, right, mlp=None, scales=(0.7, 1.2)):
    """left = (heads, kv_heads, dim, vdim, rotated dims, window, score scale), right = (heads, dim, vdim)."""
    heads, kv_heads, dim, vdim, rot, window, scale = left
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": window},
                               "rot": {"base": 5000.0, "dims": rot}},
                      "right": {"heads": right[0], "dim": right[1], "vdim": right[2]}, "left_scale": scales[0], "right_scale": scales[1]}}


def rglru(width, blocks, conv, mlp=None):
    return {"type": "rglru", "mlp": mlp, "mixer": {"width": width, "blocks": blocks, "conv": conv}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, identity, top, scale=1.5):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top, "scale": scale}}


def config(width, vocab, layers, eps=1e-5):
    return {"architecture": "Ganupel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


# sizes differ from one another in a model where they can; every mixer with every feed-forward and with none
CONFIGS = {
    "mixed": config(96, 211, [parallel((4, 2, 24, 40, 16, 19, 0.3), (3, 20, 28), moe(40, 5, 2, 3)), rglru(72, 3, 3, dense(112)),
                              parallel((6, 3, 16, 24, 16, 50, 0.2), (2, 36, 12), dense(80), (1.1, 0.4)), rglru(48, 2, 4, moe(24, 4, 1, 2, 0.8)),
                              rglru(40, 4, 2), parallel((2, 1, 32, 16, 8, 33, 0.25), (4, 16, 24))]),
    # heads of 64, states of 128 x 64, widths of whole 16-byte groups: the tensor-core kernels
    "even": config(128, 320, [parallel((8, 2, 64, 64, 64, 48, 0.13), (2, 128, 64), dense(192)), rglru(192, 3, 4, moe(96, 7, 1, 2)),
                              parallel((4, 4, 64, 64, 32, 131, 0.1), (3, 64, 128), moe(128, 6, 3, 4, 2.5))]),
    # nothing divides anything: odd widths, one expert chosen, no identity expert
    "odd": config(70, 97, [parallel((3, 3, 10, 7, 6, 5, 0.4), (5, 5, 7), dense(37)), rglru(45, 5, 5, moe(13, 3, 0, 1)),
                           parallel((9, 1, 14, 22, 14, 1, 0.3), (1, 9, 3), moe(21, 2, 5, 2))], eps=1e-3),
    # wide heads and states (norms in a launch of their own), many experts, one block, one tap
    "wide": config(160, 128, [parallel((2, 1, 136, 200, 64, 100, 0.08), (2, 136, 200), moe(32, 40, 30, 8)), rglru(160, 1, 1, dense(96)),
                              parallel((4, 2, 96, 80, 0, 64, 0.1), (2, 200, 136))]),
}


def random_tensors(cfg, seed=0, sharp=2.0, decisive=False):
    """bf16-exact weights that keep activations of order one.  `sharp` scales queries and keys, so that single keys stand out
    and a wrong one is visible in the logits.  `decisive`: corrections that choose the experts whatever the rounding."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in GanupelConfig.from_dict(cfg).tensor_shapes().items():
        leaf = name.split(".")[-1]
        if name.endswith(("norm1", "norm2", "final.norm")):
            v = rng.normal(0, 0.3, shape)
        elif leaf in ("ls1", "ls2"):
            v = rng.uniform(0.4, 1.2, shape)
        elif leaf == "pb":
            v = rng.uniform(-4.0, -2.0, shape)
        elif leaf == "lower":
            v = np.where(rng.random(shape) < 0.2, 0.0, rng.uniform(0, 0.9, shape))
        elif name.endswith("f.b"):
            v = rng.uniform(-1.0, 6.0, shape)
        elif leaf == "norm":
            v = rng.uniform(0.5, 1.5, shape)
        elif leaf == "lam":
            v = rng.uniform(-5.0, 0.0, shape)
        elif leaf == "act":
            v = rng.uniform(0.3, 0.9, shape)
        elif leaf == "correction":
            v = rng.permutation(shape[0]) * 2.0 if decisive else np.where(rng.random(shape) < 0.4, 0.3, 0.0)
        elif leaf == "conv":
            v = rng.normal(0, 0.3, shape) + (np.arange(shape[1]) == shape[1] - 1)
        elif leaf == "b":
            v = rng.normal(0, 0.3, shape)
        elif name == "embed":
            v = rng.normal(0, 1.0, shape)
        else:
            v = rng.normal(0, shape[-1] ** -0.5, shape)
            if name.endswith(("left.q", "left.k")):
                v *= sharp
            elif leaf == "router":
                v *= 3.0
        out[name] = bf16_exact(np.asarray(v, dtype=np.float32))
    return out


def build(name_or_config, dtype="bf16", seed=0, sharp=2.0):
    cfg = CONFIGS[name_or_config] if isinstance(name_or_config, str) else name_or_config
    tensors = random_tensors(cfg, seed, sharp, decisive=dtype == "bf16")
    return cfg, tensors, Ganupel(GanupelConfig.from_dict(cfg, dtype), tensors)
