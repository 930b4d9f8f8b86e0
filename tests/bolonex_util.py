"""Small random Bolonex models for the tests, and how far two sets of logits are apart."""
import numpy as np

from tnsr_b200.bolonex import Bolonex, BolonexConfig


def bf16_exact(a):
    """Nearest bf16 values (ties to even), as f32."""
    bits = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    bits = (bits + 0x7FFF + ((bits >> 16) & 1)) & 0xFFFF0000
    return bits.astype(np.uint32).view(np.float32).reshape(np.shape(a))


def attention(heads, kv_heads, dim, vdim, conv=4, rot=None, base=10000.0, scaling=None, scale=None, softcap=20.0, ff=0, weights_of=None):
    entry = {"type": "attention", "mlp": {"kind": "dense", "ff": ff} if ff else None,
             "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "scale": scale or dim ** -0.5,
                       "softcap": softcap, "rot": {"base": base, "dims": dim - dim % 2 if rot is None else rot, "scaling": scaling}}}
    if weights_of is not None:
        entry["weights_of"] = weights_of
    return entry


def mamba2(heads, vdim, state, groups=1, norm_groups=1, conv=4, ff=0, weights_of=None):
    entry = {"type": "mamba2", "mlp": {"kind": "dense", "ff": ff} if ff else None,
             "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv}}
    if weights_of is not None:
        entry["weights_of"] = weights_of
    return entry


def config(width, vocab, layers, scale=2.0, eps=1e-5):
    return {"architecture": "Bolonex", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps},
            "layers": layers}


SCALING = {"factor": 6.0, "low": 1.0, "high": 4.0, "original": 64}

# every size differs from the others in its model where it can; shared tensors, layers without a feed-forward, mixed orders
CONFIGS = {
    "mixed": config(96, 211, [attention(4, 2, 24, 40, conv=3, rot=16, scaling=SCALING, ff=112), mamba2(6, 24, 40, groups=3, norm_groups=2, conv=2, ff=80),
                              mamba2(2, 40, 16, conv=4), attention(4, 2, 24, 40, conv=3, rot=16, scaling=SCALING, ff=112, weights_of=0),
                              mamba2(6, 24, 40, groups=3, norm_groups=2, conv=2, ff=80, weights_of=1)]),
    # widths the tensor-core kernels copy 16 bytes at a time, heads of 64, a state of 128 rows
    "even": config(128, 320, [mamba2(4, 64, 128, groups=2, norm_groups=4, ff=192), attention(8, 2, 64, 64, base=5000.0, scaling=SCALING, ff=256),
                              mamba2(4, 64, 128, groups=2, norm_groups=4, ff=192, weights_of=0)], scale=1.5),
    # nothing divides anything: one head per key/value head, no cap, no frequency scaling, one tap, no feed-forward
    "odd": config(70, 97, [attention(3, 3, 10, 7, conv=1, rot=6, softcap=None), mamba2(5, 7, 5, groups=5, norm_groups=5, conv=5),
                           attention(9, 1, 14, 22, conv=6, rot=14, softcap=7.0, ff=37)], scale=1.0, eps=1e-3),
    # wide heads and states: several slices of the state, two 128-column paddings
    "wide": config(160, 128, [attention(2, 1, 136, 200, rot=64, ff=96), mamba2(2, 136, 200, ff=64), attention(4, 2, 96, 80, ff=64)]),
}


def random_tensors(cfg, seed=0, sharp=1.6):
    """bf16-exact weights that keep activations of order one.  `sharp` scales the query / key norms: scores then spread
    over tens of units and attention picks few keys, so that a wrong key is visible in the logits."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in BolonexConfig.from_dict(cfg).tensor_shapes().items():
        leaf = name.split(".")[-1]
        if name.endswith(("norm1", "final.norm")):
            v = rng.normal(0, 0.3, shape)
        elif name.endswith(("q.norm", "k.norm")):
            v = sharp * rng.uniform(0.5, 1.5, shape)
        elif leaf == "norm":
            v = rng.uniform(0.5, 1.5, shape)
        elif leaf == "conv":
            v = rng.normal(0, 0.3, shape) + (np.arange(shape[1]) == shape[1] - 1)
        elif leaf == "b":
            v = rng.normal(0, 0.3, shape)
        elif leaf == "dt_bias":
            v = rng.uniform(-4.0, 0.0, shape)
        elif leaf == "A_log":
            v = rng.uniform(-3.0, 0.7, shape)
        elif leaf == "D":
            v = rng.uniform(0.3, 1.2, shape)
        elif name == "embed":
            v = rng.normal(0, 1.0, shape)
        else:
            v = rng.normal(0, shape[1] ** -0.5, shape)
        out[name] = bf16_exact(v.astype(np.float32))
    return out


def build(name_or_config, dtype="bf16", seed=0, sharp=1.6):
    cfg = CONFIGS[name_or_config] if isinstance(name_or_config, str) else name_or_config
    tensors = random_tensors(cfg, seed, sharp)
    return cfg, tensors, Bolonex(BolonexConfig.from_dict(cfg, dtype), tensors)


def tokens_for(cfg, n, seed=1):
    return [int(t) for t in np.random.default_rng(seed).integers(0, cfg["vocab"], n)]


def row_errors(got, want):
    """Root mean square of the difference per row, mean taken off, in units of the expected logits' spread."""
    d = np.asarray(got, np.float64) - np.asarray(want, np.float64)
    d = d - d.mean(axis=-1, keepdims=True)
    return np.sqrt((d * d).mean(axis=-1)) / np.std(np.asarray(want, np.float64))
