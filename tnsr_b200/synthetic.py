"""Seeded synthetic model weights for benchmarks, examples and tests: there is no
network for checkpoints, so every workload draws its parameters from a stated
generator in a stated order and any harness can rebuild the same bytes."""
import numpy as np

from .nn import GptConfig


def normal_model_arrays(cfg: GptConfig, seed: int, std: float = 0.02, bias_std: float = 0.0):
    """Parameter arrays in ``model_parameters`` order.  One ``default_rng(seed)``
    stream; matrices are drawn N(0, std) in that order (float64 draws cast to
    f32); biases are 0 unless ``bias_std`` > 0 (then drawn in order too);
    LayerNorm weight 1, bias 0."""
    rng = np.random.default_rng(seed)
    d, f, V, ctx = cfg.embed_dim, cfg.feed_forward_dim, cfg.vocab_size, cfg.max_sequence_length

    def mat(r, c):
        return (rng.standard_normal((r, c)) * std).astype(np.float32)

    def bias(n):
        if bias_std > 0:
            return (rng.standard_normal(n) * bias_std).astype(np.float32)
        return np.zeros(n, np.float32)

    arrays = [mat(V, d), mat(ctx, d), np.ones(d, np.float32), np.zeros(d, np.float32)]
    for _ in range(cfg.num_layers):
        for _ in range(4):
            arrays += [mat(d, d), bias(d)]
        arrays += [np.ones(d, np.float32), np.zeros(d, np.float32), np.ones(d, np.float32),
                   np.zeros(d, np.float32)]
        if cfg.activation == "swiglu":
            arrays += [mat(d, f), bias(f), mat(d, f), bias(f), mat(f, d), bias(d)]
        else:
            arrays += [mat(d, f), bias(f), mat(f, d), bias(d)]
    return arrays


def bolonex_config(width, layers, heads, kv_heads, head_dim, ssm_heads, ssm_dim, state, feed_forward, vocab_size, attention_every=4,
                   max_sequence_length=2048):
    """A Bolonex of real-model proportions: every `attention_every`-th layer attention, the others mamba2, none sharing."""
    from .bolonex import BolonexConfig, LayerConfig, RotaryConfig
    rotary = RotaryConfig(head_dim, 500000.0, 8.0, 1.0, 4.0, 8192.0)
    attention = LayerConfig("attention", heads, head_dim, 4, feed_forward, kv_heads=kv_heads, dim=head_dim, rotary=rotary,
                            scale=head_dim ** -0.5, softcap=30.0)
    mamba = LayerConfig("mamba2", ssm_heads, ssm_dim, 4, feed_forward, state=state, groups=1, norm_groups=1)
    return BolonexConfig(vocab_size, width, tuple(attention if i % attention_every == 0 else mamba for i in range(layers)), 1.0, 1e-5, "bf16",
                         max_sequence_length)


def bolonex_arrays(cfg, seed: int, std: float = 0.02):
    """Parameter arrays of a Bolonex in the order of its tensor table: matrices N(0, std), norms and skips one, decays and
    step biases in the range a trained layer has."""
    rng = np.random.default_rng(seed)
    arrays = []
    for name, shape in cfg.tensor_shapes().items():
        leaf = name.split(".")[-1]
        if name.endswith(("norm1", "final.norm")) or leaf == "b":
            a = np.zeros(shape, np.float32)
        elif leaf in ("norm", "D"):
            a = np.ones(shape, np.float32)
        elif leaf == "conv":
            a = rng.uniform(-0.5, 0.5, shape).astype(np.float32)
        elif leaf == "dt_bias":
            a = rng.uniform(-4.0, -1.0, shape).astype(np.float32)
        elif leaf == "A_log":
            a = np.log(rng.uniform(1.0, 16.0, shape)).astype(np.float32)
        else:
            a = rng.standard_normal(shape, dtype=np.float32) * np.float32(std)
        arrays.append(a)
    return arrays


def ganupel_config(width, layers, heads, kv_heads, head_dim, window, rec_heads, rec_dim, rec_vdim, unit_width, unit_blocks, feed_forward,
                   experts, identity, top, expert_ff, vocab_size, max_sequence_length=2048):
    """A Ganupel of real-model proportions: two layers of attention beside HGRN2, then one linear recurrent unit, and so on;
    dense feed-forwards in the even layers, experts in the odd ones."""
    from .ganupel import Dense, Experts, GanupelConfig, Hgrn2, LayerConfig, ParallelMixer, RgLru, WindowedAttention
    mixer = ParallelMixer(WindowedAttention(heads, kv_heads, head_dim, head_dim, head_dim ** -0.5, window, head_dim, 10000.0),
                          Hgrn2(rec_heads, rec_dim, rec_vdim), 1.0, 1.0)
    unit, dense, sparse = RgLru(unit_width, unit_blocks, 4), Dense(feed_forward), Experts(expert_ff, experts, identity, top, 1.0)
    return GanupelConfig(vocab_size, width, tuple(LayerConfig(unit if i % 3 == 2 else mixer, sparse if i % 2 else dense) for i in range(layers)), 1e-5, "bf16",
                         max_sequence_length)


def ganupel_arrays(cfg, seed: int, std: float = 0.02):
    """Parameter arrays of a Ganupel in the order of its tensor table: matrices N(0, std), norms, scales and biases neutral,
    gates and decays in the range a trained layer has."""
    rng = np.random.default_rng(seed)
    arrays = []
    for name, shape in cfg.tensor_shapes().items():
        leaf = name.split(".")[-1]
        if name.endswith(("norm1", "norm2", "final.norm")) or leaf in ("b", "correction"):
            a = np.full(shape, 3.0 if name.endswith("f.b") else 0.0, np.float32)
        elif leaf in ("norm", "ls1", "ls2"):
            a = np.ones(shape, np.float32)
        elif leaf == "act":
            a = np.float32([0.5, 0.3, 0.2, 0.0])
        elif leaf == "pb":
            a = np.full(shape, -5.0, np.float32)
        elif leaf == "lower":
            a = rng.uniform(0.0, 0.9, shape).astype(np.float32)
        elif leaf == "lam":
            a = rng.uniform(-8.0, -3.0, shape).astype(np.float32)
        elif leaf == "conv":
            a = rng.uniform(-0.5, 0.5, shape).astype(np.float32)
        else:
            a = rng.standard_normal(shape, dtype=np.float32) * np.float32(std)
        arrays.append(a)
    return arrays


def config0_model(activation="relu"):
    cfg = GptConfig(vocab_size=96, max_sequence_length=128, embed_dim=128, num_heads=4,
                    feed_forward_dim=512, num_layers=4, layer_norm_epsilon=1e-5, activation=activation)
    return cfg, normal_model_arrays(cfg, seed=0)


def config0_prompt():
    return np.random.default_rng(1).integers(0, 96, size=16).astype(np.uint32)


def config4(num_layers=12, vocab_size=32000, max_sequence_length=2048):
    return GptConfig(vocab_size=vocab_size, max_sequence_length=max_sequence_length, embed_dim=768,
                     num_heads=12, feed_forward_dim=2048, num_layers=num_layers,
                     layer_norm_epsilon=1e-5, activation="swiglu", weight_dtype="bf16")


def set_model_arrays(model, arrays):
    from .nn import model_parameters
    params = model_parameters(model)
    assert len(params) == len(arrays)
    for p, a in zip(params, arrays):
        p.set_values(a)
