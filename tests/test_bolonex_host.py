"""Bolonex without a GPU: configuration, registry, weight files, and the plain restatement checked mechanism by mechanism
against independent closed forms."""
import json
import os

import numpy as np
import pytest

from oracle import bolonex as plain
from tests.bolonex_util import CONFIGS, bf16_exact, build, random_tensors, tokens_for
from tnsr_b200 import _native
from tnsr_b200.bolonex import Bolonex, BolonexConfig
from tnsr_b200.models import load_model
from tnsr_b200.nn import Backend, TnsrError
from tnsr_b200.parameters import read_safetensors, save_gpt, write_safetensors


def save(directory, cfg, tensors):
    os.makedirs(directory, exist_ok=True)
    with open(os.path.join(directory, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(directory, "model.safetensors"), tensors)


def test_folder_round_trip_through_the_registry(tmp_path):
    cfg = CONFIGS["mixed"]
    tensors = random_tensors(cfg)
    save(tmp_path, cfg, tensors)
    model = load_model(str(tmp_path), "float32")
    assert isinstance(model, Bolonex) and model.config().weight_dtype == "f32"
    assert list(model.named()) == list(model.config().tensor_shapes())
    for name, p in model.named().items():
        assert np.array_equal(p.values().reshape(p.shape), tensors[name])
    assert load_model(str(tmp_path)).config().weight_dtype == "bf16"
    with pytest.raises(TnsrError, match="unknown architecture"):
        save(tmp_path / "b", dict(cfg, architecture="Nothing"), tensors)
        load_model(str(tmp_path / "b"))
    with pytest.raises(TnsrError, match="neither"):
        load_model(str(tmp_path / "nowhere"))
    with pytest.raises(TnsrError, match="unknown dtype"):
        load_model(str(tmp_path), "float16")


def test_registry_reads_the_gpt_archive(tmp_path):
    from tests.helpers import kv_model
    save_gpt(kv_model(8), str(tmp_path))
    model = load_model(str(tmp_path), "float32")
    assert model.config().max_sequence_length == 8 and len(model.parameters()) > 4


def test_safetensors_types_and_errors(tmp_path):
    path = str(tmp_path / "x.safetensors")
    a, b = bf16_exact(np.random.default_rng(0).normal(size=(3, 5)).astype(np.float32)), np.float32([1 / 3, 2.0])
    write_safetensors(path, {"a": a, "b": b, "c": np.int32([[7, -1]])})
    blob = open(path, "rb").read()
    assert b'"BF16"' in blob and b'"F32"' in blob and b'"I32"' in blob
    got = read_safetensors(path)
    assert np.array_equal(got["a"], a) and np.array_equal(got["b"], b) and np.array_equal(got["c"], [[7, -1]])
    open(path, "wb").write(blob[:-3])
    with pytest.raises(TnsrError, match="out of bounds"):
        read_safetensors(path)


def test_configuration_errors():
    cfg = CONFIGS["mixed"]
    tensors = random_tensors(cfg)
    config = BolonexConfig.from_dict(cfg)
    assert [config.owner(i) for i in range(5)] == [0, 1, 2, 0, 1]
    with pytest.raises(TnsrError, match="missing"):
        Bolonex(config, {k: v for k, v in tensors.items() if k != "l0.mix.g"})
    with pytest.raises(TnsrError, match="unexpected"):
        Bolonex(config, dict(tensors, extra=np.zeros(1, np.float32)))
    with pytest.raises(TnsrError, match="expected shape"):
        Bolonex(config, dict(tensors, head=tensors["head"][:-1]))
    bad = json.loads(json.dumps(cfg))
    bad["layers"][3]["weights_of"] = 1
    with pytest.raises(TnsrError, match="same sizes"):
        BolonexConfig.from_dict(bad).tensor_shapes()
    bad["layers"][3]["type"] = "conv"
    with pytest.raises(TnsrError, match="unknown mixer"):
        BolonexConfig.from_dict(bad)
    with pytest.raises(TnsrError, match="malformed"):
        BolonexConfig.from_dict({k: v for k, v in cfg.items() if k != "norm"})


def test_description_handed_to_the_library():
    desc = BolonexConfig.from_dict(CONFIGS["mixed"]).stack()
    assert desc.num_layers == 5 and desc.norm_offset == 1.0 and desc.embedding_scale == 2.0
    a, m, s = desc.layers[0], desc.layers[1], desc.layers[3]
    assert (a.mixer, a.weights_of, a.heads, a.kv_heads, a.dim, a.vdim, a.conv_taps, a.rotary_dims) == (0, -1, 4, 2, 24, 40, 3, 16)
    assert (a.rotary_factor, a.rotary_low, a.rotary_high, a.rotary_original, a.score_softcap) == (6.0, 1.0, 4.0, 64.0, 20.0)
    assert (m.mixer, m.heads, m.vdim, m.state, m.groups, m.norm_groups, m.conv_taps, m.feed_forward) == (1, 6, 24, 40, 3, 2, 2, 80)
    assert s.weights_of == 0


def test_library_rejects_descriptions_it_cannot_serve():
    import ctypes as C
    from tnsr_b200 import build as product
    product.build()
    lib = _native.lib()

    def code(change, **cfg):
        config = BolonexConfig.from_dict(CONFIGS["mixed"])
        desc = config.stack()
        change(desc.layers)
        c = _native.Config(config.vocab_size, 64, config.embed_dim, 1, 1, config.num_layers, 1e-5, 0, 1, 1, cfg.get("batch", 1), 64, 0, 0, 0, 0, 0, 0, 0)
        handle = C.c_void_p()
        return lib.tnsr_b200_decoder_create_stack(C.byref(c), C.byref(desc), C.byref(handle))

    def setting(index, field, value):
        def change(layers):
            setattr(layers[index], field, value)
        return change

    for index, field, value in ((0, "kv_heads", 3), (0, "dim", 257), (0, "rotary_dims", 15), (0, "conv_taps", 0), (0, "conv_taps", 17), (1, "groups", 4),
                                (1, "norm_groups", 5), (1, "state", 257), (2, "mixer", 9), (3, "weights_of", 1), (3, "weights_of", 3), (3, "weights_of", 9),
                                (3, "heads", 2), (0, "rotary_high", 0.5)):
        assert code(setting(index, field, value)) == -1, (field, value)
    assert code(lambda layers: None, batch=0) == -1
    if lib.tnsr_b200_device_count() <= 0:
        assert code(lambda layers: None) == -9      # a sound description gets as far as looking for a device


def test_decoder_refuses_the_cpu_backend():
    _, _, model = build("odd")
    with pytest.raises(TnsrError, match="no CPU executor"):
        model.decoder_with_capacity(Backend.Cpu, 1, 8)


# ---- the plain restatement against closed forms ------------------------------------------------
def test_plain_convolution_is_a_shifted_sum():
    u = np.arange(12.0).reshape(6, 2)
    w = np.array([[0.0, 0.0, 1.0], [2.0, 0.0, 0.0]])
    y = plain.causal_conv(u, w)
    assert np.array_equal(y[:, 0], u[:, 0]) and np.array_equal(y[2:, 1], 2 * u[:4, 1]) and not y[:2, 1].any()


def test_plain_rotation_is_relative_and_leaves_the_rest():
    rot = {"base": 100.0, "dims": 4, "scaling": None}
    rng = np.random.default_rng(0)
    q, k = np.tile(rng.normal(size=(1, 1, 6)), (9, 1, 1)), np.tile(rng.normal(size=(1, 1, 6)), (9, 1, 1))
    a, b = plain.rotate_interleaved(q, rot)[:, 0], plain.rotate_interleaved(k, rot)[:, 0]
    assert np.allclose(a[3] @ b[1], a[8] @ b[6]) and np.array_equal(a[:, 4:], q[:, 0, 4:]) and np.allclose(a[0], q[0, 0])
    z = q[5, 0, 0] + 1j * q[5, 0, 1]      # pair (0, 1) turns by one radian per position
    assert np.allclose(a[5, 0] + 1j * a[5, 1], z * np.exp(5j))


def test_plain_frequency_scaling_has_three_ranges():
    rot = {"base": 1e6, "dims": 32, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 256}}
    f0, f = plain.rotation_frequencies(dict(rot, scaling=None)), plain.rotation_frequencies(rot)
    length = 2 * np.pi / f0
    assert np.allclose(f[length < 64], f0[length < 64]) and np.allclose(f[length > 256], f0[length > 256] / 8)
    between = (length > 64) & (length < 256)
    assert between.any() and np.all(f[between] < f0[between]) and np.all(f[between] > f0[between] / 8)


def test_plain_attention_cap_groups_and_causality():
    q, k = np.ones((3, 4, 2)), np.ones((3, 2, 2))
    v = np.arange(12.0).reshape(3, 2, 2)
    out = plain.attend(q, k, v, 1.0, 5.0)
    assert np.allclose(out[2, 1], v[:, 0].mean(axis=0)) and np.allclose(out[2, 2], v[:, 1].mean(axis=0)) and np.allclose(out[0, 3], v[0, 1])
    k[1] *= 1000.0      # capped: the weight of the outstanding key is at most exp(5 - 5 tanh(2 / 5)) times another one's
    w = np.exp(5.0 * np.tanh(2.0 / 5.0) - 5.0)
    assert np.allclose(plain.attend(q, k, v, 1.0, 5.0)[1, 0], (w * v[0, 0] + v[1, 0]) / (1 + w))


def test_plain_recurrence_equals_its_unrolled_sum():
    rng = np.random.default_rng(3)
    x, b, c = rng.normal(size=(7, 4, 3)), rng.normal(size=(7, 2, 5)), rng.normal(size=(7, 2, 5))
    dt, a_log, d = rng.uniform(0.1, 1, (7, 4)), rng.normal(size=4), rng.normal(size=4)
    y = plain.state_space_scan(x, b, c, dt, a_log, d)
    for h in range(4):
        cum = np.cumsum(-np.exp(a_log[h]) * dt[:, h])
        for i in range(7):
            want = d[h] * x[i, h] + sum(np.exp(cum[i] - cum[j]) * dt[j, h] * (b[j, h // 2] @ c[i, h // 2]) * x[j, h] for j in range(i + 1))
            assert np.allclose(y[i, h], want)


def test_plain_gate_comes_before_the_norm():
    y, z = np.array([[3.0, 4.0, 1.0, 2.0]]), np.array([[50.0, 50.0, -50.0, 50.0]])
    got = plain.gated_group_norm(y, z, np.ones(4), 2, 0.0)
    assert np.allclose(got, [[3 / np.sqrt(12.5), 4 / np.sqrt(12.5), 0.0, np.sqrt(2.0)]])


def test_plain_forward_is_causal_and_shares_tensors():
    cfg, tensors, _ = build("mixed")
    ids = tokens_for(cfg, 12)
    whole, after = plain.forward(cfg, tensors, ids)
    assert np.allclose(plain.forward(cfg, tensors, ids[:7])[0], whole[:7]) and after.shape == (5, 12, 96)
    cfg2 = json.loads(json.dumps(cfg))
    copies = dict(tensors)
    for i, j in ((3, 0), (4, 1)):
        del cfg2["layers"][i]["weights_of"]
        copies.update({f"l{i}." + k[3:]: v for k, v in tensors.items() if k.startswith(f"l{j}.")})
    assert np.array_equal(plain.forward(cfg2, copies, ids)[0], whole)
