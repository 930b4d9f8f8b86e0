"""Ganupel without a GPU: configuration, registry, the description handed to the library, and the plain restatement checked
mechanism by mechanism against independent closed forms."""
import ctypes as C
import json

import numpy as np
import pytest

from oracle import ganupel as plain
from tests.ganupel_util import CONFIGS, build, random_tensors, tokens_for
from tests.test_bolonex_host import save
from tnsr_b200 import _native
from tnsr_b200.ganupel import Ganupel, GanupelConfig
from tnsr_b200.models import load_model
from tnsr_b200.nn import Backend, TnsrError


def changed(cfg, *path):
    out = json.loads(json.dumps(cfg))
    at = out
    for key in path[:-2]:
        at = at[key]
    at[path[-2]] = path[-1]
    return out


def test_folder_round_trip_through_the_registry(tmp_path):
    cfg = CONFIGS["mixed"]
    tensors = random_tensors(cfg)
    save(tmp_path, cfg, tensors)
    model = load_model(str(tmp_path), "float32")
    assert isinstance(model, Ganupel) and model.config().weight_dtype == "f32" and model.config().num_layers == 6
    assert list(model.named()) == list(model.config().tensor_shapes())
    for name, p in model.named().items():
        assert np.array_equal(p.values().reshape(p.shape), tensors[name])
    assert load_model(str(tmp_path)).config().weight_dtype == "bf16"


def test_configuration_errors():
    cfg = CONFIGS["mixed"]
    tensors = random_tensors(cfg)
    config = GanupelConfig.from_dict(cfg)
    with pytest.raises(TnsrError, match="missing"):
        Ganupel(config, {k: v for k, v in tensors.items() if k != "l0.mix.left.pb"})
    with pytest.raises(TnsrError, match="unexpected"):
        Ganupel(config, dict(tensors, extra=np.zeros(1, np.float32)))
    with pytest.raises(TnsrError, match="expected shape"):
        Ganupel(config, dict(tensors, **{"l1.mix.ra": tensors["l1.mix.ra"][:-1]}))
    # a layer without a feed-forward has no use for its norm and scale, but a file may hold them
    Ganupel(config, dict(tensors, **{"l4.norm2": np.zeros(96, np.float32), "l4.ls2": np.ones(96, np.float32)}))
    for path, message in ((("layers", 0, "type", "conv"), "unknown mixer"), (("layers", 0, "mlp", "kind", "gated"), "unknown feed-forward"),
                          (("layers", 0, "mixer", "left", {}), "malformed")):
        with pytest.raises(TnsrError, match=message):
            GanupelConfig.from_dict(changed(cfg, *path))
    with pytest.raises(TnsrError, match="malformed"):
        GanupelConfig.from_dict({k: v for k, v in cfg.items() if k != "norm"})


def test_description_handed_to_the_library():
    desc = GanupelConfig.from_dict(CONFIGS["mixed"]).stack()
    assert desc.num_layers == 6 and desc.norm_offset == 1.0 and desc.embedding_scale == 1.0
    a, r = desc.layers[0], desc.layers[1]
    assert (a.mixer, a.block_form, a.heads, a.kv_heads, a.dim, a.vdim, a.rotary_dims, a.rotary_layout, a.window, a.score_kind) == (2, 1, 4, 2, 24, 40, 16, 1, 19, 1)
    assert (a.rec_heads, a.rec_dim, a.rec_vdim, a.attention_gain, a.recurrent_gain, a.score_scale) == (3, 20, 28, 0.7, 1.2, 0.3)
    assert (a.feed_forward, a.feed_forward_kind, a.experts, a.identity_experts, a.top, a.router_scale) == (40, 2, 5, 2, 3, 1.5)
    assert (r.mixer, r.width, r.blocks, r.conv_taps, r.feed_forward, r.feed_forward_kind) == (3, 72, 3, 3, 112, 1)
    assert desc.layers[4].feed_forward == 0


def test_library_rejects_descriptions_it_cannot_serve():
    from tnsr_b200 import build as product
    product.build()
    lib = _native.lib()

    def code(index=0, **fields):
        config = GanupelConfig.from_dict(CONFIGS["mixed"])
        desc = config.stack()
        for field, value in fields.items():
            setattr(desc.layers[index], field, value)
        c = _native.Config(config.vocab_size, 64, config.embed_dim, 1, 1, config.num_layers, 1e-5, 0, 1, 1, 1, 64, 0, 0, 0, 0, 0, 0, 0)
        return lib.tnsr_b200_decoder_create_stack(C.byref(c), C.byref(desc), C.byref(C.c_void_p()))

    for fields in (dict(rec_dim=257), dict(rec_heads=0), dict(rec_vdim=0), dict(window=3, mixer=0), dict(score_kind=2), dict(rotary_layout=2), dict(top=0),
                   dict(top=8), dict(experts=0), dict(experts=1023), dict(block_form=2), dict(block_form=0), dict(feed_forward_kind=3), dict(mixer=4)):
        assert code(**fields) == -1, fields
    for fields in (dict(blocks=5), dict(blocks=0), dict(width=0), dict(conv_taps=0), dict(conv_taps=17)):
        assert code(1, **fields) == -1, fields
    if lib.tnsr_b200_device_count() <= 0:
        assert code() == -9      # a sound description gets as far as looking for a device


def test_decoder_refuses_the_cpu_backend():
    _, _, model = build("odd")
    with pytest.raises(TnsrError, match="no CPU executor"):
        model.decoder_with_capacity(Backend.Cpu, 1, 8)


# ---- the plain restatement against closed forms ------------------------------------------------
def test_plain_rotation_pairs_the_halves():
    rot = {"base": 100.0, "dims": 4}
    rng = np.random.default_rng(0)
    q, k = np.tile(rng.normal(size=(1, 1, 6)), (9, 1, 1)), np.tile(rng.normal(size=(1, 1, 6)), (9, 1, 1))
    a, b = plain.rotate_halves(q, rot)[:, 0], plain.rotate_halves(k, rot)[:, 0]
    assert np.allclose(a[3] @ b[1], a[8] @ b[6]) and np.array_equal(a[:, 4:], q[:, 0, 4:]) and np.allclose(a[0], q[0, 0])
    for i, f in ((0, 1.0), (1, 0.1)):
        z = q[5, 0, i] + 1j * q[5, 0, i + 2]
        assert np.allclose(a[5, i] + 1j * a[5, i + 2], z * np.exp(5j * f))
    assert plain.rotate_halves(q, {"base": 100.0, "dims": 0}) is q


def test_plain_attention_counts_the_window_and_does_not_normalise():
    q, k, v = np.zeros((6, 2, 3)), np.zeros((6, 1, 3)), np.arange(6.0).reshape(6, 1, 1)
    out = plain.sigmoid_attend(q, k, v, 1.0, np.array([0.0, -np.log(3.0)]), 3)
    assert np.allclose(out[5, 0], 0.5 * (3 + 4 + 5)) and np.allclose(out[5, 1], 0.25 * (3 + 4 + 5)) and np.allclose(out[1, 0], 0.5)
    k[2] = 1e3                        # one saturated key, three others at sigmoid(0)
    q[:] = 1.0
    assert np.allclose(plain.sigmoid_attend(q, k, v, 1.0, np.zeros(2), 4)[5, 0], 2 + 0.5 * (3 + 4 + 5))


def test_plain_gated_scan_equals_its_unrolled_sum():
    rng = np.random.default_rng(3)
    q, f, v = rng.normal(size=(7, 2, 5)), rng.uniform(0.05, 1, (7, 2, 5)), rng.normal(size=(7, 2, 3))
    o = plain.gated_scan(q, f, v)
    for h in range(2):
        for i in range(7):
            want = sum((q[i, h] * (1 - f[j, h]) * np.prod(f[j + 1:i + 1, h], axis=0)).sum() * v[j, h] for j in range(i + 1))
            assert np.allclose(o[i, h], want)


def test_plain_linear_unit_keeps_its_variance_and_forgets():
    u, one = np.full((40, 1), 2.0), np.ones((40, 1))
    lam = np.array([np.log(np.expm1(np.log(2.0) / 8.0))])          # a = 1/2 where r = 1
    s = plain.linear_unit_scan(u, one, one, lam)
    gain = np.sqrt(0.75)
    assert np.allclose(s[0], 2 * gain) and np.allclose(s[1], 2 * gain * 1.5) and np.allclose(s[-1], 2 * gain * 2)
    assert np.allclose(plain.linear_unit_scan(u, one * 0, one, lam), 0.0)     # r = 0: nothing is forgotten, nothing written


def test_plain_block_diagonal_is_one_large_matrix():
    rng = np.random.default_rng(4)
    w, b, u = rng.normal(size=(3, 4, 4)), rng.normal(size=(3, 4)), rng.normal(size=(5, 12))
    full = np.zeros((12, 12))
    for i in range(3):
        full[4 * i:4 * i + 4, 4 * i:4 * i + 4] = w[i]
    assert np.allclose(plain.block_diagonal(u, w, b), u @ full.T + b.reshape(-1))


def test_plain_poly_norm_of_a_constant_and_of_one_spike():
    assert np.allclose(plain.poly_norm(np.full((1, 9), -3.0), [0.5, 0.25, 2.0, 0.125], 0.0), -0.5 + 0.25 - 2.0 + 0.125)
    z = np.zeros((1, 16))
    z[0, 3] = 5.0                                                    # rms of every power is the power / 4
    assert np.allclose(plain.poly_norm(z, [1.0, 10.0, 100.0, 0.0], 0.0)[0], np.where(np.arange(16) == 3, 444.0, 0.0))


def test_plain_router_corrects_the_choice_but_not_the_weights():
    h, w = np.eye(4), np.diag([3.0, 2.0, 1.0, 0.0])
    router = {"experts": 3, "identity": 1, "top": 2, "scale": 1.5}
    s = np.exp([3.0, 0, 0, 0]) / np.exp([3.0, 0, 0, 0]).sum()
    chosen, weights = plain.route(h[:1], router, w, np.zeros(4))
    assert list(chosen[0]) == [0, 1] and np.allclose(weights[0], 1.5 * s[:2] / s[:2].sum())
    chosen, weights = plain.route(h[:1], router, w, np.array([0.0, 0, 0, 5.0]))
    assert list(chosen[0]) == [3, 0] and np.allclose(weights[0], 1.5 * s[[3, 0]] / (s[3] + s[0]))
    t = {"router": w, "correction": np.array([0.0, 0, 0, 5.0])}
    t.update({f"e{e}.{n}": np.eye(4) * (e + 1) for e in range(3) for n in ("up", "down")})
    out = plain.mixture(-h[:1], {"router": router}, t, 0.0)          # relu^2 of a negative row: the identity expert alone
    _, weights = plain.route(-h[:1], router, w, t["correction"])
    assert np.allclose(out, -weights[0, 0] * h[:1])


def test_plain_forward_is_causal():
    for name in sorted(CONFIGS):
        cfg, tensors, _ = build(name)
        ids = tokens_for(cfg, 12)
        whole, after = plain.forward(cfg, tensors, ids)
        assert np.allclose(plain.forward(cfg, tensors, ids[:7])[0], whole[:7]) and after.shape == (len(cfg["layers"]), 12, cfg["width"])
