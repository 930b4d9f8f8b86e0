"""Bolonex on the GPU against the plain restatement (oracle/bolonex.py): the operators alone, whole prompts, decoding
through the caches, portions, batches of unequal sessions, reused slots and pages, shared tensors, generation, the trace
program and the command line."""
import ctypes as C
import json
import os
import subprocess
import sys

import numpy as np
import pytest

pytestmark = pytest.mark.gpu

torch = pytest.importorskip("torch")

from oracle import bolonex as plain  # noqa: E402
from tests.bolonex_util import CONFIGS, SCALING, attention, bf16_exact, build, config, mamba2, row_errors, tokens_for  # noqa: E402
from tests.gpu_util import dev, lib, ok, ptr, rel_err, stream  # noqa: E402
from tests.test_bolonex_host import save  # noqa: E402
from tnsr_b200 import _native  # noqa: E402
from tnsr_b200.nn import Backend, GptDecoderOptions, GptPrefillMode, TnsrError  # noqa: E402
from tnsr_b200.session import B200Session  # noqa: E402

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32, BF16 = 0, 1
TORCH = {F32: torch.float32, BF16: torch.bfloat16}
# f32: rounding of sums only.  bf16: activations of every product and cache row carry 8 bits, through sharp attention.
LIMIT = {"f32": 5e-5, "bf16": 0.06}


def place(sessions, chunk, position=0, positions=None):
    return _native.Place(sessions, chunk, position, 0, positions.data_ptr() if positions is not None else None)


# ---- operators -------------------------------------------------------------------------------------
@pytest.mark.parametrize("width", [64, 96, 1000, 1024, 1030, 2048, 7])
@pytest.mark.parametrize("offset", [0.0, 1.0])
def test_rmsnorm(width, offset):
    rng = np.random.default_rng(width)
    x, w = rng.normal(size=(9, width)).astype(np.float32) * 3, rng.normal(size=width).astype(np.float32)
    want = plain.rms(x.astype(np.float64), 1e-3) * (offset + w)
    for dtype, tol in ((F32, 2e-6), (BF16, 5e-3)):
        out = torch.empty((9, width), dtype=TORCH[dtype], device="cuda")
        ok(lib().tnsr_b200_rmsnorm(ptr(dev(x)), ptr(dev(w)), offset, ptr(out), 9, width, 1e-3, dtype, stream()))
        torch.cuda.synchronize()
        assert rel_err(out.float().cpu().numpy(), want) < tol


def test_gelu_tanh_epilogue():
    rng = np.random.default_rng(5)
    a, b = bf16_exact(rng.normal(size=(40, 64)).astype(np.float32)), bf16_exact(rng.normal(size=(96, 64)).astype(np.float32) * 0.4)
    out = torch.empty((40, 96), dtype=torch.float32, device="cuda")
    ok(lib().tnsr_b200_gemm_bf16(ptr(dev(a, torch.bfloat16)), ptr(dev(b, torch.bfloat16)), None, None, ptr(out), 40, 96, 64, 3, F32, stream()))
    torch.cuda.synchronize()
    assert rel_err(out.cpu().numpy(), plain.gelu_tanh(a.astype(np.float64) @ b.T.astype(np.float64))) < 1e-5


def run_attention(q, k, v, gate, positions, heads, kv_heads, scale, softcap, dtype, engine=0, workspace=True, poison=True):
    """q [s, chunk, H, dim]; k, v [s, capacity, G, width] with the rows past a session's end poisoned."""
    s, chunk, _, dim = q.shape
    capacity, vdim = k.shape[1], v.shape[3]
    k, v = k.copy(), v.copy()
    if poison:
        for i, p in enumerate(positions):
            k[i, p + chunk:] = np.nan
            v[i, p + chunk:] = np.nan
    out_cols = heads * vdim + 3
    out_ld = (out_cols + 7) // 8 * 8
    out = torch.full((s * chunk, out_ld), 7.0, dtype=TORCH[dtype], device="cuda")
    size = lib().tnsr_b200_grouped_attention_workspace(dim, vdim)
    ws = torch.zeros(size, dtype=torch.uint8, device="cuda")
    d = [dev(x.astype(np.float32), TORCH[dtype]) for x in (q, k, v)]
    g = dev(np.ascontiguousarray(gate, dtype=np.float32))
    args = _native.GroupedAttentionArgs(d[0].data_ptr(), d[1].data_ptr(), d[2].data_ptr(), g.data_ptr(), out.data_ptr(),
                                        ws.data_ptr() if workspace else None, None, size if workspace else 0, heads, kv_heads, dim, vdim, capacity,
                                        gate.shape[-1], out_ld, out_cols, scale, softcap or 0.0, dtype, engine)
    pos = dev(np.asarray(positions, np.uint32).view(np.int32))
    where = place(s, chunk, positions[0]) if len(set(positions)) == 1 else place(s, chunk, positions=pos)
    results = []
    for _ in range(2):       # twice: merge counters must come back to zero
        ok(lib().tnsr_b200_grouped_attention(C.byref(args), C.byref(where), stream()))
        torch.cuda.synchronize()
        results.append(out.float().cpu().numpy())
    assert np.array_equal(results[0], results[1])
    assert np.all(results[0][:, heads * vdim:out_cols] == 0.0) and np.all(results[0][:, out_cols:] == 7.0)
    return results[0][:, :heads * vdim].reshape(s, chunk, heads, vdim)


def attention_case(seed, positions, chunk, capacity, heads, kv_heads, dim, vdim, planted=None):
    """Random rows (bf16-exact); planted = (key position, query index): that key of every session is aligned with that
    query of every head, so that its score stands out of all others."""
    rng = np.random.default_rng(seed)
    s = len(positions)
    q = rng.normal(size=(s, chunk, heads, dim)) * 0.5
    k = rng.normal(size=(s, capacity, kv_heads, dim)) * 0.5
    v = rng.normal(size=(s, capacity, kv_heads, vdim))
    if planted is not None:
        key, query = planted
        u = rng.normal(size=dim)
        q[:, query] = u * 2.0
        k[:, key] = u * 2.0
    gate = rng.normal(size=(s * chunk, heads + 2))
    return [bf16_exact(x.astype(np.float32)) for x in (q, k, v)] + [gate.astype(np.float32)]


def expected_attention(q, k, v, gate, positions, scale, softcap):
    out = np.zeros(q.shape[:3] + (v.shape[3],))
    s, chunk, heads = q.shape[:3]
    for i, p in enumerate(positions):
        n = p + chunk
        full = np.zeros((n, heads, q.shape[3]))
        full[p:] = q[i]
        out[i] = plain.attend(full, k[i, :n].astype(np.float64), v[i, :n].astype(np.float64), scale, softcap)[p:]
        out[i] *= plain.sigmoid(gate.astype(np.float64).reshape(s, chunk, -1)[i, :, :heads])[:, :, None]
    return out


SHAPES = [(4, 2, 64, 64), (6, 2, 40, 24), (8, 1, 128, 128), (3, 3, 10, 7), (2, 1, 200, 136), (12, 1, 16, 32), (20, 1, 64, 48)]


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("chunk,positions", [(1, (0, 37, 200, 15)), (2, (0, 14, 63)), (5, (11, 0)), (64, (0, 5)), (131, (0, 70)), (33, (31, 32))])
def test_grouped_attention(shape, chunk, positions):
    heads, kv_heads, dim, vdim = shape
    for softcap in (8.0, None):
        case = attention_case(chunk + dim, positions, chunk, 256, heads, kv_heads, dim, vdim)
        want = expected_attention(*case, positions, 0.3, softcap)
        got = run_attention(*case, positions, heads, kv_heads, 0.3, softcap, BF16)
        assert rel_err(got, want) < 4e-3
        assert rel_err(run_attention(*case, positions, heads, kv_heads, 0.3, softcap, BF16, engine=1), want) < 4e-3
        assert rel_err(run_attention(*case, positions, heads, kv_heads, 0.3, softcap, F32), want) < 2e-6


@pytest.mark.parametrize("heads,kv_heads", [(4, 2), (3, 3), (12, 1)])
@pytest.mark.parametrize("softcap", [6.0, None])
def test_long_chunks_on_every_engine(heads, kv_heads, softcap):
    """Heads of 64 at a position the host knows: the tcgen05 kernel (engine 0) and the warp-level one (2), whole and ragged
    query tiles, positions around key blocks."""
    for chunk, position in ((32, 0), (33, 1), (127, 0), (128, 128), (129, 63), (200, 100), (256, 127), (40, 300)):
        positions = (position, position)
        case = attention_case(chunk, positions, chunk, position + chunk + 3, heads, kv_heads, 64, 64)
        want = expected_attention(*case, positions, 0.4, softcap)
        for engine in (0, 2):
            assert rel_err(run_attention(*case, positions, heads, kv_heads, 0.4, softcap, BF16, engine=engine), want) < 6e-3, (chunk, position, engine)


@pytest.mark.parametrize("engine", [0, 2])
@pytest.mark.parametrize("dim,vdim", [(64, 64), (72, 40)])
def test_grouped_attention_finds_one_outstanding_key_anywhere(dim, vdim, engine):
    """One planted key must carry its query's output wherever it lies: first rows, tile borders, the query itself."""
    for total, chunk in ((400, 1), (400, 3), (200, 130)):
        position = total - chunk
        for key in (0, 1, 15, 16, 17, 63, 64, 65, 127, 128, position - 1, position, total - 1):
            query = chunk - 1
            case = attention_case(key, (position,), chunk, 416, 4, 2, dim, vdim, planted=(key, query))
            got = run_attention(*case, (position,), 4, 2, 0.5, 100.0, BF16, engine=engine)
            want = expected_attention(*case, (position,), 0.5, 100.0)
            assert rel_err(got, want) < 4e-3, (total, chunk, key)
            gate = plain.sigmoid(case[3][query, :4].astype(np.float64))
            seen = want[0, query] / gate[:, None]
            assert np.abs(seen - case[2][0, key, [0, 0, 1, 1]]).max() < 0.05      # the case does what it says
    # a key just past the query stays out: planted at the next row, the output is that of a case without it
    case = attention_case(9, (20,), 40, 416, 4, 2, dim, vdim, planted=(50, 29))     # query 29 stands at 49
    want = expected_attention(*case, (20,), 0.5, 100.0)
    assert rel_err(run_attention(*case, (20,), 4, 2, 0.5, 100.0, BF16, engine=engine), want) < 4e-3
    assert np.abs(want[0, 29]).max() < 2.0


def test_grouped_attention_without_workspace_and_large_scores():
    case = attention_case(3, (250,), 1, 256, 8, 2, 64, 64)
    want = expected_attention(*case, (250,), 20.0, 30.0)
    assert rel_err(run_attention(*case, (250,), 8, 2, 20.0, 30.0, BF16, workspace=False), want) < 4e-3
    assert rel_err(run_attention(*case, (250,), 8, 2, 20.0, 30.0, BF16), want) < 4e-3


def run_mamba2(shape, u, t, portions, dtype, engine=0, positions=None, state=None):
    """Feeds the projected rows u [s, n, cols] (z | x | B | C | dt) in portions; returns (out [s, n, inner], final state)."""
    heads, vdim, n_state, groups, norm_groups, taps = shape
    inner, gn = heads * vdim, groups * n_state
    channels, proj = inner + 2 * gn, 2 * inner + 2 * gn
    s, n, _ = u.shape
    ld = (proj + 31) // 32 * 32
    ring, ssm = state if state else (torch.full((s, taps, channels), float("nan"), dtype=TORCH[dtype], device="cuda"),
                                     torch.full((s, heads, n_state, vdim), float("nan"), dtype=torch.float32, device="cuda"))
    w = {k: dev(np.ascontiguousarray(v, dtype=np.float32)) for k, v in t.items()}
    outs, at = [], 0
    for chunk in portions:
        part = u[:, at:at + chunk]
        rows = np.zeros((s * chunk, ld), np.float32)
        rows[:, :proj] = part[:, :, :proj].reshape(s * chunk, proj)
        d_rows = dev(rows, TORCH[dtype])
        d_dt = dev(np.ascontiguousarray(part[:, :, proj:].reshape(s * chunk, heads), dtype=np.float32))
        out_ld = (inner + 7) // 8 * 8
        out = torch.full((s * chunk, out_ld), 7.0, dtype=TORCH[dtype], device="cuda")
        xbc = torch.empty((s * chunk, channels), dtype=TORCH[dtype], device="cuda")
        gated = torch.empty((s * chunk, inner), dtype=TORCH[dtype], device="cuda")
        args = _native.Mamba2Args(d_rows.data_ptr(), d_dt.data_ptr(), w["conv"].data_ptr(), w["conv.b"].data_ptr(), w["dt_bias"].data_ptr(),
                                  w["A_log"].data_ptr(), w["D"].data_ptr(), w["norm"].data_ptr(), ring.data_ptr(), ssm.data_ptr(), xbc.data_ptr(),
                                  gated.data_ptr(), out.data_ptr(), ld, heads, heads, vdim, n_state, groups, norm_groups, taps, out_ld, out_ld,
                                  1e-5, dtype, engine, 0)
        pos = dev((np.asarray(positions or [0] * s) + at).astype(np.uint32).view(np.int32))
        ok(lib().tnsr_b200_mamba2(C.byref(args), C.byref(place(s, chunk, positions=pos)), stream()))
        torch.cuda.synchronize()
        o = out.float().cpu().numpy()
        assert np.all(o[:, inner:] == 0.0)
        outs.append(o[:, :inner].reshape(s, chunk, inner))
        at += chunk
    return np.concatenate(outs, axis=1), (ring, ssm)


def mamba2_case(shape, s, n, seed=0):
    heads, vdim, n_state, groups, norm_groups, taps = shape
    rng = np.random.default_rng(seed)
    inner, gn = heads * vdim, groups * n_state
    u = bf16_exact(rng.normal(size=(s, n, 2 * inner + 2 * gn + heads)).astype(np.float32))
    t = {"conv": rng.normal(0, 0.3, (inner + 2 * gn, taps)) + (np.arange(taps) == taps - 1), "conv.b": rng.normal(0, 0.3, inner + 2 * gn),
         "dt_bias": rng.uniform(-4, 0.5, heads), "A_log": rng.uniform(-3, 0.7, heads), "D": rng.uniform(0.3, 1.2, heads),
         "norm": rng.uniform(0.5, 1.5, inner)}
    return u, {k: bf16_exact(v.astype(np.float32)) for k, v in t.items()}


def expected_mamba2(shape, u, t):
    """The mixer of the plain restatement with identity projections."""
    heads, vdim, n_state, groups, norm_groups, taps = shape
    inner = heads * vdim
    m = dict(heads=heads, vdim=vdim, state=n_state, groups=groups, norm_groups=norm_groups)
    weights = {k: v.astype(np.float64) for k, v in t.items()}
    weights.update({"in": np.eye(u.shape[2]), "o": np.eye(inner)})
    return np.stack([plain.mamba2_mixer(x.astype(np.float64), m, weights, 1e-5) for x in u])


MAMBA_SHAPES = [(4, 64, 128, 2, 4, 4), (3, 24, 40, 3, 1, 2), (2, 7, 5, 1, 2, 5), (2, 136, 200, 1, 1, 3), (2, 32, 64, 1, 1, 1), (8, 16, 16, 4, 2, 9)]


@pytest.mark.parametrize("shape", MAMBA_SHAPES)
def test_mamba2_portions_and_tokens(shape):
    n = 150
    u, t = mamba2_case(shape, 2, n)
    want = expected_mamba2(shape, u, t)
    for portions in ([n], [64, 64, 22], [63, 65, 22], [1] * 9 + [2, 3, 16, 17, 40, 1, 1, 61], [2] * 75):
        got, state = run_mamba2(shape, u, t, portions, BF16)
        # a norm over few nearly cancelled values magnifies rounding: the mean is tight, the maximum is not
        assert np.sqrt(np.mean((got - want) ** 2)) < 5e-3 * np.std(want) and rel_err(got, want) < 3e-2, portions
        got32, state32 = run_mamba2(shape, u, t, portions, F32)
        assert rel_err(got32, want) < 1e-5, portions
        # the carried state is f32 in both; its inputs x, B are bf16 in one
        assert rel_err(state[1].cpu().numpy(), state32[1].cpu().numpy()) < 6e-3
    token_by_token, _ = run_mamba2(shape, u, t, [n], BF16, engine=1)
    assert rel_err(run_mamba2(shape, u, t, [n], BF16)[0], token_by_token) < 2e-2


def test_mamba2_state_keeps_32_bits_over_a_long_run():
    """Slow decay over 600 tokens: the chunked scan and the token kernel must agree to more than bf16 has."""
    shape = (2, 64, 64, 1, 1, 4)
    u, t = mamba2_case(shape, 1, 600, seed=4)
    t["A_log"][:], t["dt_bias"][:] = -6.0, -2.0
    _, scan = run_mamba2(shape, u, t, [600], BF16)
    _, token = run_mamba2(shape, u, t, [600], BF16, engine=1)
    assert rel_err(scan[1].cpu().numpy(), token[1].cpu().numpy()) < 2e-5


def test_mamba2_session_at_position_zero_ignores_what_its_slot_holds():
    shape = (3, 24, 40, 3, 1, 4)
    u, t = mamba2_case(shape, 2, 20)
    want = expected_mamba2(shape, u, t)
    for portions in ([20], [1, 1, 1, 17], [3, 17]):
        _, used = run_mamba2(shape, u[::-1].copy(), t, [20], F32)
        assert rel_err(run_mamba2(shape, u, t, portions, F32, state=used)[0], want) < 1e-5


# ---- whole models --------------------------------------------------------------------------------------
def logits_of(decoder, ids, portions=None):
    vocab = decoder._model.config().vocab_size
    decoder.reset()
    out, at = [], 0
    for n in portions or [len(ids)]:
        out.append(decoder.decode(ids[at:at + n]).reshape(n, vocab))
        at += n
    assert at == len(ids)
    return np.concatenate(out)


PORTIONS = [[2] * 10 + [80, 1, 1, 68], [1] * 40 + [130], [7, 16, 17, 31, 32, 33, 34], [64, 2, 64, 2, 38], [15, 155], [168, 2]]


@pytest.mark.parametrize("name", sorted(CONFIGS))
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_prompt_decoding_and_portions(name, dtype):
    cfg, tensors, model = build(name, dtype)
    ids = tokens_for(cfg, 170)
    want, _ = plain.forward(cfg, tensors, ids)
    decoder = model.decoder_with_capacity(Backend.Cuda, 1, 170)
    whole = logits_of(decoder, ids)
    assert row_errors(whole, want).max() < LIMIT[dtype]
    for portions in PORTIONS:
        got = logits_of(decoder, ids, portions)
        assert row_errors(got, want).max() < LIMIT[dtype], portions
    # one token, and a prompt that fills the capacity exactly
    assert row_errors(logits_of(decoder, ids[:1]), want[:1]).max() < LIMIT[dtype]


@pytest.mark.parametrize("name", ["mixed", "even"])
def test_scalar_prefill_is_the_same_function(name):
    cfg, tensors, model = build(name, "bf16")
    ids = tokens_for(cfg, 90)
    want, _ = plain.forward(cfg, tensors, ids)
    decoder = model.decoder_with_options(Backend.Cuda, 1, 90, GptDecoderOptions(prefill=GptPrefillMode.Scalar))
    assert row_errors(logits_of(decoder, ids), want).max() < LIMIT["bf16"]


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_each_constant_matters(dtype):
    """A change of any constant of the configuration must show in the logits far above the comparison's limit."""
    base = config(64, 101, [attention(4, 2, 16, 24, conv=3, rot=12, scaling=dict(SCALING, original=32), softcap=6.0, ff=48),
                            mamba2(4, 16, 24, groups=2, norm_groups=2, ff=48)], scale=1.5, eps=1e-2)
    cfg, tensors, model = build(base, dtype)
    ids = tokens_for(cfg, 60)
    want, _ = plain.forward(cfg, tensors, ids)
    got = logits_of(model.decoder_with_capacity(Backend.Cuda, 1, 60), ids)
    assert row_errors(got, want).max() < LIMIT[dtype]
    changes = {"embedding.scale": ("embedding", "scale", 1.0), "eps": ("norm", "eps", 1e-5)}
    for path in (("softcap", 12.0), ("scale", 0.4)):
        changes[path[0]] = ("layers", 0, "mixer", path[0], path[1])
    for key, value in (("base", 900.0), ("dims", 8)):
        changes["rot." + key] = ("layers", 0, "mixer", "rot", key, value)
    for key, value in (("factor", 2.0), ("low", 2.0), ("high", 16.0), ("original", 200)):
        changes["scaling." + key] = ("layers", 0, "mixer", "rot", "scaling", key, value)
    changes["norm_groups"] = ("layers", 1, "mixer", "norm_groups", 4)
    for label, path in changes.items():
        other = json.loads(json.dumps(cfg))
        at = other
        for key in path[:-2]:
            at = at[key]
        at[path[-2]] = path[-1]
        wrong, _ = plain.forward(other, tensors, ids)
        assert row_errors(wrong, want).max() > (20 if dtype == "f32" else 0.2) * LIMIT[dtype], label
        from tnsr_b200.bolonex import Bolonex, BolonexConfig
        follows = logits_of(Bolonex(BolonexConfig.from_dict(other, dtype), tensors).decoder_with_capacity(Backend.Cuda, 1, 60), ids)
        assert row_errors(follows, wrong).max() < LIMIT[dtype], label


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_planted_far_token_decides(dtype):
    """q and k of one layer depend on the token alone, and the last token's query matches one earlier token's key only:
    wherever that token lies, the logits must follow its value."""
    cfg, tensors, model = build(config(64, 50, [attention(2, 1, 32, 32, conv=2, rot=0, softcap=90.0)]), dtype)
    rng = np.random.default_rng(2)
    e = rng.normal(size=(50, 64))
    e[7, :32] = 6.0 * np.sign(e[7, :32])
    e[9] = e[7]
    e[9, 32:] = rng.normal(size=32)
    tensors = dict(tensors)
    tensors["embed"] = bf16_exact(e.astype(np.float32))
    w = np.concatenate([np.eye(32), np.zeros((32, 32))], axis=1)
    tensors["l0.mix.k"], tensors["l0.mix.q"] = bf16_exact(w.astype(np.float32)), bf16_exact(np.concatenate([w, w]).astype(np.float32))
    for name in ("q", "k"):
        tensors[f"l0.mix.{name}.b"] = np.zeros_like(tensors[f"l0.mix.{name}.b"])
        tensors[f"l0.mix.{name}.norm"] = np.full(32, 3.5, np.float32)
        conv = np.zeros_like(tensors[f"l0.mix.{name}.conv"])
        conv[:, -1] = 1.0
        tensors[f"l0.mix.{name}.conv"] = conv
    tensors["l0.mix.o"] = bf16_exact(tensors["l0.mix.o"] * 24)      # the mixer, not the embedding, makes the logits
    from tnsr_b200.bolonex import Bolonex, BolonexConfig
    model = Bolonex(BolonexConfig.from_dict(cfg, dtype), tensors)
    decoder = model.decoder_with_capacity(Backend.Cuda, 1, 300)
    filler = [int(x) for x in rng.integers(10, 50, 300)]
    without, _ = plain.forward(cfg, tensors, filler[:299] + [7])
    for at in (0, 1, 15, 16, 63, 64, 128, 255, 256, 297):
        ids = list(filler[:299]) + [7]
        ids[at] = 9
        want, _ = plain.forward(cfg, tensors, ids)
        assert row_errors(want[-1:], without[-1:]).max() > 0.15
        for portions in ([300], [299, 1], [256, 42, 2]):
            assert row_errors(logits_of(decoder, ids, portions)[-1:], want[-1:]).max() < LIMIT[dtype] / 2, (at, portions)


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_long_decoding(dtype):
    cfg, tensors, model = build("mixed", dtype)
    ids = tokens_for(cfg, 420)
    want, _ = plain.forward(cfg, tensors, ids)
    decoder = model.decoder_with_capacity(Backend.Cuda, 1, 420)
    got = logits_of(decoder, ids, [5] + [1] * 415)
    assert row_errors(got, want).max() < LIMIT[dtype]
    with pytest.raises(TnsrError, match="capacity exceeded"):
        decoder.decode([1])


@pytest.mark.parametrize("name", ["mixed", "even", "odd"])
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_rectangular_batch_equals_each_session_alone(name, dtype):
    cfg, tensors, model = build(name, dtype)
    rows = [tokens_for(cfg, 60, seed=i) for i in range(5)]
    decoder = model.decoder_with_capacity(Backend.Cuda, 5, 64)
    vocab = cfg["vocab"]
    parts = []
    for a, b in ((0, 33), (33, 34), (34, 36), (36, 60)):
        parts.append(decoder.decode([t for r in rows for t in r[a:b]]).reshape(5, b - a, vocab))
    got = np.concatenate(parts, axis=1)
    for i, r in enumerate(rows):
        assert row_errors(got[i], plain.forward(cfg, tensors, r)[0]).max() < LIMIT[dtype]


@pytest.mark.parametrize("paged", [False, True])
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_unequal_sessions_slots_and_pages_used_again(paged, dtype):
    """Ragged steps: sessions start, end and are replaced at different times; every logits row must be that of the
    session alone.  The pool has fewer pages than slots x capacity."""
    cfg, tensors, model = build("mixed", dtype)
    config_ = model.config()
    kw = dict(kv_page_rows=16, kv_pool_pages=11) if paged else {}
    sess = B200Session(config_, 3, 96, logits_mode="all", **kw)
    for i, p in enumerate(model.parameters()):
        sess.refresh(i, p.values())
    lengths = [50, 17, 33, 64, 16, 40, 65, 1]
    requests = [tokens_for(cfg, n, seed=20 + i) for i, n in enumerate(lengths)]
    want = [plain.forward(cfg, tensors, r)[0] for r in requests]
    waiting, slots, at = list(range(len(requests))), [None] * 3, [0] * 3
    spare = sess.free_pages() if paged else 0
    worst = 0.0
    for _ in range(400):
        for b in range(3):
            if slots[b] is None and waiting:
                slots[b], at[b] = waiting.pop(0), 0
        if not any(x is not None for x in slots):
            break
        tokens = [requests[slots[b]][at[b]] if slots[b] is not None else 0 for b in range(3)]
        logits, _ = sess.decode_ragged(np.array(tokens), np.array([at[b] if slots[b] is not None else 0 for b in range(3)]))
        logits = logits.reshape(3, -1)
        for b in range(3):
            if slots[b] is None:
                if paged:
                    sess.release(b)
                continue
            worst = max(worst, row_errors(logits[b:b + 1], want[slots[b]][at[b]:at[b] + 1])[0])
            at[b] += 1
            if at[b] == len(requests[slots[b]]):
                slots[b] = None
                if paged:
                    sess.release(b)
    assert not waiting and worst < LIMIT[dtype] * 1.5
    if paged:
        assert sess.free_pages() == spare
    sess.close()


def test_paged_prompts():
    cfg, tensors, model = build("even", "bf16")
    ids = tokens_for(cfg, 150)
    want, _ = plain.forward(cfg, tensors, ids)
    sess = B200Session(model.config(), 1, 160, logits_mode="all", kv_page_rows=32)
    for i, p in enumerate(model.parameters()):
        sess.refresh(i, p.values())
    runs = []
    for _ in range(2):       # the second time on pages that were given back
        out, at = [], 0
        for n in (100, 1, 1, 48):
            out.append(sess.decode_full(np.array([ids[at:at + n]]), at)[0].reshape(n, -1))
            at += n
        runs.append(np.concatenate(out))
        assert row_errors(runs[-1], want).max() < LIMIT["bf16"]
        sess.release(0)
    assert np.array_equal(runs[0], runs[1])
    sess.close()


def test_replayed_steps_have_the_bits_of_direct_ones(monkeypatch):
    cfg, _, model = build("even", "bf16")
    ids = tokens_for(cfg, 60)
    graph = logits_of(model.decoder_with_capacity(Backend.Cuda, 1, 64), ids, [20] + [1] * 40)
    monkeypatch.setenv("TNSR_B200_NO_GRAPH", "1")
    monkeypatch.setenv("TNSR_B200_NO_PDL", "1")
    assert np.array_equal(graph, logits_of(model.decoder_with_capacity(Backend.Cuda, 1, 64), ids, [20] + [1] * 40))


def greedy(cfg, tensors, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(np.argmax(plain.forward(cfg, tensors, ids)[0][-1])))
    return ids


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_greedy_generation(name):
    cfg, tensors, model = build(name, "f32")
    prompt = tokens_for(cfg, 11)
    want = greedy(cfg, tensors, prompt, 20)
    assert model.generate_cached(Backend.Cuda, prompt, 20) == want
    assert model.generate(Backend.Cuda, prompt, 6) == want[:17]
    assert np.array_equal(model.forward(Backend.Cuda, [want[:20]])[0, -1].argmax(), want[20])


@pytest.mark.parametrize("mode", ["none", "last"])
def test_device_greedy_and_sampling_follow_the_logits(mode):
    from oracle.sampler import sample_row
    cfg, tensors, model = build("even", "bf16")
    prompts = np.array([tokens_for(cfg, 12, seed=s) for s in range(3)])
    full = model.decoder_with_capacity(Backend.Cuda, 3, 32)
    sess = B200Session(model.config(), 3, 32, logits_mode=mode)
    for i, p in enumerate(model.parameters()):
        sess.refresh(i, p.values())
    for sampled in (False, True):
        full.reset()
        sess.reset()
        if sampled:
            sess.set_sampler(0.8, 5, 1234)
        logits = full.decode(prompts.reshape(-1).tolist()).reshape(3, 12, -1)[:, -1]
        _, ids = sess.decode_full(prompts, 0)
        for step in range(8):
            expect = [sample_row(logits[b], 0.8, 5, 1234, 12 + step, b) if sampled else int(np.argmax(logits[b])) for b in range(3)]
            assert list(ids) == expect
            logits = full.decode([int(t) for t in ids]).reshape(3, -1)
            _, ids = sess.decode_full(ids.reshape(3, 1), 12 + step)
    sess.close()


def test_saved_state_continues_with_the_same_bits(tmp_path):
    for dtype in ("bf16", "f32"):
        cfg, _, model = build("mixed", dtype)
        ids = tokens_for(cfg, 40)
        a = model.decoder_with_capacity(Backend.Cuda, 1, 48)
        a.decode(ids[:30])
        a.save_state(str(tmp_path / dtype))
        want = np.concatenate([a.decode(ids[30:31]), a.decode(ids[31:])])
        b = model.decoder_with_capacity(Backend.Cuda, 1, 48)
        b.load_state(str(tmp_path / dtype))
        assert b.len() == 30
        assert np.array_equal(np.concatenate([b.decode(ids[30:31]), b.decode(ids[31:])]), want)


def test_weights_uploaded_again_take_effect():
    cfg, tensors, model = build("mixed", "f32")
    ids = tokens_for(cfg, 20)
    decoder = model.decoder_with_capacity(Backend.Cuda, 1, 20)
    logits_of(decoder, ids)
    changed = dict(tensors)
    for name in ("l0.mix.v.b", "l1.mix.in", "l0.mlp.down", "head"):
        changed[name] = bf16_exact(tensors[name] * 1.5 + 0.01)
        model.named()[name].set_values(changed[name])
    assert row_errors(logits_of(decoder, ids), plain.forward(cfg, changed, ids)[0]).max() < LIMIT["f32"]


def test_trace_program(tmp_path):
    cfg, tensors, _ = build("mixed")
    save(tmp_path / "model", cfg, tensors)
    requests = {"x": tokens_for(cfg, 41, seed=5), "y": tokens_for(cfg, 9, seed=6)}
    want = {k: plain.forward(cfg, tensors, v)[0] for k, v in requests.items()}
    steps, expect = [], []
    for rid, cuts in (("x", [20, 1, 1, 2, 17]), ("y", [9])):
        at = 0
        for n in cuts:
            places = [p for p in range(n) if (at + p) % 3 != 1]
            steps.append({"step": len(steps), "entries": [{"id": rid, "tokens": requests[rid][at:at + n], "want": places}], "end": []})
            expect.append(want[rid][[at + p for p in places]])
            at += n
        steps[-1]["end"] = [rid]
    for dtype, limit in (("bfloat16", LIMIT["bf16"]), ("float32", LIMIT["f32"])):
        out = tmp_path / dtype
        out.mkdir()
        run = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "model"), "--dtype", dtype, "--out", str(out),
                              "--max-tokens", "48"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
        assert run.returncode == 0, run.stderr[-2000:]
        assert [x for x in run.stdout.splitlines() if x] == [f"done {i}" for i in range(len(steps))]
        for i, rows in enumerate(expect):
            if len(rows) == 0:
                assert not (out / f"{i}.f32").exists()
                continue
            got = np.fromfile(out / f"{i}.f32", "<f4").reshape(rows.shape)
            assert row_errors(got, rows).max() < limit * 1.5


def test_command_line_generation(tmp_path):
    cfg, tensors, _ = build("odd")
    save(tmp_path, cfg, tensors)
    prompt = tokens_for(cfg, 6)
    run = subprocess.run([sys.executable, "-m", "tnsr_b200.generate", "--model", str(tmp_path), "--dtype", "float32", "--max-new-tokens", "8",
                          "--prompt", " ".join(map(str, prompt))], capture_output=True, text=True, timeout=300, cwd=ROOT)
    assert run.returncode == 0, run.stderr[-2000:]
    assert [int(x) for x in run.stdout.split()] == greedy(cfg, tensors, prompt, 8)[6:]
