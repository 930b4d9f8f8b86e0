"""Ganupel on the GPU against the plain restatement (oracle/ganupel.py): the operators alone, whole prompts, decoding through
caches and states, portions, batches of unequal sessions, reused slots and pages, windows, generation, the trace program
and the command line."""
import ctypes as C
import json
import os
import subprocess
import sys

import numpy as np
import pytest

pytestmark = pytest.mark.gpu

torch = pytest.importorskip("torch")

from oracle import bolonex as interleaved  # noqa: E402
from oracle import ganupel as plain  # noqa: E402
from tests.ganupel_util import (CONFIGS, bf16_exact, build, config, dense, moe, parallel, random_tensors, rglru, row_errors,  # noqa: E402
                                tokens_for)
from tests.gpu_util import dev, lib, ok, ptr, rel_err, stream  # noqa: E402
from tests.test_bolonex_host import save  # noqa: E402
from tnsr_b200 import _native  # noqa: E402
from tnsr_b200.ganupel import Ganupel, GanupelConfig  # noqa: E402
from tnsr_b200.nn import Backend, GptDecoderOptions, GptPrefillMode, TnsrError  # noqa: E402
from tnsr_b200.session import B200Session  # noqa: E402

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32, BF16 = 0, 1
TORCH = {F32: torch.float32, BF16: torch.bfloat16}
# f32: rounding of sums only.  bf16: activations of every product and cache row carry 8 bits, and a norm over few nearly
# cancelled values magnifies them: most rows are far below the limit.
LIMIT = {"f32": 5e-5, "bf16": 0.12}


def close(errors, dtype, limit=1.0):
    return errors.max() < limit * LIMIT[dtype] and (dtype == "f32" or np.quantile(errors, 0.9) < limit * LIMIT[dtype] / 2)


def place(sessions, chunk, position=0, positions=None):
    return _native.Place(sessions, chunk, position, 0, positions.data_ptr() if positions is not None else None)


def placed(positions, chunk):
    """Host position when all sessions stand at one place, else an array on the device."""
    if len(set(positions)) == 1:
        return place(len(positions), chunk, positions[0])
    return place(len(positions), chunk, positions=dev(np.asarray(positions, np.uint32).view(np.int32)))


# ---- rotation ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("shape", [(4, 2, 64, 64, 64), (6, 3, 40, 24, 16), (8, 1, 128, 72, 96), (3, 3, 10, 7, 6), (2, 1, 16, 32, 0)])
@pytest.mark.parametrize("layout", ["halves", "interleaved"])
def test_rotary(dtype, shape, layout):
    heads, kv_heads, dim, vdim, dims = shape
    rng = np.random.default_rng(dim)
    rot = {"base": 300.0, "dims": dims, "scaling": None}
    capacity, positions, chunk = 60, (0, 17, 39), 21
    cols = heads * dim + kv_heads * (dim + vdim)
    ld = (cols + 31) // 32 * 32
    rows = bf16_exact(rng.normal(size=(3, chunk, ld)).astype(np.float32))
    d_rows = dev(rows.reshape(-1, ld), TORCH[dtype])
    f = 300.0 ** (-2.0 * np.arange(dims // 2) / max(dims, 1))
    angle = np.arange(capacity)[:, None] * f[None]
    table = dev(np.stack([np.cos(angle), np.sin(angle)], axis=-1).astype(np.float32))
    q = torch.full((3, chunk, heads, dim), 7.0, dtype=TORCH[dtype], device="cuda")
    k = torch.full((3, capacity, kv_heads, dim), 7.0, dtype=TORCH[dtype], device="cuda")
    v = torch.full((3, capacity, kv_heads, vdim), 7.0, dtype=TORCH[dtype], device="cuda")
    args = _native.RotaryArgs(d_rows.data_ptr(), table.data_ptr() if dims else None, q.data_ptr(), k.data_ptr(), v.data_ptr(), ld, heads, kv_heads, dim,
                              vdim, dims, _native.ROTARY[layout], capacity, dtype, 0)
    ok(lib().tnsr_b200_rotary(C.byref(args), C.byref(placed(positions, chunk)), stream()))
    torch.cuda.synchronize()
    rotate = plain.rotate_halves if layout == "halves" else lambda x, r: interleaved.rotate_interleaved(x, r) if dims else x
    tol = 1e-6 if dtype == F32 else 4e-3
    for s, p in enumerate(positions):
        full = np.zeros((p + chunk, ld))
        full[p:] = rows[s]
        fq = rotate(full[:, :heads * dim].reshape(-1, heads, dim), rot)[p:]
        fk = rotate(full[:, heads * dim:heads * dim + kv_heads * dim].reshape(-1, kv_heads, dim), rot)[p:]
        fv = full[p:, heads * dim + kv_heads * dim:cols].reshape(-1, kv_heads, vdim)
        assert rel_err(q[s].float().cpu().numpy(), fq) < tol
        assert rel_err(k[s, p:p + chunk].float().cpu().numpy(), fk) < tol
        assert np.array_equal(v[s, p:p + chunk].float().cpu().numpy(), fv)
        for cache in (k, v):       # nothing but the new rows is written
            other = cache[s].float().cpu().numpy()
            assert np.all(other[:p] == 7.0) and np.all(other[p + chunk:] == 7.0)


# ---- windowed attention ----------------------------------------------------------------------------------
def run_attention(q, k, v, bias, positions, scale, window, dtype, engine=0, workspace=True, gain=0.75, kind="sigmoid"):
    """q [s, chunk, H, dim]; k, v [s, capacity, G, width], with every row that no query may see poisoned."""
    s, chunk, heads, dim = q.shape
    capacity, kv_heads, vdim = k.shape[1], k.shape[2], v.shape[3]
    k, v = k.copy(), v.copy()
    for i, p in enumerate(positions):
        k[i, p + chunk:], v[i, p + chunk:] = np.nan, np.nan
        if window and p >= window:
            # finite, because a tile that holds both visible and hidden rows is multiplied by zero weights
            k[i, :p + 1 - window], v[i, :p + 1 - window] = 50.0, 1e4
    out_cols = heads * vdim + 3
    out_ld = (out_cols + 7) // 8 * 8
    out = torch.full((s * chunk, out_ld), 7.0, dtype=TORCH[dtype], device="cuda")
    size = lib().tnsr_b200_grouped_attention_workspace(dim, vdim)
    ws = torch.zeros(size, dtype=torch.uint8, device="cuda")
    d = [dev(x.astype(np.float32), TORCH[dtype]) for x in (q, k, v)]
    b = dev(np.asarray(bias, np.float32))
    args = _native.GroupedAttentionArgs(d[0].data_ptr(), d[1].data_ptr(), d[2].data_ptr(), None, out.data_ptr(), ws.data_ptr() if workspace else None, None,
                                        size if workspace else 0, heads, kv_heads, dim, vdim, capacity, 0, out_ld, out_cols, scale, 0.0, dtype, engine,
                                        b.data_ptr() if kind == "sigmoid" else None, window, _native.SCORE[kind], gain, 0)
    results = []
    for _ in range(2):       # twice: merge counters must come back to zero
        ok(lib().tnsr_b200_grouped_attention(C.byref(args), C.byref(placed(positions, chunk)), stream()))
        torch.cuda.synchronize()
        results.append(out.float().cpu().numpy())
    assert np.array_equal(results[0], results[1])
    assert np.all(results[0][:, heads * vdim:out_cols] == 0.0) and np.all(results[0][:, out_cols:] == 7.0)
    return results[0][:, :heads * vdim].reshape(s, chunk, heads, vdim) / gain


def attention_case(seed, positions, chunk, capacity, heads, kv_heads, dim, vdim, planted=None):
    """planted = (key, query): that key of every session is aligned with that query of every head, and its value is large,
    so that whether it is seen decides the query's output."""
    rng = np.random.default_rng(seed)
    s = len(positions)
    q, k = rng.normal(size=(s, chunk, heads, dim)) * 0.5, rng.normal(size=(s, capacity, kv_heads, dim)) * 0.5
    v = rng.normal(size=(s, capacity, kv_heads, vdim))
    if planted is not None:
        key, query = planted
        u = rng.normal(size=dim)
        q[:, query], k[:, key] = u * 2.0, u * 2.0
        v[:, key] *= 20.0
    return [bf16_exact(x.astype(np.float32)) for x in (q, k, v)] + [rng.uniform(-4, -1, heads)]


def expected_attention(q, k, v, bias, positions, scale, window, kind="sigmoid"):
    out = np.zeros(q.shape[:3] + (v.shape[3],))
    s, chunk, heads = q.shape[:3]
    for i, p in enumerate(positions):
        full = np.zeros((p + chunk, heads, q.shape[3]))
        full[p:] = q[i]
        kk, vv = k[i, :p + chunk].astype(np.float64), v[i, :p + chunk].astype(np.float64)
        if kind == "sigmoid":
            out[i] = plain.sigmoid_attend(full, kk, vv, scale, bias, window or 1 << 30)[p:]
            continue
        for t in range(chunk):      # softmax over the window: the tail of the sequence alone
            at = p + t
            low = max(0, at + 1 - window) if window else 0
            out[i, t] = interleaved.attend(np.broadcast_to(full[at], (at + 1 - low,) + full[at].shape), kk[low:at + 1], vv[low:at + 1], scale, None)[-1]
    return out


SHAPES = [(4, 2, 64, 64), (6, 2, 40, 24), (8, 1, 128, 128), (3, 3, 10, 7), (2, 1, 200, 136), (12, 1, 16, 32)]


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("chunk,positions", [(1, (0, 37, 200, 15)), (2, (0, 14, 63)), (5, (11, 0)), (64, (5, 5)), (131, (0, 70)), (40, (200, 200))])
def test_sigmoid_attention(shape, chunk, positions):
    heads, kv_heads, dim, vdim = shape
    for window in (0, 1, 17, 64, 100):
        case = attention_case(chunk + dim, positions, chunk, 256, heads, kv_heads, dim, vdim)
        want = expected_attention(*case, positions, 0.3, window)
        assert rel_err(run_attention(*case, positions, 0.3, window, BF16), want) < 5e-3, window
        assert rel_err(run_attention(*case, positions, 0.3, window, BF16, engine=1), want) < 5e-3, window
        assert rel_err(run_attention(*case, positions, 0.3, window, F32), want) < 2e-6, window
    assert rel_err(run_attention(*case, positions, 0.3, 100, BF16, workspace=False), want) < 5e-3


@pytest.mark.parametrize("heads,kv_heads", [(4, 2), (3, 3), (12, 1)])
@pytest.mark.parametrize("kind", ["sigmoid", "softmax"])
def test_long_windowed_chunks_on_every_engine(heads, kv_heads, kind):
    """Heads of 64 at a position the host knows: the tcgen05 kernel (engine 0) and the warp-level one (2), windows around the
    key blocks, whole and ragged query tiles."""
    for chunk, position in ((32, 0), (127, 0), (129, 63), (256, 127), (40, 300)):
        for window in (1, 63, 127, 128, 129, 200):
            positions = (position, position)
            case = attention_case(chunk, positions, chunk, position + chunk + 3, heads, kv_heads, 64, 64)
            want = expected_attention(*case, positions, 0.4, window, kind)
            for engine in (0, 2):
                got = run_attention(*case, positions, 0.4, window, BF16, engine=engine, kind=kind)
                assert rel_err(got, want) < 8e-3, (chunk, position, window, engine)


@pytest.mark.parametrize("engine", [0, 1, 2])
@pytest.mark.parametrize("dim,vdim", [(64, 64), (72, 40)])
def test_one_outstanding_key_just_inside_and_just_outside_a_window(dim, vdim, engine):
    for total, chunk in ((400, 1), (400, 3), (300, 130)):
        position, query = total - chunk, chunk - 1
        for window in (1, 15, 16, 17, 64, 127, 128, 129, 250):
            edge = total - window             # first key that the last query sees
            for key in {edge, max(0, edge - 1), total - 1, (edge + total) // 2}:
                case = attention_case(key, (position,), chunk, 416, 4, 2, dim, vdim, planted=(key, query))
                want = expected_attention(*case, (position,), 0.5, window)
                got = run_attention(*case, (position,), 0.5, window, BF16, engine=engine)
                assert rel_err(got, want) < 5e-3, (total, chunk, window, key)
                q, k, v, bias = case
                v = v.copy()
                v[:, key] = 0.0
                other = expected_attention(q, k, v, bias, (position,), 0.5, window)
                assert (np.abs(want - other)[0, query].max() > 5.0) == (key >= edge)      # the case does what it says


# ---- HGRN2 -------------------------------------------------------------------------------------------------
def hgrn2_case(shape, s, n, seed=0, low=0.2):
    heads, dim, vdim = shape
    rng = np.random.default_rng(seed)
    u = bf16_exact(rng.normal(size=(s, n, 2 * heads * dim + heads * vdim)).astype(np.float32))      # f | q | v
    u[:, :, :heads * dim] *= 2.0
    t = {"f.b": rng.uniform(-1, 5, heads * dim), "lower": np.where(rng.random(heads * dim) < low, 0.0, rng.uniform(0, 0.9, heads * dim)),
         "norm": rng.uniform(0.5, 1.5, vdim)}
    return u, {k: bf16_exact(v.astype(np.float32)) for k, v in t.items()}


def expected_hgrn2(shape, u, t):
    """The mixer of the plain restatement with projections that pick columns."""
    heads, dim, vdim = shape
    k, eye = heads * dim, np.eye(u.shape[2])
    w = {name: v.astype(np.float64) for name, v in t.items()}
    w.update({"f": eye[:k], "q": eye[k:2 * k], "v": eye[2 * k:], "o": np.eye(heads * vdim)})
    return np.stack([plain.hgrn2(x.astype(np.float64), dict(heads=heads, dim=dim, vdim=vdim), w, 1e-5) for x in u])


def run_hgrn2(shape, u, t, portions, dtype, engine=0, positions=None, state=None):
    heads, dim, vdim = shape
    k = heads * dim
    s = u.shape[0]
    state = state if state is not None else torch.full((s, heads, dim, vdim), float("nan"), device="cuda")
    w = {name: dev(np.ascontiguousarray(v, dtype=np.float32)) for name, v in t.items()}
    q_cols = (k + 7) // 8 * 8
    ld = (q_cols + heads * vdim + 7) // 8 * 8
    outs, at = [], 0
    for chunk in portions:
        part = u[:, at:at + chunk].reshape(s * chunk, -1)
        rows = np.zeros((s * chunk, ld), np.float32)
        rows[:, :k], rows[:, q_cols:q_cols + heads * vdim] = part[:, k:2 * k], part[:, 2 * k:]
        d_rows, d_f = dev(rows, TORCH[dtype]), dev(np.ascontiguousarray(part[:, :k]))
        out_cols = heads * vdim + 5
        out_ld = (out_cols + 7) // 8 * 8
        out = torch.full((s * chunk, out_ld), 7.0, dtype=TORCH[dtype], device="cuda")
        raw = torch.empty((s * chunk, heads * vdim), device="cuda")
        args = _native.Hgrn2Args(d_rows.data_ptr(), d_rows.data_ptr() + q_cols * d_rows.element_size(), d_f.data_ptr(), w["f.b"].data_ptr(),
                                 w["lower"].data_ptr(), w["norm"].data_ptr(), state.data_ptr(), raw.data_ptr(), out.data_ptr(), ld, k, heads, dim, vdim,
                                 out_ld, out_cols, 1e-5, 0.5, dtype, engine, 0)
        pos = dev((np.asarray(positions or [0] * s) + at).astype(np.uint32).view(np.int32))
        ok(lib().tnsr_b200_hgrn2(C.byref(args), C.byref(place(s, chunk, positions=pos)), stream()))
        torch.cuda.synchronize()
        o = out.float().cpu().numpy()
        assert np.all(o[:, heads * vdim:out_cols] == 0.0) and np.all(o[:, out_cols:] == 7.0)
        outs.append(2.0 * o[:, :heads * vdim].reshape(s, chunk, -1))
        at += chunk
    return np.concatenate(outs, axis=1), state


HGRN2_SHAPES = [(4, 128, 64), (3, 64, 128), (3, 20, 28), (5, 5, 7), (2, 136, 200), (1, 200, 33), (2, 256, 256), (6, 32, 32)]


@pytest.mark.parametrize("shape", HGRN2_SHAPES)
def test_hgrn2_portions_and_tokens(shape):
    n = 150
    u, t = hgrn2_case(shape, 2, n)
    want = expected_hgrn2(shape, u, t)
    for portions in ([n], [64, 64, 22], [15, 17, 33, 16, 69], [1] * 9 + [2, 3, 16, 17, 40, 1, 1, 61], [2] * 75):
        got, state = run_hgrn2(shape, u, t, portions, BF16)
        assert np.sqrt(np.mean((got - want) ** 2)) < 4e-3 * np.std(want) and rel_err(got, want) < 2e-2, portions
        got32, state32 = run_hgrn2(shape, u, t, portions, F32)
        assert rel_err(got32, want) < 1e-5, portions
        # inputs are bf16-exact here, so the carried f32 states agree far below bf16's rounding
        assert rel_err(state.cpu().numpy(), state32.cpu().numpy()) < 1e-4
    token_by_token, _ = run_hgrn2(shape, u, t, [n], BF16, engine=1)
    assert rel_err(token_by_token, want) < 2e-2


@pytest.mark.parametrize("shape", [(2, 64, 64), (2, 20, 28), (1, 128, 128)])
def test_hgrn2_gates_that_all_but_vanish(shape):
    """Gates near zero make the running products of a chunk underflow: single channels, single tokens, whole chunks."""
    heads, dim, vdim = shape
    u, t = hgrn2_case(shape, 2, 100, low=0.5)
    f = u[:, :, :heads * dim].reshape(2, 100, heads, dim)
    f[:, 20:30, :, 3] = -30.0          # one channel for ten tokens
    f[:, 47] = -60.0                   # every channel of one token
    f[:, 64:, :, 5:9] = -9.0           # a run of small gates over several chunks
    f[1, 80:90] = -200.0
    want = expected_hgrn2(shape, u, t)
    for portions in ([100], [50, 50], [37, 1, 62]):
        got, state = run_hgrn2(shape, u, t, portions, BF16)
        assert np.isfinite(got).all() and np.sqrt(np.mean((got - want) ** 2)) < 4e-3 * np.std(want) and rel_err(got, want) < 2e-2, portions
        got32, state32 = run_hgrn2(shape, u, t, portions, F32)
        assert rel_err(got32, want) < 1e-5
        assert rel_err(state.cpu().numpy(), state32.cpu().numpy()) < 1e-4


def test_hgrn2_state_keeps_32_bits_over_a_long_run():
    """Gates close to one over 800 tokens: what is written per token is 1e-4, and the scan must add it up like the token
    kernel does."""
    shape = (2, 64, 64)
    u, t = hgrn2_case(shape, 1, 800, seed=4)
    t["f.b"][:], t["lower"][:] = 9.0, 0.5
    _, scan = run_hgrn2(shape, u, t, [800], BF16)
    _, token = run_hgrn2(shape, u, t, [800], BF16, engine=1)
    assert rel_err(scan.cpu().numpy(), token.cpu().numpy()) < 5e-5


def test_sessions_at_position_zero_ignore_what_their_slot_holds():
    shape = (3, 20, 28)
    u, t = hgrn2_case(shape, 2, 40)
    want = expected_hgrn2(shape, u, t)
    for portions in ([40], [1, 1, 1, 37], [3, 37]):
        _, used = run_hgrn2(shape, u[::-1].copy(), t, [40], F32)
        assert rel_err(run_hgrn2(shape, u, t, portions, F32, state=used)[0], want) < 1e-5
    shape = (48, 2, 3)
    x, w = rglru_case(shape, 2, 40)
    want = expected_rglru(shape, x, w)
    for portions in ([40], [1, 1, 1, 37], [3, 37]):
        _, used = run_rglru(shape, x[::-1].copy(), w, [40], F32)
        assert rel_err(run_rglru(shape, x, w, portions, F32, state=used)[0], want) < 1e-5


# ---- real-gated linear recurrent unit -----------------------------------------------------------------------
def rglru_case(shape, s, n, seed=0):
    width, blocks, taps = shape
    part = width // blocks
    rng = np.random.default_rng(seed)
    u = bf16_exact(rng.normal(size=(s, n, 2 * width)).astype(np.float32))                            # y | x
    t = {"conv": rng.normal(0, 0.3, (width, taps)) + (np.arange(taps) == taps - 1), "conv.b": rng.normal(0, 0.3, width),
         "ra": rng.normal(0, part ** -0.5, (blocks, part, part)), "ra.b": rng.normal(0, 1, (blocks, part)),
         "ri": rng.normal(0, part ** -0.5, (blocks, part, part)), "ri.b": rng.normal(0, 1, (blocks, part)), "lam": rng.uniform(-7, 1, width)}
    return u, {k: bf16_exact(v.astype(np.float32)) for k, v in t.items()}


def expected_rglru(shape, x, t):
    """The recurrent block with projections that pick columns; its first branch arrives activated."""
    width = shape[0]
    w = {k: v.astype(np.float64) for k, v in t.items()}
    out = []
    for rows in x.astype(np.float64):
        u = plain.causal_conv(rows[:, width:], w["conv"], w["conv.b"])
        r, i = (plain.sigmoid(plain.block_diagonal(u, w[n], w[n + ".b"])) for n in ("ra", "ri"))
        out.append(plain.linear_unit_scan(u, r, i, w["lam"]) * rows[:, :width])
    return np.stack(out)


def run_rglru(shape, x, t, portions, dtype, positions=None, state=None):
    width, blocks, taps = shape
    part, s = width // blocks, x.shape[0]
    ring, carried = state if state else (torch.full((s, taps, width), float("nan"), dtype=TORCH[dtype], device="cuda"),
                                         torch.full((s, width), float("nan"), device="cuda"))
    w = {k: dev(np.ascontiguousarray(v, dtype=np.float32)) for k, v in t.items()}
    gate_w = dev(np.concatenate([t["ra"], t["ri"]], axis=1), TORCH[dtype])
    x_col = (width + 31) // 32 * 32
    ld = 2 * x_col
    outs, at = [], 0
    for chunk in portions:
        rows = np.zeros((s * chunk, ld), np.float32)
        rows[:, :width] = x[:, at:at + chunk, :width].reshape(s * chunk, width)
        rows[:, x_col:x_col + width] = x[:, at:at + chunk, width:].reshape(s * chunk, width)
        d_rows = dev(rows, TORCH[dtype])
        out_cols = width + 3
        out_ld = (out_cols + 7) // 8 * 8
        out = torch.full((s * chunk, out_ld), 7.0, dtype=TORCH[dtype], device="cuda")
        u = torch.empty((s * chunk, width), dtype=TORCH[dtype], device="cuda")
        gates = torch.empty((s * chunk, 2 * width), device="cuda")
        args = _native.RglruArgs(d_rows.data_ptr(), gate_w.data_ptr(), w["conv"].data_ptr(), w["conv.b"].data_ptr(), w["ra.b"].data_ptr(), w["ri.b"].data_ptr(),
                                 w["lam"].data_ptr(), ring.data_ptr(), carried.data_ptr(), u.data_ptr(), gates.data_ptr(), out.data_ptr(), None, ld, x_col,
                                 width, blocks, taps, out_ld, out_cols, dtype)
        pos = dev((np.asarray(positions or [0] * s) + at).astype(np.uint32).view(np.int32))
        ok(lib().tnsr_b200_rglru(C.byref(args), C.byref(place(s, chunk, positions=pos)), stream()))
        torch.cuda.synchronize()
        o = out.float().cpu().numpy()
        assert np.all(o[:, width:out_cols] == 0.0) and np.all(o[:, out_cols:] == 7.0)
        outs.append(o[:, :width].reshape(s, chunk, width))
        at += chunk
    return np.concatenate(outs, axis=1), (ring, carried)


@pytest.mark.parametrize("shape", [(128, 4, 4), (72, 3, 3), (45, 5, 5), (160, 1, 1), (96, 12, 16), (30, 2, 2), (33, 33, 4), (320, 4, 4)])
def test_rglru_portions_and_tokens(shape):
    n = 300
    x, t = rglru_case(shape, 2, n)
    want = expected_rglru(shape, x, t)
    for portions in ([n], [128, 129, 43], [127, 2, 171], [1] * 9 + [2, 3, 16, 17, 40, 1, 1, 61, 150], [2] * 150):
        got32, state32 = run_rglru(shape, x, t, portions, F32)
        assert rel_err(got32, want) < 2e-5, portions
        got, state = run_rglru(shape, x, t, portions, BF16)
        # u = conv(x) is rounded to bf16 before the gates and the recurrence
        assert np.sqrt(np.mean((got - want) ** 2)) < 6e-3 * np.std(want) and rel_err(got, want) < 2e-2, portions
        assert rel_err(state[1].cpu().numpy(), state32[1].cpu().numpy()) < 1e-2


# ---- feed-forwards ----------------------------------------------------------------------------------------
@pytest.mark.parametrize("width", [8, 64, 37, 392, 1000, 2048, 8200, 9000, 7])
def test_polynorm(width):
    rng = np.random.default_rng(width)
    z, act = bf16_exact((rng.normal(size=(5, width)) * [[0.03], [1], [4], [20], [0]]).astype(np.float32)), np.float32([0.7, -0.4, 0.9, 0.2])
    want = plain.poly_norm(z.astype(np.float64), act.astype(np.float64), 1e-3)
    out_cols, out_ld = width + 3, (width + 3 + 7) // 8 * 8
    for dtype, tol in ((F32, 2e-6), (BF16, 5e-3)):
        out = torch.full((5, out_ld), 7.0, dtype=TORCH[dtype], device="cuda")
        ok(lib().tnsr_b200_polynorm(ptr(dev(z, TORCH[dtype])), ptr(dev(act)), ptr(out), 5, width, out_ld, out_cols, 1e-3, dtype, stream()))
        torch.cuda.synchronize()
        got = out.float().cpu().numpy()
        assert rel_err(got[:, :width], want) < tol
        assert np.all(got[:, width:out_cols] == 0.0) and np.all(got[:, out_cols:] == 7.0)


def grouped(a, w, offsets, activation, dtype, out_dtype, engine=0):
    rows, (groups, n, k) = a.shape[0], w.shape
    out = torch.full((rows, n), 7.0, dtype=TORCH[out_dtype], device="cuda")
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    off = dev(np.asarray(offsets, np.uint32).view(np.int32)) if offsets is not None else None
    ok(lib().tnsr_b200_gemm_grouped(ptr(dev(a, TORCH[dtype])), ptr(dev(w, TORCH[dtype])), ptr(out), ptr(off), groups, rows, n, k, activation, dtype, out_dtype,
                                    engine, ptr(status), stream()))
    torch.cuda.synchronize()
    assert int(status[0]) == 0
    return out.float().cpu().numpy()


@pytest.mark.parametrize("counts", [[3, 0, 17, 1], [0, 0, 5], [40, 33, 0, 64, 9], [128, 1, 200], [300, 257, 0, 511], [16, 16, 16], [1]])
@pytest.mark.parametrize("n,k", [(64, 64), (320, 72), (96, 200), (33, 40), (130, 13)])
def test_grouped_products(counts, n, k):
    rng = np.random.default_rng(n + k + len(counts))
    spare = 5                                  # rows that belong to no group stay as they are
    rows, offsets = sum(counts) + spare, np.concatenate([[0], np.cumsum(counts)])
    a = bf16_exact(rng.normal(size=(rows, k)).astype(np.float32))
    w = bf16_exact((rng.normal(size=(len(counts), n, k)) * k ** -0.5).astype(np.float32))
    want = np.full((rows, n), 7.0)
    for g in range(len(counts)):
        want[offsets[g]:offsets[g + 1]] = a[offsets[g]:offsets[g + 1]].astype(np.float64) @ w[g].astype(np.float64).T
    squared = np.where(np.arange(rows)[:, None] < offsets[-1], np.maximum(want, 0.0) ** 2, 7.0)
    for dtype, out_dtype, engine, tol in ((BF16, F32, 0, 2e-6), (BF16, BF16, 0, 5e-3), (BF16, F32, 1, 2e-6), (F32, F32, 0, 2e-6)):
        got = grouped(a, w, offsets, -1, dtype, out_dtype, engine)
        assert rel_err(got, want) < tol and np.all(got[offsets[-1]:] == 7.0), (dtype, out_dtype, engine)
        assert rel_err(grouped(a, w, offsets, 4, dtype, out_dtype, engine), squared) < tol
    if rows % len(counts) == 0:
        equal = a.reshape(len(counts), -1, k).astype(np.float64) @ w.astype(np.float64).transpose(0, 2, 1)
        assert rel_err(grouped(a, w, None, -1, BF16, F32), equal.reshape(rows, n)) < 2e-6


def test_grouped_product_refuses_what_it_cannot_address():
    a, w = np.zeros((10, 64), np.float32), np.zeros((3, 32, 64), np.float32)
    out = torch.zeros((10, 32), device="cuda")
    call = lib().tnsr_b200_gemm_grouped
    assert call(ptr(dev(a)), ptr(dev(w)), ptr(out), None, 3, 10, 32, 64, -1, F32, F32, 0, None, stream()) == -1      # 10 rows in 3 equal groups
    assert call(ptr(dev(a)), ptr(dev(w)), ptr(out), None, 2000, 10, 32, 64, -1, F32, F32, 0, None, stream()) == -1


EXPERT_SHAPES = [(64, 48, 5, 2, 3), (96, 40, 40, 30, 8), (70, 13, 3, 0, 1), (128, 128, 8, 1, 9), (64, 32, 1, 3, 2), (64, 16, 300, 20, 32)]


@pytest.mark.parametrize("shape", EXPERT_SHAPES)
@pytest.mark.parametrize("rows", [1, 7, 64, 300, 700])
def test_experts(shape, rows):
    """Routing, identity experts, weights and the fused norm; 300 rows and more are sorted over several blocks."""
    d, ff, experts, identity, top = shape
    rng = np.random.default_rng(rows + d)
    total = experts + identity
    t = {f"e{e}.up": rng.normal(size=(ff, d)) * d ** -0.5 for e in range(experts)}
    t.update({f"e{e}.down": rng.normal(size=(d, ff)) * ff ** -0.5 for e in range(experts)})
    t = {k: bf16_exact(v.astype(np.float32)) for k, v in t.items()}
    correction = np.where(rng.random(total) < 0.3, 0.25, 0.0).astype(np.float32)
    logits = (rng.normal(size=(rows, total + 3)) * 3).astype(np.float32)
    h = bf16_exact(rng.normal(size=(rows, d)).astype(np.float32))
    x, scale, norm_w = rng.normal(size=(rows, d)).astype(np.float32), rng.uniform(0.4, 1.2, d).astype(np.float32), rng.normal(size=d).astype(np.float32)
    # the router's product is taken out: its logits are given
    router = {"experts": experts, "identity": identity, "top": top, "scale": 1.7}
    chosen, weights = plain.route(np.eye(rows), router, logits[:, :total].T.astype(np.float64), correction)
    z = np.exp(logits[:, :total].astype(np.float64) - logits[:, :total].max(axis=1, keepdims=True))
    ranked = np.sort(z / z.sum(axis=1, keepdims=True) + correction, axis=1)[:, ::-1]
    gap = ranked[:, top - 1] - ranked[:, top] if top < total else np.ones(rows)      # how close the last choice was
    out = np.zeros((rows, d))
    for i in range(rows):
        for e, w in zip(chosen[i], weights[i]):
            row = h[i].astype(np.float64)
            out[i] += w * (row if e >= experts else np.maximum(row @ t[f"e{e}.up"].T.astype(np.float64), 0.0) ** 2 @ t[f"e{e}.down"].T.astype(np.float64))
    want = x + scale * out
    normed = plain.norm_around_zero(want, norm_w, 1e-4)
    up, down = np.stack([t[f"e{e}.up"] for e in range(experts)]), np.stack([t[f"e{e}.down"] for e in range(experts)])
    for dtype, tol in ((F32, 1e-5), (BF16, 1e-2)):
        size = lib().tnsr_b200_experts_workspace(rows, d, ff, experts, top, dtype)
        ws = torch.empty(size, dtype=torch.uint8, device="cuda")
        d_x, d_h = dev(x.copy()), dev(h, TORCH[dtype])
        ids, got_w = torch.zeros((rows, top), dtype=torch.int32, device="cuda"), torch.zeros((rows, top), device="cuda")
        keep = [dev(logits), dev(correction), dev(up, TORCH[dtype]), dev(down, TORCH[dtype]), dev(scale), dev(norm_w)]
        args = _native.ExpertsArgs(keep[0].data_ptr(), keep[1].data_ptr(), d_h.data_ptr(), keep[2].data_ptr(), keep[3].data_ptr(), d_x.data_ptr(),
                                   keep[4].data_ptr(), keep[5].data_ptr(), d_h.data_ptr(), ws.data_ptr(), size, ids.data_ptr(), got_w.data_ptr(), None,
                                   rows, total + 3, d, ff, experts, identity, top, 1.7, 1.0, 1e-4, dtype, 0)
        ok(lib().tnsr_b200_experts(C.byref(args), stream()))       # the norm overwrites h
        torch.cuda.synchronize()
        ids, got_w = ids.cpu().numpy(), got_w.cpu().numpy()
        order, expect = np.argsort(ids, axis=1), np.argsort(chosen, axis=1)
        same = (np.take_along_axis(ids, order, 1) == np.take_along_axis(chosen, expect, 1)).all(axis=1)
        assert np.all(same | (gap < 1e-6)) and same.mean() > 0.97
        assert rel_err(np.take_along_axis(got_w, order, 1)[same], np.take_along_axis(weights, expect, 1)[same]) < 1e-5
        assert rel_err((d_x.cpu().numpy() - x)[same], (scale * out)[same]) < tol
        assert rel_err(d_h.float().cpu().numpy()[same], normed[same]) < tol


# ---- whole models --------------------------------------------------------------------------------------------
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
    assert close(row_errors(logits_of(decoder, ids), want), dtype)
    for portions in PORTIONS:
        assert close(row_errors(logits_of(decoder, ids, portions), want), dtype), portions
    assert close(row_errors(logits_of(decoder, ids[:1]), want[:1]), dtype)


def test_experts_follow_the_tokens_in_bf16():
    """Routing that depends on the token: a choice may fall the other way in 16 bits only where two scores are close."""
    cfg, _, _ = build("mixed", "bf16")
    tensors = random_tensors(cfg, seed=3, decisive=False)
    ids = tokens_for(cfg, 100)
    want, _ = plain.forward(cfg, tensors, ids)
    decoder = Ganupel(GanupelConfig.from_dict(cfg, "bf16"), tensors).decoder_with_capacity(Backend.Cuda, 1, 100)
    errors = row_errors(logits_of(decoder, ids), want)
    assert np.median(errors) < LIMIT["bf16"] / 2 and np.mean(errors > LIMIT["bf16"]) < 0.2


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_layers_wide_enough_for_the_few_row_products(dtype):
    """2048 channels: single tokens take the weight-streaming products, with layer scales in their epilogues."""
    cfg, tensors, model = build(config(2048, 64, [rglru(2048, 16, 4, dense(2048)), parallel((16, 4, 64, 64, 64, 8, 0.1), (8, 64, 64))]), dtype)
    ids = tokens_for(cfg, 40)
    want, _ = plain.forward(cfg, tensors, ids)
    decoder = model.decoder_with_capacity(Backend.Cuda, 1, 40)
    for portions in ([40], [34, 1, 1, 1, 1, 1, 1], [17, 23]):
        assert close(row_errors(logits_of(decoder, ids, portions), want), dtype), portions


@pytest.mark.parametrize("name", ["mixed", "even"])
def test_scalar_prefill_is_the_same_function(name):
    cfg, tensors, model = build(name, "bf16")
    ids = tokens_for(cfg, 90)
    want, _ = plain.forward(cfg, tensors, ids)
    decoder = model.decoder_with_options(Backend.Cuda, 1, 90, GptDecoderOptions(prefill=GptPrefillMode.Scalar))
    assert close(row_errors(logits_of(decoder, ids), want), "bf16")


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_each_constant_matters(dtype):
    """A change of any constant of the configuration must show in the logits far above the comparison's limit."""
    cfg, tensors, _ = build(config(64, 101, [parallel((4, 2, 16, 24, 12, 9, 0.5), (3, 12, 20), moe(40, 4, 1, 2, 1.5)), rglru(48, 2, 3, dense(56))], eps=1e-1), dtype)
    ids = tokens_for(cfg, 60)
    want, _ = plain.forward(cfg, tensors, ids)
    left = ("layers", 0, "mixer", "left")
    changes = [("norm", "eps", 1e-4), ("layers", 0, "mixer", "left_scale", 1.4), ("layers", 0, "mixer", "right_scale", 0.6), left + ("scale", 0.1),
               left + ("mask", "size", 10), left + ("mask", "size", 8), left + ("rot", "base", 40.0), left + ("rot", "dims", 8),
               ("layers", 0, "mlp", "router", "scale", 0.7), ("layers", 0, "mlp", "router", "top", 3)]
    for path in [()] + changes:
        other = json.loads(json.dumps(cfg))
        if path:
            at = other
            for key in path[:-2]:
                at = at[key]
            at[path[-2]] = path[-1]
        wrong, _ = plain.forward(other, tensors, ids)
        if path:
            assert row_errors(wrong, want).max() > (20 if dtype == "f32" else 0.5) * LIMIT[dtype], path
        follows = logits_of(Ganupel(GanupelConfig.from_dict(other, dtype), tensors).decoder_with_capacity(Backend.Cuda, 1, 60), ids)
        assert close(row_errors(follows, wrong), dtype), path


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("window", [16, 45, 129])
def test_planted_token_at_the_window_edge_decides(dtype, window):
    """q and k of the only layer depend on the token alone, and the last token's query matches one earlier token's key only:
    the logits must follow its value up to the window's last place, and not beyond."""
    cfg = config(64, 50, [parallel((2, 1, 32, 32, 0, window, 1.0), (1, 4, 4))])
    tensors = random_tensors(cfg)
    rng = np.random.default_rng(2)
    e = rng.normal(size=(50, 64))
    e[7, :32] = 3.0 * np.sign(e[7, :32])
    e[9] = e[7]
    e[9, 32:] = rng.normal(size=32)
    tensors["embed"] = bf16_exact(e.astype(np.float32))
    w = np.concatenate([np.eye(32), np.zeros((32, 32))], axis=1).astype(np.float32)
    tensors["l0.mix.left.k"], tensors["l0.mix.left.q"] = w, np.concatenate([w, w])
    tensors["l0.norm1"][:] = 0.0
    tensors["l0.mix.left.pb"][:] = -20.0
    tensors["l0.mix.left.o"] = bf16_exact(tensors["l0.mix.left.o"] * 16)      # the attention, not the embedding, makes the logits
    decoder = Ganupel(GanupelConfig.from_dict(cfg, dtype), tensors).decoder_with_capacity(Backend.Cuda, 1, 300)
    for total in (300, 131):
        filler = [int(x) for x in rng.integers(10, 50, total)]
        without, _ = plain.forward(cfg, tensors, filler[:total - 1] + [7])
        for back in (1, window // 2, window - 2, window - 1, window, window + 1):
            ids = list(filler[:total - 1]) + [7]
            ids[total - 1 - back] = 9
            want, _ = plain.forward(cfg, tensors, ids)
            # the filler's token was not seen and token 9 is: the difference shows exactly when it is inside the window
            moved = row_errors(want[-1:], without[-1:]).max() > 0.15
            assert moved == (back < window), (total, back)
            for portions in ([total], [total - 1, 1], [total - 40, 38, 2], [total - 3] + [1] * 3):
                assert close(row_errors(logits_of(decoder, ids, portions)[-1:], want[-1:]), dtype, 0.5), (total, back, portions)


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_long_decoding(dtype):
    cfg, tensors, model = build("mixed", dtype)
    ids = tokens_for(cfg, 420)
    want, _ = plain.forward(cfg, tensors, ids)
    decoder = model.decoder_with_capacity(Backend.Cuda, 1, 420)
    assert close(row_errors(logits_of(decoder, ids, [5] + [1] * 415), want), dtype)
    with pytest.raises(TnsrError, match="capacity exceeded"):
        decoder.decode([1])


@pytest.mark.parametrize("name", ["mixed", "even", "odd"])
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_rectangular_batch_equals_each_session_alone(name, dtype):
    cfg, tensors, model = build(name, dtype)
    rows = [tokens_for(cfg, 120, seed=i) for i in range(5)]
    decoder = model.decoder_with_capacity(Backend.Cuda, 5, 128)
    parts = []
    for a, b in ((0, 70), (70, 71), (71, 73), (73, 120)):       # 350 rows at first: experts are sorted over several blocks
        parts.append(decoder.decode([t for r in rows for t in r[a:b]]).reshape(5, b - a, cfg["vocab"]))
    got = np.concatenate(parts, axis=1)
    for i, r in enumerate(rows):
        assert close(row_errors(got[i], plain.forward(cfg, tensors, r)[0]), dtype)


@pytest.mark.parametrize("paged", [False, True])
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_unequal_sessions_slots_and_pages_used_again(paged, dtype):
    """Ragged steps: sessions start, end and are replaced at different times; every logits row must be that of the
    session alone.  The pool has fewer pages than slots x capacity."""
    cfg, tensors, model = build("mixed", dtype)
    kw = dict(kv_page_rows=16, kv_pool_pages=11) if paged else {}
    sess = B200Session(model.config(), 3, 96, logits_mode="all", **kw)
    for i, p in enumerate(model.parameters()):
        sess.refresh(i, p.values())
    requests = [tokens_for(cfg, n, seed=20 + i) for i, n in enumerate([50, 17, 33, 64, 16, 40, 65, 1])]
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
        assert close(row_errors(runs[-1], want), "bf16")
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
@pytest.mark.parametrize("name", ["even", "mixed"])
def test_device_greedy_and_sampling_follow_the_logits(mode, name):
    """A last layer with experts and one without a feed-forward: logits of last rows only."""
    from oracle.sampler import sample_row
    cfg, tensors, model = build(name, "bf16")
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
    new = dict(tensors)
    for name in ("l0.mix.left.pb", "l0.mix.right.f.b", "l0.mlp.e1.down", "l0.mlp.router", "l1.mix.ri", "l1.mlp.act", "l1.ls2", "l3.mix.lam", "head"):
        new[name] = bf16_exact(tensors[name] * 1.5 + 0.01)
        model.named()[name].set_values(new[name])
    assert close(row_errors(logits_of(decoder, ids), plain.forward(cfg, new, ids)[0]), "f32")


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
    cfg, tensors, _ = build("odd", "f32")
    save(tmp_path, cfg, tensors)
    prompt = tokens_for(cfg, 6)
    run = subprocess.run([sys.executable, "-m", "tnsr_b200.generate", "--model", str(tmp_path), "--dtype", "float32", "--max-new-tokens", "8",
                          "--prompt", " ".join(map(str, prompt))], capture_output=True, text=True, timeout=300, cwd=ROOT)
    assert run.returncode == 0, run.stderr[-2000:]
    assert [int(x) for x in run.stdout.split()] == greedy(cfg, tensors, prompt, 8)[6:]


# ---- mechanisms in other company -------------------------------------------------------------------------------
class OtherDesign:
    """The block forms, mixers and feed-forwards of the library in combinations that no model here has."""
    vocab_size, embed_dim, num_layers, layer_norm_epsilon, max_sequence_length = 83, 64, 4, 1e-4, 1 << 20
    layers = (0, 1, 2, 3)

    def __init__(self, weight_dtype):
        self.weight_dtype = weight_dtype

    def stack(self):
        a = (_native.LayerDesc * 4)()
        for x in a:
            x.weights_of, x.feed_forward = -1, 40
        a[0].mixer, a[0].block_form, a[0].heads, a[0].vdim, a[0].state, a[0].groups, a[0].norm_groups, a[0].conv_taps = 1, 1, 4, 16, 24, 2, 2, 3
        b = a[1]       # a parallel block of softmax attention in a window beside HGRN2
        b.mixer, b.heads, b.kv_heads, b.dim, b.vdim, b.window, b.score_kind, b.score_scale = 2, 4, 2, 24, 16, 9, 0, 0.4
        b.rotary_dims, b.rotary_layout, b.rotary_base, b.rec_heads, b.rec_dim, b.rec_vdim, b.attention_gain, b.recurrent_gain = 8, 0, 50.0, 2, 12, 20, 1.3, 0.6
        a[2].mixer, a[2].width, a[2].blocks, a[2].conv_taps = 3, 96, 3, 4
        c = a[3]
        c.mixer, c.block_form, c.heads, c.kv_heads, c.dim, c.vdim, c.conv_taps, c.score_scale = 0, 1, 4, 1, 16, 24, 2, 0.5
        c.rotary_dims, c.rotary_base, c.feed_forward_kind, c.experts, c.identity_experts, c.top, c.router_scale = 16, 50.0, 2, 3, 2, 2, 1.2
        return _native.StackDesc(1.5, 1.0, a, 4)

    def tensor_shapes(self):
        d = 64
        s = {"embed": (83, d), "head": (83, d), "final.norm": (d,)}
        s.update({"0.norm1": (d,), "0.in": (64 + 160 + 4, d), "0.conv": (160, 3), "0.conv.b": (160,), "0.dt_bias": (4,), "0.A_log": (4,), "0.D": (4,),
                  "0.norm": (64,), "0.o": (d, 64), "0.ls1": (d,), "0.norm2": (d,), "0.up": (40, d), "0.down": (d, 40), "0.ls2": (d,)})
        s.update({"1.norm1": (d,), "1.left.q": (96, d), "1.left.k": (48, d), "1.left.v": (32, d), "1.left.o": (d, 64), "1.right.q": (24, d), "1.right.f": (24, d),
                  "1.right.f.b": (24,), "1.right.lower": (24,), "1.right.v": (40, d), "1.right.norm": (20,), "1.right.o": (d, 40), "1.up": (40, d),
                  "1.down": (d, 40)})
        s.update({"2.norm1": (d,), "2.y": (96, d), "2.y.b": (96,), "2.x": (96, d), "2.x.b": (96,), "2.conv": (96, 4), "2.conv.b": (96,), "2.ra": (3, 32, 32),
                  "2.ra.b": (3, 32), "2.ri": (3, 32, 32), "2.ri.b": (3, 32), "2.lam": (96,), "2.o": (d, 96), "2.up": (40, d), "2.down": (d, 40)})
        s.update({"3.norm1": (d,), "3.q": (64, d), "3.q.b": (64,), "3.k": (16, d), "3.k.b": (16,), "3.v": (24, d), "3.v.b": (24,), "3.q.norm": (16,), "3.k.norm": (16,),
                  "3.q.conv": (64, 2), "3.k.conv": (16, 2), "3.v.conv": (24, 2), "3.g": (4, d), "3.o": (d, 96), "3.ls1": (d,), "3.norm2": (d,)})
        for e in range(3):
            s[f"3.e{e}.up"], s[f"3.e{e}.down"] = (40, d), (d, 40)
        s.update({"3.router": (5, d), "3.correction": (5,), "3.ls2": (d,)})
        return s

    def forward(self, tensors, tokens):
        get, eps = {k: v.astype(np.float64) for k, v in tensors.items()}, self.layer_norm_epsilon

        def of(i):
            return plain.under(get, f"{i}.")

        def gelu(h, t):
            return plain.gelu_tanh(h @ t["up"].T) @ t["down"].T

        x = get["embed"][np.asarray(tokens)] * 1.5
        t = of(0)
        x = x + interleaved.mamba2_mixer(plain.norm_around_zero(x, t["norm1"], eps), dict(heads=4, vdim=16, state=24, groups=2, norm_groups=2), t, eps) * t["ls1"]
        x = x + gelu(plain.norm_around_zero(x, t["norm2"], eps), t) * t["ls2"]
        t = of(1)
        h, n = plain.norm_around_zero(x, t["norm1"], eps), len(tokens)
        rot = {"base": 50.0, "dims": 8, "scaling": None}
        q, k = (interleaved.rotate_interleaved((h @ t["left." + name].T).reshape(n, -1, 24), rot) for name in "qk")
        v = (h @ t["left.v"].T).reshape(n, 2, 16)
        o = expected_attention(q[None], k[None], v[None], None, (0,), 0.4, 9, "softmax")[0]
        right = plain.hgrn2(h, dict(heads=2, dim=12, vdim=20), plain.under(t, "right."), eps)
        x = x + 1.3 * o.reshape(n, -1) @ t["left.o"].T + 0.6 * right + gelu(h, t)
        t = of(2)
        h = plain.norm_around_zero(x, t["norm1"], eps)
        x = x + plain.rglru_mixer(h, None, t, eps) + gelu(h, t)
        t = of(3)
        m = dict(heads=4, kv_heads=1, dim=16, vdim=24, scale=0.5, rot={"base": 50.0, "dims": 16, "scaling": None})
        x = x + interleaved.attention_mixer(plain.norm_around_zero(x, t["norm1"], eps), m, t, eps) * t["ls1"]
        router = {"experts": 3, "identity": 2, "top": 2, "scale": 1.2}
        x = x + plain.mixture(plain.norm_around_zero(x, t["norm2"], eps), {"router": router}, t, eps) * t["ls2"]
        return plain.norm_around_zero(x, get["final.norm"], eps) @ get["head"].T


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_mechanisms_combine_freely(dtype):
    from tnsr_b200.described import DescribedModel
    design, rng = OtherDesign(dtype), np.random.default_rng(8)
    tensors = {}
    for name, shape in design.tensor_shapes().items():
        leaf = name.split(".")[-1]
        scale = {"conv": 0.4, "b": 0.3, "norm1": 0.3, "norm2": 0.3, "A_log": 0.5, "dt_bias": 1.0}.get(leaf, shape[-1] ** -0.5)
        v = rng.normal(0, 1.0 if name == "embed" else scale, shape)
        if leaf in ("ls1", "ls2", "norm", "D") and name != "final.norm":
            v = rng.uniform(0.5, 1.3, shape)
        elif leaf == "lower":
            v = rng.uniform(0, 0.9, shape)
        elif leaf == "lam":
            v = rng.uniform(-5, 0, shape)
        elif leaf == "correction":
            v = np.array([4.0, 0.0, 2.0, 8.0, 0.0])
        tensors[name] = bf16_exact(v.astype(np.float32))
    model = DescribedModel(design, tensors)
    ids = [int(x) for x in rng.integers(0, 83, 90)]
    want = design.forward(tensors, ids)
    decoder = model.decoder_with_capacity(Backend.Cuda, 1, 90)
    for portions in ([90], [40] + [1] * 50, [2, 17, 33, 38]):
        assert close(row_errors(logits_of(decoder, ids, portions), want), dtype), portions
