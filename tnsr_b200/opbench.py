"""Operator-level measurements of the kernels behind the C ABI.

    python -m tnsr_b200.opbench gemm        # configuration 1: square sweep + skinny decode shapes
    python -m tnsr_b200.opbench skinny_gemm # only the skinny decode shapes of configuration 1 (M = 1, 8, 64; bf16 out)
    python -m tnsr_b200.opbench serving_gemms  # configuration 4's projection shapes at prefill and decode size
    python -m tnsr_b200.opbench mlp         # configuration 2: fused SwiGLU MLP 4096 x 2048 -> 5632 -> 2048
    python -m tnsr_b200.opbench attention   # configuration 3: 64 sessions x 16 heads x 64, ragged lengths <= 4096
    python -m tnsr_b200.opbench serving_attention  # configuration 4's decode attention: 256 x 12 x 64, 641 live keys
    python -m tnsr_b200.opbench elementwise # LayerNorm, SwiGLU, embedding, greedy pick
    python -m tnsr_b200.opbench prefill_attention  # configuration 4's prefill attention on both engines
    python -m tnsr_b200.opbench mixers      # the mixers of described models: grouped attention, mamba2, RMS norm
    python -m tnsr_b200.opbench ganupel     # windowed sigmoid attention, HGRN2, linear recurrent unit, PolyNorm, experts
    python -m tnsr_b200.opbench all

Every line is one JSON object: algorithmic flops / bytes, CUDA-event time (median of `--samples`
after 3 warm-up launches), achieved TFLOP/s or GB/s and the fraction of the measured peak
(MEASURED_PEAKS.json when present, else 6650 GB/s / 1590 TFLOP/s).  Between timed launches the
operands rotate through enough distinct copies to exceed the 126 MB L2 (or, where one operand set
is larger than L2 anyway, stay put).  torch only owns device memory and events here.
"""
from __future__ import annotations

import argparse
import ctypes as C
import json
import os
import sys

import numpy as np
import torch

from . import _native

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
L2_BYTES = 126 << 20


def peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(path):
        with open(path) as f:
            d = json.load(f)
        return float(d["hbm_gbs"]), float(d["bf16_tflops"]), "measured"
    return 6650.0, 1590.0, "fallback"


def lib():
    return _native.lib()


def ptr(t):
    return C.c_void_p(t.data_ptr()) if t is not None else None


def stream():
    return C.c_void_p(torch.cuda.current_stream().cuda_stream)


def ok(code):
    if code != 0:
        raise RuntimeError(f"{_native.STATUS.get(code, code)}: {_native.last_error(None)}")


def timed(launch, sets, samples):
    """Median milliseconds of launch(i) over `samples` launches, rotating i over `sets` operand copies."""
    for i in range(3):
        launch(i % sets)
    torch.cuda.synchronize()
    times = []
    for i in range(samples):
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        launch((i + 3) % sets)
        e1.record()
        e1.synchronize()
        times.append(e0.elapsed_time(e1))
    return float(np.median(times)), times


def timed_graph(launch, sets, samples, reps=None):
    """Per-launch milliseconds of a SHORT kernel: `reps` launches, rotating over the operand copies, are captured into
    one CUDA graph and the replay is timed -- a single launch between two events would mostly measure the host (tensor-map
    encoding, the ctypes call, the launch itself), not the GPU.  Includes the ~1.2 us a dependent graph node costs."""
    reps = reps or max(sets, 16)
    side = torch.cuda.Stream()
    with torch.cuda.stream(side):
        for i in range(3):
            launch(i % sets)
        torch.cuda.synchronize()
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph, stream=side):
            for i in range(reps):
                launch(i % sets)
        times = []
        for i in range(samples + 2):
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            graph.replay()
            e1.record()
            e1.synchronize()
            if i >= 2:
                times.append(e0.elapsed_time(e1) / reps)
    torch.cuda.synchronize()
    return float(np.median(times)), times


def copies_for(bytes_per_set):
    return max(1, min(64, -(-2 * L2_BYTES // max(bytes_per_set, 1))))


RESULTS = []      # every emitted record, for callers that import the bench functions
QUIET = False     # True: collect only


def emit(**kw):
    RESULTS.append(kw)
    if not QUIET:
        print(json.dumps(kw), flush=True)


def bench_gemm(samples, shapes=None, outs=("bf16", "f32")):
    hbm, tf, kind = peaks()
    if shapes is None:
        shapes = [(n, n, n) for n in (1024, 2048, 4096, 8192)] + [(m, 4096, 4096) for m in (1, 8, 64)]
    g = torch.Generator(device="cuda").manual_seed(2)
    for m, n, k in shapes:
        for out_dtype, name in ((1, "bf16"), (0, "f32")):
            if name not in outs:
                continue
            osz = 2 if out_dtype else 4
            per_set = 2 * (m * k + n * k) + osz * m * n
            sets = copies_for(per_set)
            a = [(torch.rand((m, k), device="cuda", generator=g) * 2 - 1).to(torch.bfloat16) for _ in range(sets)]
            b = [(torch.rand((n, k), device="cuda", generator=g) * 2 - 1).to(torch.bfloat16) for _ in range(sets)]
            o = [torch.empty((m, n), device="cuda", dtype=torch.bfloat16 if out_dtype else torch.float32) for _ in range(sets)]

            ws = torch.zeros(lib().tnsr_b200_gemm_workspace(), dtype=torch.uint8, device="cuda") if m <= 64 else None

            def launch(i):
                if ws is None:
                    ok(lib().tnsr_b200_gemm_bf16(ptr(a[i]), ptr(b[i]), None, None, ptr(o[i]), m, n, k, -1, out_dtype, stream()))
                else:   # few rows: lend split-K scratch, as a decoder session does
                    ok(lib().tnsr_b200_gemm_bf16_ws(ptr(a[i]), ptr(b[i]), None, None, ptr(o[i]), m, n, k, -1, out_dtype,
                                                    ptr(ws), ws.numel(), stream()))

            ms, _ = timed_graph(launch, sets, samples) if m <= 64 else timed(launch, sets, samples)
            ref = (a[0].float() @ b[0].float().T)
            launch(0)
            torch.cuda.synchronize()
            err = float((o[0].float() - ref).abs().max() / ref.abs().max())
            flops, nbytes = 2.0 * m * n * k, float(per_set)
            skinny = m <= 64
            emit(op="gemm_bf16", m=m, n=n, k=k, out=name, ms=ms, tflops=flops / ms / 1e9, frac_tensor=flops / ms / 1e9 / tf,
                 gbs=nbytes / ms / 1e6, frac_hbm=nbytes / ms / 1e6 / hbm, bound="hbm" if skinny else "tensor",
                 rel_err_vs_torch=err, operand_sets=sets, peaks=kind)
            del a, b, o


def bench_serving_gemms(samples):
    """The four projection shapes of configuration 4 at prefill (131 072 rows) and decode (256 rows) size."""
    hbm, tf, kind = peaks()
    g = torch.Generator(device="cuda").manual_seed(5)
    for rows in (131072, 256):
        for name, n, k, out_dtype, resid in (("qkv", 2304, 768, 1, False), ("attn_out", 768, 768, 0, True),
                                             ("gate_up", 4096, 768, 1, False), ("ffn_down", 768, 2048, 0, True)):
            osz = 2 if out_dtype else 4
            per_set = 2 * (rows * k + n * k) + osz * rows * n * (2 if resid else 1)
            sets = copies_for(per_set) if rows <= 1024 else 1    # small operands would otherwise sit in L2 between launches
            a = [(torch.randn((rows, k), device="cuda", generator=g)).to(torch.bfloat16) for _ in range(sets)]
            b = [(torch.randn((n, k), device="cuda", generator=g) * 0.02).to(torch.bfloat16) for _ in range(sets)]
            r = [torch.randn((rows, n), device="cuda", generator=g) if resid else None for _ in range(sets)]
            o = [torch.empty((rows, n), device="cuda", dtype=torch.bfloat16 if out_dtype else torch.float32) for _ in range(sets)]

            def launch(i):
                ok(lib().tnsr_b200_gemm_bf16(ptr(a[i]), ptr(b[i]), None, ptr(r[i]), ptr(o[i]), rows, n, k, -1, out_dtype, stream()))

            # decode-size launches are a few microseconds: time them inside a graph, as the decoder runs them
            ms, _ = timed_graph(launch, sets, samples) if rows <= 1024 else timed(launch, 1, samples)
            flops = 2.0 * rows * n * k
            emit(op="serving_gemm", which=name, rows=rows, n=n, k=k, out="bf16" if out_dtype else "f32+residual", ms=ms,
                 tflops=flops / ms / 1e9, frac_tensor=flops / ms / 1e9 / tf, operand_sets=sets,
                 timing="graph of back-to-back launches over rotating operand sets" if rows <= 1024 else "one launch between events",
                 peaks=kind)
            del a, b, r, o


def bench_mlp(samples):
    hbm, tf, kind = peaks()
    rows, d, f = 4096, 2048, 5632
    g = torch.Generator(device="cuda").manual_seed(3)
    x = torch.randn((rows, d), device="cuda", generator=g).to(torch.bfloat16)
    wg = (torch.randn((d, f), device="cuda", generator=g) * 0.02).to(torch.bfloat16)
    wu = (torch.randn((d, f), device="cuda", generator=g) * 0.02).to(torch.bfloat16)
    wd = (torch.randn((f, d), device="cuda", generator=g) * 0.02).to(torch.bfloat16)
    packed = torch.empty((2 * f, d), device="cuda", dtype=torch.bfloat16)
    ok(lib().tnsr_b200_pack_gate_up(ptr(wg), ptr(wu), None, None, ptr(packed), None, d, f, stream()))
    wdt = torch.empty((d, f), device="cuda", dtype=torch.bfloat16)
    ok(lib().tnsr_b200_transpose_bf16(ptr(wd), ptr(wdt), f, d, stream()))
    hidden = torch.empty((rows, f), device="cuda", dtype=torch.bfloat16)
    out = torch.empty((rows, d), device="cuda", dtype=torch.bfloat16)

    def launch(_):
        ok(lib().tnsr_b200_swiglu_mlp(ptr(x), ptr(packed), None, ptr(wdt), None, ptr(hidden), ptr(out), rows, d, f, stream()))

    ms, _ = timed(launch, 1, samples)
    ref = (torch.nn.functional.silu(x.float() @ wg.float()) * (x.float() @ wu.float())).to(torch.bfloat16).float() @ wd.float()
    err = float((out.float() - ref).abs().max() / ref.abs().max())
    flops = 3 * 2.0 * rows * d * f
    emit(op="swiglu_mlp", rows=rows, d=d, f=f, ms=ms, tflops=flops / ms / 1e9, frac_tensor=flops / ms / 1e9 / tf,
         rel_err_vs_torch=err, note="two launches: gate/up GEMM with SwiGLU epilogue, down GEMM; operands (170 MB) exceed L2",
         peaks=kind)


def bench_attention(samples, serving=False):
    """Configuration 3 (ragged lengths), or with serving=True the decode attention of configuration 4:
    256 sessions x 12 heads x 64 at 641 live keys (the mean over the 256 benchmark steps)."""
    hbm, _, kind = peaks()
    if serving:
        batch, heads, hd, capacity = 256, 12, 64, 769
        lengths = np.full(batch, 641, dtype=np.uint32)
    else:
        batch, heads, hd, capacity = 64, 16, 64, 4096
        lengths = np.random.default_rng(4).integers(1, capacity + 1, size=batch).astype(np.uint32)
    d = heads * hd
    g = torch.Generator(device="cuda").manual_seed(4)
    q = torch.randn((batch, d), device="cuda", generator=g).to(torch.bfloat16)
    kc = torch.randn((batch, capacity, d), device="cuda", generator=g).to(torch.bfloat16)
    vc = torch.randn((batch, capacity, d), device="cuda", generator=g).to(torch.bfloat16)
    ln = torch.from_numpy(lengths.view(np.int32)).cuda()
    out = torch.empty((batch, d), device="cuda", dtype=torch.bfloat16)
    ws_bytes = lib().tnsr_b200_decode_attention_workspace(batch, capacity, heads, hd)
    ws = torch.zeros(ws_bytes, dtype=torch.uint8, device="cuda")

    def launch(_):
        ok(lib().tnsr_b200_decode_attention(ptr(q), ptr(kc), ptr(vc), ptr(ln), ptr(out), ptr(ws), ws_bytes, batch, capacity,
                                            heads, hd, stream()))

    # plan + scan are a few launches of ~100 us in total: time a graph of 8 calls so that the host side (three ctypes
    # calls per launch) does not count; the live K/V rows (>= 505 MB) exceed L2 by themselves
    ms, _ = timed_graph(launch, 1, samples, reps=8)
    nbytes = float(lengths.astype(np.int64).sum()) * 4 * d + batch * 4 * d
    emit(op="decode_attention", batch=batch, heads=heads, head_dim=hd, capacity=capacity, live_keys=int(lengths.sum()),
         ms=ms, gbs=nbytes / ms / 1e6, frac_hbm=nbytes / ms / 1e6 / hbm, algorithmic_bytes=nbytes,
         note="plan + scan kernels per call (status-word memset included); live K/V (%.0f MB) exceeds L2" % (nbytes / 1e6),
         peaks=kind)


def bench_prefill_attention(samples, sessions=64):
    """Prefill attention of configuration 4 (512 new queries at position 0, 12 heads x 64, capacity 768) on both
    engines: tcgen05 (engine 0) and warp-level mma.sync (engine 1).  Causal FLOPs: 4 * hd per (query, visible key)."""
    _, tf, kind = peaks()
    heads, hd, chunk, position, capacity = 12, 64, 512, 0, 768
    d = heads * hd
    g = torch.Generator(device="cuda").manual_seed(6)
    q = torch.randn((sessions, chunk, d), device="cuda", generator=g).to(torch.bfloat16)
    kc = torch.randn((sessions, capacity, d), device="cuda", generator=g).to(torch.bfloat16)
    vc = torch.randn((sessions, capacity, d), device="cuda", generator=g).to(torch.bfloat16)
    out = torch.empty((sessions, chunk, d), device="cuda", dtype=torch.bfloat16)
    pairs = sessions * heads * sum(position + t + 1 for t in range(chunk))
    flops = 4.0 * hd * pairs
    results = {}
    for engine, name in ((0, "tcgen05"), (1, "mma.sync")):
        ok(lib().tnsr_b200_set_gemm_engine(engine))
        try:
            ms, _ = timed(lambda _: ok(lib().tnsr_b200_prefill_attention(ptr(q), ptr(kc), ptr(vc), ptr(out), sessions, chunk,
                                                                         position, capacity, heads, hd, stream())), 1, samples)
        finally:
            lib().tnsr_b200_set_gemm_engine(0)
        results[name] = out.float().clone()
        emit(op="prefill_attention", engine=name, sessions=sessions, chunk=chunk, position=position, heads=heads, head_dim=hd,
             ms=ms, causal_tflops=flops / ms / 1e9, frac_tensor=flops / ms / 1e9 / tf, peaks=kind)
    emit(op="prefill_attention", max_abs_difference_between_engines=float((results["tcgen05"] - results["mma.sync"]).abs().max()))


def bench_elementwise(samples):
    hbm, _, kind = peaks()
    rows, d = 131072, 768
    x = torch.randn((rows, d), device="cuda")
    w, b = torch.ones(d, device="cuda"), torch.zeros(d, device="cuda")
    y = torch.empty((rows, d), device="cuda", dtype=torch.bfloat16)
    ms, _ = timed(lambda _: ok(lib().tnsr_b200_layernorm(ptr(x), ptr(w), ptr(b), ptr(y), rows, d, 1e-5, 1, 0, stream())), 1, samples)
    nbytes = rows * d * 6.0
    emit(op="layernorm_f32_to_bf16", rows=rows, width=d, ms=ms, gbs=nbytes / ms / 1e6, frac_hbm=nbytes / ms / 1e6 / hbm, peaks=kind)
    n = 4096 * 5632 * 8
    gate = torch.randn(n, device="cuda").to(torch.bfloat16)
    up = torch.randn(n, device="cuda").to(torch.bfloat16)
    o = torch.empty(n, device="cuda", dtype=torch.bfloat16)
    ms, _ = timed(lambda _: ok(lib().tnsr_b200_swiglu(ptr(gate), ptr(up), ptr(o), n, stream())), 1, samples)
    emit(op="swiglu_elementwise", elems=n, ms=ms, gbs=6.0 * n / ms / 1e6, frac_hbm=6.0 * n / ms / 1e6 / hbm, peaks=kind)
    rows, vocab = 4096, 32000
    logits = torch.randn((rows, vocab), device="cuda")
    ids = torch.empty(rows, device="cuda", dtype=torch.int32)
    ms, _ = timed(lambda _: ok(lib().tnsr_b200_argmax(ptr(logits), ptr(ids), rows, vocab, stream())), 1, samples)
    nbytes = rows * vocab * 4.0
    emit(op="argmax", rows=rows, vocab=vocab, ms=ms, gbs=nbytes / ms / 1e6, frac_hbm=nbytes / ms / 1e6 / hbm, peaks=kind)


def bench_grouped_attention(samples, sessions, chunk, position, heads, kv_heads, hd, softcap, name, window=0, scores="softmax"):
    """Grouped-query attention with capped scores and gates: `chunk` queries per session after `position` cached rows.
    Algorithmic bytes: the live K/V rows and q / out once; flops: 4 hd per (query, head, visible key)."""
    hbm, tf, kind = peaks()
    capacity = position + chunk
    g = torch.Generator(device="cuda").manual_seed(8)
    randn = lambda *shape: torch.randn(shape, device="cuda", generator=g).to(torch.bfloat16)
    live = min(position + chunk, window + chunk - 1) if window else position + chunk
    nbytes = sessions * 2.0 * (live * kv_heads * 2 * hd + chunk * heads * 2 * hd)
    sets = copies_for(int(nbytes))
    q = [randn(sessions * chunk, heads * hd) for _ in range(sets)]
    k = [randn(sessions, capacity, kv_heads * hd) for _ in range(sets)]
    v = [randn(sessions, capacity, kv_heads * hd) for _ in range(sets)]
    gate = torch.randn((sessions * chunk, 32), device="cuda", generator=g)
    out = torch.empty((sessions * chunk, heads * hd), device="cuda", dtype=torch.bfloat16)
    size = lib().tnsr_b200_grouped_attention_workspace(hd, hd)
    ws = torch.zeros(size, dtype=torch.uint8, device="cuda")
    where = _native.Place(sessions, chunk, position, 0, None)
    args = [_native.GroupedAttentionArgs(q[i].data_ptr(), k[i].data_ptr(), v[i].data_ptr(), gate.data_ptr(), out.data_ptr(), ws.data_ptr(), None, size,
                                         heads, kv_heads, hd, hd, capacity, 32, heads * hd, heads * hd, hd ** -0.5, softcap, 1, 0,
                                         gate.data_ptr() if scores == "sigmoid" else None, window, _native.SCORE[scores], 1.0, 0) for i in range(sets)]
    if scores == "sigmoid":
        for a in args:
            a.gate = None
    ms, _ = timed_graph(lambda i: ok(lib().tnsr_b200_grouped_attention(C.byref(args[i]), C.byref(where), stream())), sets, samples, reps=8)
    pairs = sessions * heads * sum(min(position + t + 1, window or position + t + 1) for t in range(chunk))
    flops = 4.0 * hd * pairs
    emit(op="grouped_attention", window=window, scores=scores, case=name, sessions=sessions, chunk=chunk, position=position, heads=heads, kv_heads=kv_heads, head_dim=hd,
         softcap=softcap, ms=ms, gbs=nbytes / ms / 1e6, frac_hbm=nbytes / ms / 1e6 / hbm, tflops=flops / ms / 1e9, frac_tensor=flops / ms / 1e9 / tf,
         peaks=kind)


def bench_mamba2(samples, sessions, chunk, heads, vdim, state, groups, name):
    """The mamba2 mixer between its projections.  Algorithmic bytes: projected rows in, mixer rows out, the f32 state in and
    out; flops of the chunked form (chunks of 64): C B^T (causal half), weights x, C S and B x^T per head."""
    hbm, tf, kind = peaks()
    inner, gn = heads * vdim, groups * state
    channels, proj = inner + 2 * gn, 2 * inner + 2 * gn
    rows = sessions * chunk
    g = torch.Generator(device="cuda").manual_seed(9)
    nbytes = rows * 2.0 * (proj + inner) + rows * 4.0 * heads + sessions * heads * state * vdim * 8.0
    sets = min(8, copies_for(int(nbytes)))
    ld = (proj + 31) // 32 * 32
    u = [torch.randn((rows, ld), device="cuda", generator=g).to(torch.bfloat16) for _ in range(sets)]
    ssm = [torch.zeros((sessions, heads, state, vdim), device="cuda") for _ in range(sets)]
    dt = torch.randn((rows, heads), device="cuda", generator=g)
    f32 = lambda *shape: torch.rand(shape, device="cuda", generator=g)
    conv, conv_b, vec, norm = f32(channels, 4), f32(channels), f32(heads), f32(inner)
    ring = torch.zeros((sessions, 4, channels), device="cuda", dtype=torch.bfloat16)
    xbc = torch.empty((rows, channels), device="cuda", dtype=torch.bfloat16)
    gated = torch.empty((rows, inner), device="cuda", dtype=torch.bfloat16)
    out = torch.empty((rows, inner), device="cuda", dtype=torch.bfloat16)
    where = _native.Place(sessions, chunk, 64, 0, None)
    args = [_native.Mamba2Args(u[i].data_ptr(), dt.data_ptr(), conv.data_ptr(), conv_b.data_ptr(), vec.data_ptr(), vec.data_ptr(), vec.data_ptr(),
                               norm.data_ptr(), ring.data_ptr(), ssm[i].data_ptr(), xbc.data_ptr(), gated.data_ptr(), out.data_ptr(), ld, heads,
                               heads, vdim, state, groups, groups, 4, inner, inner, 1e-5, 1, 0, 0) for i in range(sets)]
    ms, _ = timed_graph(lambda i: ok(lib().tnsr_b200_mamba2(C.byref(args[i]), C.byref(where), stream())), sets, samples, reps=8)
    q = 64
    flops = rows * (2.0 * q * state * groups / 2 + heads * (2.0 * q * vdim / 2 + 4.0 * state * vdim)) if chunk > 1 else rows * heads * 6.0 * state * vdim
    emit(op="mamba2", case=name, sessions=sessions, chunk=chunk, heads=heads, vdim=vdim, state=state, groups=groups, ms=ms, gbs=nbytes / ms / 1e6,
         frac_hbm=nbytes / ms / 1e6 / hbm, tflops=flops / ms / 1e9, frac_tensor=flops / ms / 1e9 / tf, peaks=kind)


def bench_mixers(samples):
    """Beside the GPT kernels of the same sizes (serving_attention, prefill_attention, elementwise)."""
    bench_attention(samples, serving=True)
    bench_grouped_attention(samples, 256, 1, 640, 12, 12, 64, 30.0, "decode, a key/value head per head")
    bench_grouped_attention(samples, 256, 1, 640, 12, 4, 64, 30.0, "decode, 3 heads per key/value head")
    bench_grouped_attention(samples, 64, 1, 1536, 16, 2, 128, 30.0, "decode, 8 heads of 128 per key/value head")
    bench_grouped_attention(samples, 1, 1, 8191, 12, 4, 64, 30.0, "decode, one long session")
    bench_prefill_attention(samples)
    bench_grouped_attention(samples, 64, 512, 0, 12, 12, 64, 30.0, "prefill, a key/value head per head")
    bench_grouped_attention(samples, 64, 512, 0, 12, 12, 64, 0.0, "prefill, a key/value head per head, no cap")
    bench_grouped_attention(samples, 64, 512, 0, 12, 4, 64, 30.0, "prefill, 3 heads per key/value head")
    bench_grouped_attention(samples, 16, 1024, 0, 16, 2, 128, 30.0, "prefill, 8 heads of 128 per key/value head")
    bench_mamba2(samples, 256, 1, 24, 64, 128, 1, "decode")
    bench_mamba2(samples, 32, 1, 24, 64, 128, 1, "decode, 32 sessions")
    bench_mamba2(samples, 64, 512, 24, 64, 128, 1, "prefill")
    bench_mamba2(samples, 256, 512, 24, 64, 128, 1, "prefill, 256 sessions")
    bench_mamba2(samples, 1, 4096, 24, 64, 128, 1, "prefill, one long prompt")
    hbm, _, kind = peaks()
    rows, d = 131072, 768
    x, w = torch.randn((rows, d), device="cuda"), torch.ones(d, device="cuda")
    y = torch.empty((rows, d), device="cuda", dtype=torch.bfloat16)
    ms, _ = timed(lambda _: ok(lib().tnsr_b200_rmsnorm(ptr(x), ptr(w), 1.0, ptr(y), rows, d, 1e-5, 1, stream())), 1, samples)
    nbytes = rows * d * 6.0
    emit(op="rmsnorm_f32_to_bf16", rows=rows, width=d, ms=ms, gbs=nbytes / ms / 1e6, frac_hbm=nbytes / ms / 1e6 / hbm, peaks=kind)


def bench_hgrn2(samples, sessions, chunk, heads, dim, vdim, name):
    """HGRN2 between its projections.  Algorithmic bytes: q, v (bf16) and gates (f32) in, bf16 rows out, the f32 state in and
    out; flops: q S and k v^T per token and head (the inner weights of a chunk are small beside them)."""
    hbm, tf, kind = peaks()
    k, inner, rows = heads * dim, heads * vdim, sessions * chunk
    nbytes = rows * (2.0 * (k + inner) + 4.0 * k + 2.0 * inner) + sessions * heads * dim * vdim * 8.0
    sets = min(8, copies_for(int(nbytes)))
    g = torch.Generator(device="cuda").manual_seed(10)
    u = [torch.randn((rows, k + inner), device="cuda", generator=g).to(torch.bfloat16) for _ in range(sets)]
    f = [torch.randn((rows, k), device="cuda", generator=g) for _ in range(sets)]
    state = [torch.zeros((sessions, heads, dim, vdim), device="cuda") for _ in range(sets)]
    bias, lower, norm = torch.full((k,), 3.0, device="cuda"), torch.rand(k, device="cuda", generator=g) * 0.9, torch.ones(vdim, device="cuda")
    out = torch.empty((rows, inner), device="cuda", dtype=torch.bfloat16)
    raw = torch.empty((rows, inner), device="cuda")
    where = _native.Place(sessions, chunk, 64, 0, None)
    args = [_native.Hgrn2Args(u[i].data_ptr(), u[i].data_ptr() + 2 * k, f[i].data_ptr(), bias.data_ptr(), lower.data_ptr(), norm.data_ptr(), state[i].data_ptr(),
                              raw.data_ptr(), out.data_ptr(), k + inner, k, heads, dim, vdim, inner, inner, 1e-5, 1.0, 1, 0, 0) for i in range(sets)]
    ms, _ = timed_graph(lambda i: ok(lib().tnsr_b200_hgrn2(C.byref(args[i]), C.byref(where), stream())), sets, samples, reps=8)
    flops = rows * heads * 4.0 * dim * vdim
    emit(op="hgrn2", case=name, sessions=sessions, chunk=chunk, heads=heads, dim=dim, vdim=vdim, ms=ms, gbs=nbytes / ms / 1e6, frac_hbm=nbytes / ms / 1e6 / hbm,
         tflops=flops / ms / 1e9, frac_tensor=flops / ms / 1e9 / tf, peaks=kind)


def bench_rglru(samples, sessions, chunk, width, blocks, name):
    """The recurrent unit between its projections: convolution, gate products, scan.  Algorithmic bytes: y and x in, rows out,
    the convolved rows and the f32 gates out and in, the state in and out."""
    hbm, _, kind = peaks()
    rows, part = sessions * chunk, width // blocks
    nbytes = rows * width * (2.0 * 3 + 2.0 * 3 + 8.0 * 2) + sessions * width * 8.0 + 4.0 * width * part
    sets = min(8, copies_for(int(nbytes)))
    g = torch.Generator(device="cuda").manual_seed(11)
    u = [torch.randn((rows, 2 * width), device="cuda", generator=g).to(torch.bfloat16) for _ in range(sets)]
    w = (torch.randn((blocks, 2 * part, part), device="cuda", generator=g) * part ** -0.5).to(torch.bfloat16)
    conv, vec, lam = torch.rand((width, 4), device="cuda", generator=g), torch.zeros(width, device="cuda"), torch.full((width,), -5.0, device="cuda")
    ring, state = torch.zeros((sessions, 4, width), device="cuda", dtype=torch.bfloat16), torch.zeros((sessions, width), device="cuda")
    conv_out, gates = torch.empty((rows, width), device="cuda", dtype=torch.bfloat16), torch.empty((rows, 2 * width), device="cuda")
    out = torch.empty((rows, width), device="cuda", dtype=torch.bfloat16)
    where = _native.Place(sessions, chunk, 64, 0, None)
    args = [_native.RglruArgs(u[i].data_ptr(), w.data_ptr(), conv.data_ptr(), vec.data_ptr(), vec.data_ptr(), vec.data_ptr(), lam.data_ptr(), ring.data_ptr(),
                              state.data_ptr(), conv_out.data_ptr(), gates.data_ptr(), out.data_ptr(), None, 2 * width, width, width, blocks, 4, width, width,
                              1) for i in range(sets)]
    ms, _ = timed_graph(lambda i: ok(lib().tnsr_b200_rglru(C.byref(args[i]), C.byref(where), stream())), sets, samples, reps=8)
    emit(op="rglru", case=name, sessions=sessions, chunk=chunk, width=width, blocks=blocks, ms=ms, gbs=nbytes / ms / 1e6, frac_hbm=nbytes / ms / 1e6 / hbm,
         peaks=kind)


def bench_grouped_gemm(samples, groups, rows, n, k, activation, name):
    """One product per group of rows (sizes of a uniform routing).  Flops of the real rows; bytes: rows, weights, results."""
    hbm, tf, kind = peaks()
    rng = np.random.default_rng(12)
    counts = np.bincount(rng.integers(0, groups, rows), minlength=groups)
    offsets = torch.from_numpy(np.concatenate([[0], np.cumsum(counts)]).astype(np.int32)).cuda()
    nbytes = 2.0 * (rows * (n + k) + (counts > 0).sum() * n * k)
    sets = min(16, copies_for(int(nbytes)))
    g = torch.Generator(device="cuda").manual_seed(13)
    a = [torch.randn((rows, k), device="cuda", generator=g).to(torch.bfloat16) for _ in range(sets)]
    w = [(torch.randn((groups, n, k), device="cuda", generator=g) * 0.02).to(torch.bfloat16) for _ in range(sets)]
    out = torch.empty((rows, n), device="cuda", dtype=torch.bfloat16)
    status = torch.zeros(1, device="cuda", dtype=torch.int32)
    ms, _ = timed_graph(lambda i: ok(lib().tnsr_b200_gemm_grouped(ptr(a[i]), ptr(w[i]), ptr(out), ptr(offsets), groups, rows, n, k, activation, 1, 1, 0,
                                                                  ptr(status), stream())), sets, samples, reps=8)
    flops = 2.0 * rows * n * k
    emit(op="gemm_grouped", case=name, groups=groups, rows=rows, n=n, k=k, ms=ms, tflops=flops / ms / 1e9, frac_tensor=flops / ms / 1e9 / tf,
         gbs=nbytes / ms / 1e6, frac_hbm=nbytes / ms / 1e6 / hbm, peaks=kind)


def bench_experts(samples, rows, d, ff, experts, identity, top, name):
    """Routing, gather, both products and the weighted sum with the next norm.  Flops of the products of real experts."""
    hbm, tf, kind = peaks()
    total = experts + identity
    g = torch.Generator(device="cuda").manual_seed(14)
    logits, correction = torch.randn((rows, total), device="cuda", generator=g), torch.zeros(total, device="cuda")
    h = torch.randn((rows, d), device="cuda", generator=g).to(torch.bfloat16)
    up = (torch.randn((experts, ff, d), device="cuda", generator=g) * 0.02).to(torch.bfloat16)
    down = (torch.randn((experts, d, ff), device="cuda", generator=g) * 0.02).to(torch.bfloat16)
    x, one, normed = torch.zeros((rows, d), device="cuda"), torch.ones(d, device="cuda"), torch.empty((rows, d), device="cuda", dtype=torch.bfloat16)
    size = lib().tnsr_b200_experts_workspace(rows, d, ff, experts, top, 1)
    ws = torch.empty(size, dtype=torch.uint8, device="cuda")
    status = torch.zeros(1, device="cuda", dtype=torch.int32)
    args = _native.ExpertsArgs(logits.data_ptr(), correction.data_ptr(), h.data_ptr(), up.data_ptr(), down.data_ptr(), x.data_ptr(), one.data_ptr(),
                               one.data_ptr(), normed.data_ptr(), ws.data_ptr(), size, None, None, status.data_ptr(), rows, total, d, ff, experts, identity,
                               top, 1.0, 1.0, 1e-5, 1, 0)
    ms, _ = timed_graph(lambda _: ok(lib().tnsr_b200_experts(C.byref(args), stream())), 1, samples, reps=8)
    pairs = rows * top * experts / total
    flops, weights = pairs * 4.0 * d * ff, min(experts, pairs) * 4.0 * d * ff
    nbytes = weights + rows * (2.0 * d * 2 + 4.0 * d * 2) + pairs * (2.0 * d * 4 + 2.0 * ff * 2)
    emit(op="experts", case=name, rows=rows, d=d, ff=ff, experts=experts, identity=identity, top=top, ms=ms, tflops=flops / ms / 1e9,
         frac_tensor=flops / ms / 1e9 / tf, gbs=nbytes / ms / 1e6, frac_hbm=nbytes / ms / 1e6 / hbm, peaks=kind)


def bench_polynorm(samples, rows, width):
    hbm, _, kind = peaks()
    z, act = torch.randn((rows, width), device="cuda").to(torch.bfloat16), torch.tensor([0.5, 0.3, 0.2, 0.0], device="cuda")
    out = torch.empty_like(z)
    ms, _ = timed(lambda _: ok(lib().tnsr_b200_polynorm(ptr(z), ptr(act), ptr(out), rows, width, width, width, 1e-5, 1, stream())), 1, samples)
    nbytes = rows * width * 4.0
    emit(op="polynorm", rows=rows, width=width, ms=ms, gbs=nbytes / ms / 1e6, frac_hbm=nbytes / ms / 1e6 / hbm, peaks=kind)


def bench_rotary(samples, sessions, chunk, heads, kv_heads, hd):
    hbm, _, kind = peaks()
    rows, cols = sessions * chunk, (heads + 2 * kv_heads) * hd
    u = torch.randn((rows, cols), device="cuda").to(torch.bfloat16)
    table = torch.rand((chunk, hd), device="cuda")
    q = torch.empty((rows, heads * hd), device="cuda", dtype=torch.bfloat16)
    k, v = (torch.empty((rows, kv_heads * hd), device="cuda", dtype=torch.bfloat16) for _ in range(2))
    args = _native.RotaryArgs(u.data_ptr(), table.data_ptr(), q.data_ptr(), k.data_ptr(), v.data_ptr(), cols, heads, kv_heads, hd, hd, hd, 1, chunk, 1, 0)
    where = _native.Place(sessions, chunk, 0, 0, None)
    ms, _ = timed(lambda _: ok(lib().tnsr_b200_rotary(C.byref(args), C.byref(where), stream())), 1, samples)
    nbytes = rows * cols * 4.0
    emit(op="rotary", rows=rows, heads=heads, kv_heads=kv_heads, head_dim=hd, ms=ms, gbs=nbytes / ms / 1e6, frac_hbm=nbytes / ms / 1e6 / hbm, peaks=kind)


def bench_ganupel(samples):
    """Beside the like kernels of Bolonex (mixers) and of the GPT (serving_gemms, elementwise)."""
    bench_grouped_attention(samples, 256, 1, 640, 12, 4, 64, 30.0, "Bolonex decode")
    bench_grouped_attention(samples, 256, 1, 640, 12, 4, 64, 0.0, "decode, window 256", 256, "sigmoid")
    bench_grouped_attention(samples, 256, 1, 640, 12, 4, 64, 0.0, "decode, no window", 0, "sigmoid")
    bench_grouped_attention(samples, 64, 512, 0, 12, 4, 64, 30.0, "Bolonex prefill")
    bench_grouped_attention(samples, 64, 512, 0, 12, 4, 64, 0.0, "prefill, window 256", 256, "sigmoid")
    bench_grouped_attention(samples, 64, 512, 0, 12, 4, 64, 0.0, "prefill, no window", 0, "sigmoid")
    bench_mamba2(samples, 256, 1, 24, 64, 128, 1, "Bolonex decode")
    bench_hgrn2(samples, 256, 1, 12, 64, 64, "decode")
    bench_hgrn2(samples, 256, 1, 8, 128, 128, "decode, 128 x 128")
    bench_hgrn2(samples, 32, 1, 12, 64, 64, "decode, 32 sessions")
    bench_mamba2(samples, 256, 512, 24, 64, 128, 1, "Bolonex prefill, 256 sessions")
    bench_hgrn2(samples, 256, 512, 12, 64, 64, "prefill, 256 sessions")
    bench_hgrn2(samples, 64, 1024, 8, 128, 128, "prefill, 128 x 128")
    bench_hgrn2(samples, 64, 512, 12, 128, 64, "prefill, 128 x 64")
    bench_hgrn2(samples, 1, 4096, 12, 64, 64, "prefill, one long prompt")
    bench_rglru(samples, 256, 1, 1024, 8, "decode")
    bench_rglru(samples, 256, 512, 1024, 8, "prefill, 256 sessions")
    bench_rglru(samples, 1, 4096, 1024, 8, "prefill, one long prompt")
    bench_polynorm(samples, 131072, 3072)
    bench_rotary(samples, 256, 512, 12, 4, 64)
    bench_grouped_gemm(samples, 16, 131072 * 4, 768, 768, 4, "up, prefill")
    bench_grouped_gemm(samples, 16, 131072 * 4, 768, 768, -1, "down, prefill")
    bench_grouped_gemm(samples, 32, 65536 * 4, 1024, 1024, 4, "up, prefill, 32 experts")
    bench_grouped_gemm(samples, 16, 256 * 4, 768, 768, 4, "up, decode of 256")
    bench_grouped_gemm(samples, 64, 64 * 4, 1024, 1024, 4, "up, decode of 64, 64 experts")
    bench_experts(samples, 131072, 768, 768, 16, 2, 4, "prefill")
    bench_experts(samples, 256, 768, 768, 16, 2, 4, "decode of 256")
    bench_experts(samples, 32, 768, 768, 16, 2, 4, "decode of 32")


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("what", choices=["gemm", "skinny_gemm", "serving_gemms", "mlp", "attention", "serving_attention", "elementwise", "prefill_attention", "mixers", "ganupel", "all"])
    ap.add_argument("--samples", type=int, default=20)
    args = ap.parse_args()
    if not torch.cuda.is_available():
        sys.exit("opbench needs a CUDA device")
    todo = (["gemm", "serving_gemms", "mlp", "attention", "serving_attention", "elementwise", "prefill_attention", "mixers", "ganupel"]
            if args.what == "all" else [args.what])
    for name in todo:
        {"gemm": bench_gemm, "skinny_gemm": lambda n: bench_gemm(n, shapes=[(m, 4096, 4096) for m in (1, 8, 64)], outs=("bf16",)),
         "serving_gemms": bench_serving_gemms, "mlp": bench_mlp, "attention": bench_attention,
         "serving_attention": lambda n: bench_attention(n, serving=True),
         "elementwise": bench_elementwise, "prefill_attention": bench_prefill_attention, "mixers": bench_mixers, "ganupel": bench_ganupel}[name](args.samples)


if __name__ == "__main__":
    main()
