"""`python bench.py --workload dugulorn`: prompt passes and decode steps of the Dugulorn family at sizes that resemble a real
model's layers (random weights), beside Pefolix at equal width, heads and feed-forward, and the kernels of both one by one
against their rooflines. One JSON line, one GPU; how things are timed is in bench_pefolix.py.

Rooflines: bytes over the measured copy rate, 16-bit products over the measured bf16 rate, and for the recurrences, whose
arithmetic is 32-bit, operations of the recurrence as it is written over the nominal f32 rate of the FMA pipes.
"""
from __future__ import annotations

import ctypes as C
import json
import tempfile
from pathlib import Path

from bench_pefolix import CONTEXT, fast_checkpoint, graph_us, time_model

ROT, Q_RANK, KV_RANK, TAPS, LOW = 64, 1536, 512, 4, 128
F32_TFLOPS = 148 * 128 * 2 * 1.965e9 / 1e12
# name: width, heads, head size, feed-forward, layers (of the pattern below), vocabulary
MODELS = {"2560 wide": (2560, 20, 128, 6912, 8, 32000), "4096 wide": (4096, 32, 128, 14336, 4, 32000)}
PEFOLIX = {"2560 wide": (2560, 20, 5, 128, 6912, 8, 32000), "4096 wide": (4096, 32, 8, 128, 14336, 4, 32000)}
MIXERS = ("mixed", "latent", "lightning", "delta")


def config(dg, name, kind="mixed"):
    W, H, D, F, L, V = MODELS[name]
    decay = [0.5 + 0.499 * h / H for h in range(H)]
    layers = []
    for i in range(L):
        k = ("lightning", "latent", "delta", "shared")[i % 4] if kind == "mixed" else kind
        if k in ("latent", "shared"):
            layers.append(dg.latent_layer(H, D, ROT, D, Q_RANK, KV_RANK, None, 1e6, dg.yarn(4.0, 4096), i - 2 if k == "shared" else None, F))
        elif k == "lightning":
            layers.append(dg.lightning_layer(H, D, D, decay, F))
        else:
            layers.append(dg.delta_layer(H, H, D, D, TAPS, F))
    return dg.make_config(V, W, layers)


def step_bytes(cfg, dg, batch):
    """HBM bytes of a decode step: weights once, the head, latents of the context, states twice."""
    n = 0
    for name, shape in dg.tensor_shapes(cfg, LOW):
        size = 2
        for d in shape:
            size *= d
        n += size if name != "embed" else 0
    n += 2 * cfg["vocab"] * cfg["width"]
    for layer in cfg["layers"]:
        mx = layer["mixer"]
        if layer["type"] == "latent_attention":
            n += batch * CONTEXT * (mx["kv_rank"] + mx["rot_dim"]) * 2
        else:
            n += batch * mx["heads"] * mx["dim"] * mx["vdim"] * 8
    return n


def kernels(torch, ctx, peaks):
    from lemonade_burn_b200 import _lib, mixers
    lib, chk, h = _lib.load(), _lib.check, ctx.handle
    hbm, tc16 = peaks["hbm_gbs"], peaks["bf16_tflops"]
    st = lambda: torch.cuda.current_stream().cuda_stream
    rows = []

    def add(kind, what, family, us, nbytes=0, flops=0, f32=0):
        t = {"HBM": nbytes / hbm / 1e3, "tensor": flops / tc16 / 1e6, "f32": f32 / F32_TFLOPS / 1e6}
        bound = max(t, key=t.get)
        rows.append({"kind": kind, "what": what, "family": family, "us": round(us, 2), "roofline_us": round(t[bound], 2), "bound": bound,
                     "fraction": round(t[bound] / us, 3)})

    def bf16(*s):
        return (torch.randn(*s, device="cuda") * 0.02).to(torch.bfloat16)

    # projections of the mixers and feed-forwards (the same kernels as Pefolix's; bias and activation in the epilogue)
    for W, F, H in ((2560, 6912, 20), (4096, 14336, 32)):
        shapes = (("up + bias + relu^2", F, W, 1), ("gate/up", F, W, 2), ("lightning q/k/v/g + silu", 4 * H * 128, W, 0), ("latent in", Q_RANK + KV_RANK + ROT + H, W, 3),
                  ("latent queries", H * (128 + ROT), Q_RANK, 3))
        for m in (1, 16, 2048):
            for name, r, c, kind in shapes:
                gated = kind == 2
                wr = r * (2 if gated else 1)
                nbytes = wr * c * 2
                copies = max(2, min(40, int(300e6 / nbytes) + 1)) if m < 2048 else 2
                ws = [bf16(wr, c) for _ in range(copies)]
                x, bias = bf16(m, c), torch.zeros(wr, device="cuda")
                f32 = kind == 3
                out = torch.zeros(m, r, device="cuda", dtype=torch.float32 if f32 else torch.bfloat16)
                if gated:
                    calls = [(lambda w=w: chk(lib.lbk_dense_linear(h, 0, x.data_ptr(), c, m, w.data_ptr(), c, wr, c, 1, r, 0, out.data_ptr(), r, 0, None, 0, st()))) for w in ws]
                else:
                    act, to = ((1, r) if kind == 1 else (2, r * 3 // 4)) if kind < 2 else (0, r)
                    calls = [(lambda w=w: chk(lib.lbk_dense_linear_act(h, 0, x.data_ptr(), c, m, w.data_ptr(), c, r, c, bias.data_ptr() if kind == 1 else None, act, to,
                                                                       out.data_ptr(), r, int(f32), st()))) for w in ws]
                us = graph_us(torch, calls * (1 if m < 2048 else 5))
                if not gated:  # the like kernel at equal size: the same projection with Pefolix's epilogue
                    plain = [(lambda w=w: chk(lib.lbk_dense_linear(h, 0, x.data_ptr(), c, m, w.data_ptr(), c, wr, c, 0, r, 0, out.data_ptr(), r, int(f32), None, 0, st()))) for w in ws]
                    add("projection", f"{c} -> {r}, {m} tokens", "Pefolix", graph_us(torch, plain * (1 if m < 2048 else 5)), nbytes + m * c * 2 + out.numel() * out.element_size(), 2.0 * m * wr * c)
                add("projection", f"{name} {c} -> {r}, {m} tokens", "Pefolix" if gated else "Dugulorn", us, nbytes + m * c * 2 + out.numel() * out.element_size(), 2.0 * m * wr * c)
                del ws
        torch.cuda.empty_cache()

    freq, factor = mixers.rotation_frequencies(ROT, 1e6, (4.0, 4096.0, 32.0, 1.0))
    fd = torch.from_numpy(freq).cuda()
    # decode: latent attention over 4096 positions, recurrences; Pefolix's attention over as many keys
    for b, nh, kvh in ((1, 20, 5), (16, 20, 5), (16, 32, 8)):
        pos, cap, sets = CONTEXT - 1, CONTEXT + 64, 2 if b > 1 else 24
        posd = torch.full((b,), pos, dtype=torch.int32, device="cuda")
        d = mixers.LatentDesc(nh, 128, ROT, 128, KV_RANK, Q_RANK, fd.data_ptr(), factor)
        pitch, qp = lib.lbk_latent_pitch(C.byref(d)), lib.lbk_latent_query_pitch(C.byref(d))
        caches = [bf16(b, cap, pitch) for _ in range(sets)]
        ukvs = [bf16(nh * 256, KV_RANK) for _ in range(sets)]
        q, gate, out = bf16(b, nh, qp), torch.zeros(b, nh, device="cuda"), bf16(b, nh * 128)
        work = torch.empty(lib.lbk_latent_work_bytes(h, 0, C.byref(d), b, cap, 0), dtype=torch.uint8, device="cuda")
        calls = [(lambda k=k, w=w: chk(lib.lbk_latent_attn(h, 0, C.byref(d), q.data_ptr(), b, -1, posd.data_ptr(), cap, k.data_ptr(), w.data_ptr(), KV_RANK, 0.07,
                                                           gate.data_ptr(), nh, 0, work.data_ptr(), out.data_ptr(), nh * 128, st()))) for k, w in zip(caches, ukvs)]
        add("decode attention", f"latent, {b} sequences, {nh} heads, {CONTEXT} positions", "Dugulorn", graph_us(torch, calls * 8), b * CONTEXT * (KV_RANK + ROT) * 2 + nh * 256 * KV_RANK * 2,
            2.0 * b * nh * CONTEXT * (2 * KV_RANK + ROT))
        del caches, ukvs
        kv = [(bf16(b, kvh, cap, 128), bf16(b, kvh, cap, 128)) for _ in range(2 if b > 1 else 16)]
        q16, o16 = bf16(b, nh, 128), bf16(b, nh * 128)
        scr = torch.empty(int(lib.lbk_attn_window_scratch(b, nh, 128)), device="cuda")
        calls = [(lambda k=k, v=v: chk(lib.lbk_attn_window(h, 0, q16.data_ptr(), k.data_ptr(), v.data_ptr(), posd.data_ptr(), b, -1, nh, kvh, 128, 128, 128, 128, cap, 0.088, 0, 0, 1,
                                                           scr.data_ptr(), o16.data_ptr(), nh * 128, st()))) for k, v in kv]
        add("decode attention", f"{b} sequences, {nh}/{kvh} heads, {CONTEXT} keys", "Pefolix", graph_us(torch, calls * 8), b * kvh * CONTEXT * 512)
        del kv
        for delta in (0, 1):
            rd = mixers.RecurrenceDesc(delta, nh, nh, 128, 128, TAPS)
            width = 3 * nh * 128
            x, o = bf16(b, width), torch.zeros(b, nh * 128, device="cuda")
            states = [torch.zeros(b * lib.lbk_recurrence_state_floats(C.byref(rd)), device="cuda") for _ in range(max(2, int(300e6 / (b * nh * 65536)) + 1))]
            conv, ring = torch.randn(TAPS, width, device="cuda"), bf16(b, TAPS, width)
            a, al, dt, be, dec = torch.randn(b, nh * 128, device="cuda"), torch.zeros(nh, device="cuda"), torch.zeros(nh * 128, device="cuda"), torch.zeros(b, nh, device="cuda"), torch.full((nh,), 0.9, device="cuda")
            calls = [(lambda s=s: chk(lib.lbk_recurrence(h, 0, C.byref(rd), x.data_ptr(), width, b, -1, posd.data_ptr(), None, cap, dec.data_ptr(), conv.data_ptr(), ring.data_ptr(), a.data_ptr(),
                                                         al.data_ptr(), dt.data_ptr(), be.data_ptr(), s.data_ptr(), None, 0, o.data_ptr(), st()))) for s in states]
            add("decode recurrence", f"{'delta rule' if delta else 'lightning'}, {b} sequences, {nh} heads of 128 x 128", "Dugulorn", graph_us(torch, calls * 4), b * nh * 128 * 128 * 8)
            del states
    for n, nh, kvh in ((2048, 20, 5), (2048, 32, 8)):
        pos0, cap = torch.zeros(1, dtype=torch.int32, device="cuda"), n
        d = mixers.LatentDesc(nh, 128, ROT, 128, KV_RANK, Q_RANK, fd.data_ptr(), factor)
        pitch, qp = lib.lbk_latent_pitch(C.byref(d)), lib.lbk_latent_query_pitch(C.byref(d))
        cache, ukv, q = bf16(1, cap, pitch), bf16(nh * 256, KV_RANK), bf16(n, nh, qp)
        gate, out = torch.zeros(n, nh, device="cuda"), bf16(n, nh * 128)
        work = torch.empty(lib.lbk_latent_work_bytes(h, 0, C.byref(d), n, cap, n), dtype=torch.uint8, device="cuda")
        us = graph_us(torch, [lambda: chk(lib.lbk_latent_attn(h, 0, C.byref(d), q.data_ptr(), n, 0, pos0.data_ptr(), cap, cache.data_ptr(), ukv.data_ptr(), KV_RANK, 0.07, gate.data_ptr(), nh,
                                                              n, work.data_ptr(), out.data_ptr(), nh * 128, st()))] * 10)
        add("prompt attention", f"latent, {n} rows, {nh} heads (keys and values written out, rotation, attention)", "Dugulorn", us,
            flops=2.0 * n * nh * 256 * KV_RANK + 2.0 * nh * (256 + ROT) * n * (n + 1) / 2)
        k, v = bf16(1, kvh, n, 128), bf16(1, kvh, n, 128)
        q16, o16 = bf16(n, nh, 128), bf16(n, nh * 128)
        us = graph_us(torch, [lambda: chk(lib.lbk_attn_window(h, 0, q16.data_ptr(), k.data_ptr(), v.data_ptr(), pos0.data_ptr(), n, 0, nh, kvh, 128, 128, 128, 128, cap, 0.088, 0, 0, 1, None,
                                                              o16.data_ptr(), nh * 128, st()))] * 10)
        add("prompt attention", f"{n} rows, {nh}/{kvh} heads", "Pefolix", us, flops=4.0 * nh * 128 * n * (n + 1) / 2)
        for delta in (0, 1):
            rd = mixers.RecurrenceDesc(delta, nh, nh, 128, 128, TAPS)
            width = 3 * nh * 128
            x, o = bf16(n, width), torch.zeros(n, nh * 128, device="cuda")
            state = torch.zeros(lib.lbk_recurrence_state_floats(C.byref(rd)), device="cuda")
            rr = 1024
            rec = torch.zeros(lib.lbk_recurrence_record_floats(C.byref(rd), rr), device="cuda")
            conv, ring = torch.randn(TAPS, width, device="cuda"), bf16(1, TAPS, width)
            a, al, dt, be, dec = torch.randn(n, nh * 128, device="cuda"), torch.zeros(nh, device="cuda"), torch.zeros(nh * 128, device="cuda"), torch.zeros(n, nh, device="cuda"), torch.full((nh,), 0.9, device="cuda")
            us = graph_us(torch, [lambda: chk(lib.lbk_recurrence(h, 0, C.byref(rd), x.data_ptr(), width, n, 0, pos0.data_ptr(), None, cap, dec.data_ptr(), conv.data_ptr(), ring.data_ptr(), a.data_ptr(),
                                                                 al.data_ptr(), dt.data_ptr(), be.data_ptr(), state.data_ptr(), rec.data_ptr(), rr, o.data_ptr(), st()))] * 5)
            add("prompt recurrence", f"{'delta rule' if delta else 'lightning'}, {n} rows, {nh} heads of 128 x 128", "Dugulorn", us, n * width * 2 + n * nh * 128 * (8 if delta else 4),
                f32=n * nh * 128.0 * 128 * (7 if delta else 5))
        g = bf16(n, nh * 128)
        for group in (nh * 128, 128):
            os_ = [torch.randn(n, nh * 128, device="cuda") for _ in range(6)]
            w = torch.ones(group, device="cuda")
            us = graph_us(torch, [(lambda o=o: chk(lib.lbk_gated_norm(h, 0, o.data_ptr(), n, nh * 128, group, w.data_ptr(), g.data_ptr(), nh * 128, 1e-6, out.data_ptr(), nh * 128, st()))) for o in os_] * 4)
            add("norm", f"gated, {n} x {nh * 128}, groups of {group}", "Dugulorn", us, n * nh * 128 * 8)
    for n, W in ((2048, 2560), (2048, 4096)):
        sets = [(torch.randn(n, W, device="cuda"), torch.randn(n, W, device="cuda")) for _ in range(6)]
        w, o = torch.ones(W, device="cuda"), bf16(n, W)
        for family, fn, wn, nb in (("Dugulorn", lib.lbk_sandwich_rms_norm, None, 14), ("Pefolix", lib.lbk_sandwich_norm, w.data_ptr(), 14)):
            calls = [(lambda x=x, y=y: chk(fn(h, x.data_ptr(), y.data_ptr(), w.data_ptr(), wn, n, W, 1e-6, None, o.data_ptr(), W, st()))) for x, y in sets]
            add("norm", f"{n} x {W}", family, graph_us(torch, calls * 4), n * W * nb)
    ctx.check_device_error()
    return rows


def run(args, sampler_cls):
    import torch
    from lemonade_burn_b200 import dugulorn, pefolix, ternary
    torch.cuda.set_device(0)
    path = Path(__file__).resolve().parent / "MEASURED_PEAKS.json"  # a copy and a cuBLAS product on this pool's GPUs
    peaks = json.loads(path.read_text()) if path.exists() else {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}
    ctx = ternary.Context(0)
    sampler = sampler_cls(0)
    sampler.start()
    out = {"workload": "dugulorn", "data": "synthetic", "dtype": "bf16", "context": CONTEXT, "hbm_gbs": peaks["hbm_gbs"], "bf16_tflops": peaks["bf16_tflops"],
           "f32_tflops_nominal": round(F32_TFLOPS, 1), "models": {}, "kernels": []}
    parts = set(args.parts.split(","))
    if "kernels" in parts:
        out["kernels"] = kernels(torch, ctx, peaks)
    if "models" in parts:
        class Shapes:  # the low ranks of a real model
            tensor_shapes = staticmethod(lambda cfg: dugulorn.tensor_shapes(cfg, LOW))
            bf16_bits = staticmethod(dugulorn.bf16_bits)
        for name in MODELS:
            for kind in MIXERS:
                cfg = config(dugulorn, name, kind)
                with tempfile.TemporaryDirectory() as d:
                    dugulorn.save_checkpoint(d, cfg, fast_checkpoint(Shapes, cfg, 3))
                    net = dugulorn.NativeDugulorn(d, ctx)
                r = time_model(torch, net, cfg["vocab"])
                for b in (1, 16):
                    r[f"decode_batch{b}"]["fraction_of_hbm"] = round(step_bytes(cfg, dugulorn, b) / peaks["hbm_gbs"] / 1e6 / r[f"decode_batch{b}"]["ms"], 3)
                r["layers"] = len(cfg["layers"])
                out["models"][f"Dugulorn {name}, {kind}"] = r
                net.close()
            W, H, G, D, F, L, V = PEFOLIX[name]
            cfg = pefolix.make_config(V, W, [pefolix.attention_layer(H, G, D, D, None, 0, None, pefolix.dense_mlp(F))] * L)
            with tempfile.TemporaryDirectory() as d:
                pefolix.save_checkpoint(d, cfg, fast_checkpoint(pefolix, cfg, 3))
                net = pefolix.NativePefolix(d, ctx)
            r = time_model(torch, net, V)
            for b in (1, 16):
                nb = L * (2 * W * D * (2 * H + 2 * G) + 6 * W * F) + 2 * V * W + L * b * CONTEXT * G * D * 4
                r[f"decode_batch{b}"]["fraction_of_hbm"] = round(nb / peaks["hbm_gbs"] / 1e6 / r[f"decode_batch{b}"]["ms"], 3)
            r["layers"] = L
            out["models"]["Pefolix " + name] = r
            net.close()
    out["clocks"] = sampler.stop()
    print(json.dumps(out))
    return 0
