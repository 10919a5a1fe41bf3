"""`python bench.py --workload pefolix`: prompt passes and decode steps of the Pefolix family at sizes that resemble a
real model's layers (random weights), beside BitNet at equal size, and the kernels of both one by one against their
rooflines. One JSON line, one GPU.

Models are timed through the runtime's own calls: lbk_model_decode (the recorded step, CUDA events on the launching
stream) and lbk_model_forward (a prompt pass, wall clock of the synchronous call). Every model's weights exceed L2, so
a decode step streams them from HBM. Kernels are timed as CUDA-graph replays of calls that rotate over enough copies of
their operands to exceed L2.
"""
from __future__ import annotations

import json
import tempfile
import time
from pathlib import Path

import numpy as np

CONTEXT, PROMPT = 4096, 2048
# name: width, heads, kv heads, head size, feed-forward, layers, vocabulary, window, kept tokens, experts (None: dense)
MODELS = {
    "2560 wide, dense, full context": (2560, 20, 5, 128, 6912, 8, 32000, None, 0, None),
    "2560 wide, dense, window 1024 + 4": (2560, 20, 5, 128, 6912, 8, 32000, 1024, 4, None),
    "4096 wide, dense, full context": (4096, 32, 8, 128, 14336, 4, 32000, None, 0, None),
    "4096 wide, 64 experts of 1408, 6 a token, shared 2816, window 4096": (4096, 32, 8, 128, 1408, 2, 32000, 4096, 4, (64, 6, 2816)),
}
BITNET = {"2560 wide": (2560, 20, 5, 6912, 8, 32000), "4096 wide": (4096, 32, 8, 14336, 4, 32000)}


def fast_checkpoint(p, cfg, seed):
    """Random bf16 bits: random sign and mantissa, one magnitude per matrix (quick at sizes where normals are not)."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in p.tensor_shapes(cfg):
        if len(shape) == 1:
            out[name] = p.bf16_bits(np.ones(shape, np.float32))
            continue
        exp = int(round(np.log2((1.0 if name == "embed" else shape[1] ** -0.5) / 1.5))) + 127
        out[name] = (rng.integers(0, 1 << 16, size=shape, dtype=np.uint16) & np.uint16(0x807F)) | np.uint16(exp << 7)
    return out


def graph_us(torch, calls, reps=3):
    """Microseconds per call of a CUDA graph of `calls` (a list of functions), replayed."""
    for c in calls[:3]:
        c()
    torch.cuda.synchronize()
    s = torch.cuda.Stream()
    with torch.cuda.stream(s):
        g = torch.cuda.CUDAGraph()
        with torch.cuda.graph(g, stream=s):
            for c in calls:
                c()
        for _ in range(3):
            g.replay()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        e0.record(s)
        for _ in range(reps):
            g.replay()
        e1.record(s)
        torch.cuda.synchronize()
    return e0.elapsed_time(e1) * 1e3 / (reps * len(calls))


def kernels(torch, ctx, peaks):
    from lemonade_burn_b200 import _lib, ops, runtime  # noqa: F401
    from lemonade_burn_b200.pack import row_bytes
    lib, chk, h = _lib.load(), _lib.check, ctx.handle
    hbm, tc16 = peaks["hbm_gbs"], peaks["bf16_tflops"]
    int8 = ctx.int8_peak_tops(192)
    st = lambda: torch.cuda.current_stream().cuda_stream
    rows = []

    def add(kind, what, family, us, nbytes=None, flops=None, peak_t=None):
        t_mem = (nbytes or 0) / hbm / 1e3                    # us at the measured copy rate
        t_mm = (flops or 0) / (peak_t or tc16) / 1e6
        rows.append({"kind": kind, "what": what, "family": family, "us": round(us, 2), "roofline_us": round(max(t_mem, t_mm), 2),
                     "bound": "HBM" if t_mem >= t_mm else "tensor", "fraction": round(max(t_mem, t_mm) / us, 3)})

    def bf16(*s):
        return torch.randn(*s, device="cuda").to(torch.bfloat16) * 0.02

    for W, F in ((2560, 6912), (4096, 14336)):
        for m in (1, 16, 64, 2048):
            for name, r, c, gated in (("gate/up", F, W, 1), ("down", W, F, 0)):
                nbytes = r * c * 2 * (2 if gated else 1)
                copies = max(2, min(24, int(300e6 / nbytes) + 1)) if m < 2048 else 2
                ws = [bf16(r * (2 if gated else 1), c) for _ in range(copies)]
                x = bf16(m, c)
                out = torch.zeros(m, r, device="cuda", dtype=torch.bfloat16 if gated else torch.float32)
                calls = [(lambda w=w: chk(lib.lbk_dense_linear(h, 0, x.data_ptr(), c, m, w.data_ptr(), c, w.shape[0], c, gated, r, 0, out.data_ptr(), r,
                                                                0 if gated else 1, None, 0, st()))) for w in ws]
                us = graph_us(torch, calls * (1 if m < 2048 else 5))
                add("projection", f"{name} {c} -> {r}{' x2' if gated else ''}, {m} tokens", "Pefolix", us, nbytes + m * c * 2 + out.numel() * out.element_size(),
                    2.0 * m * r * c * (2 if gated else 1))
                del ws
                # BitNet: the same group, packed ternary
                pk = row_bytes(c) * r
                nmat = 2 if gated else 1
                copies = max(2, min(64, int(300e6 / (pk * nmat)) + 1)) if m < 2048 else 2
                groups = []
                for _ in range(copies):
                    lins = []
                    for _ in range(nmat):
                        b = torch.randint(0, 256, (r, row_bytes(c)), dtype=torch.uint8, device="cuda")
                        lins.append(ops.TernaryLinear(b & ~((b >> 1) & b & 0x55), 60.0, c, ctx))
                    groups.append(lins)
                xf = torch.randn(m, c, device="cuda")
                if m < 9:
                    calls = [(lambda g=g: ops.ternary_linear_multi(xf, g)) for g in groups]
                else:
                    q8 = torch.randint(-127, 128, (m, row_bytes(c) * 4), dtype=torch.int8, device="cuda")
                    qs, qsum = torch.ones(m, device="cuda"), torch.zeros(m, dtype=torch.int32, device="cuda")
                    calls = [(lambda g=g: ops.ternary_gemm_q(q8, qs, qsum, m, g)) for g in groups]
                us = graph_us(torch, calls * (1 if m < 2048 else 5))
                add("projection", f"{name} {c} -> {r}{' x2' if gated else ''}, {m} tokens", "BitNet", us, pk * nmat + m * c * (4 if m < 9 else 1) + m * r * nmat * 4,
                    2.0 * m * r * c * nmat, int8)
                del groups
        torch.cuda.empty_cache()

    # attention at head size 128: one token of b sequences, and prompt rows
    for b, nh, kvh, pos in ((1, 20, 5, 4095), (16, 20, 5, 4095), (16, 32, 8, 4095)):
        cap, sets = 4160, 2 if b > 1 else 16
        kv = [(bf16(b, kvh, cap, 128), bf16(b, kvh, cap, 128)) for _ in range(sets)]
        q16, qf = bf16(b, nh, 128), torch.randn(b, nh, 128, device="cuda")
        kn, vn = torch.randn(b, kvh, 128, device="cuda"), torch.randn(b, kvh, 128, device="cuda")
        posd = torch.full((b,), pos, dtype=torch.int32, device="cuda")
        scr = torch.empty(max(int(lib.lbk_attn_window_scratch(b, nh, 128)), b * nh * 256 * 132), device="cuda")
        cnt = torch.zeros(b * kvh, dtype=torch.int32, device="cuda")
        o16, of = bf16(b, nh * 128), torch.zeros(b, nh * 128, device="cuda")
        cs, sn = torch.rand(cap, 128, device="cuda"), torch.rand(cap, 128, device="cuda")
        for win, keep in ((0, 0), (1024, 4)):
            calls = [(lambda k=k, v=v: chk(lib.lbk_attn_window(h, 0, q16.data_ptr(), k.data_ptr(), v.data_ptr(), posd.data_ptr(), b, -1, nh, kvh, 128, 128, 128,
                                                               128, cap, 0.088, win, keep, 1, scr.data_ptr(), o16.data_ptr(), nh * 128, st()))) for k, v in kv]
            seen = pos + 1 if not win else win + keep
            add("decode attention", f"{b} sequences, {nh}/{kvh} heads, {seen} keys", "Pefolix", graph_us(torch, calls * 8), b * kvh * seen * 512)
        splits = min(256, (cap + 31) // 32)
        calls = [(lambda k=k, v=v: chk(lib.lbk_attn_decode_fused_seq(h, qf.data_ptr(), kn.data_ptr(), vn.data_ptr(), cs.data_ptr(), sn.data_ptr(), posd.data_ptr(),
                                                                     b, nh, kvh, 128, cap, splits, k.data_ptr(), v.data_ptr(), scr.data_ptr(), cnt.data_ptr(),
                                                                     of.data_ptr(), st()))) for k, v in kv]
        add("decode attention", f"{b} sequences, {nh}/{kvh} heads, {pos + 1} keys", "BitNet", graph_us(torch, calls * 8), b * kvh * (pos + 1) * 512)
        del kv
    for n, nh, kvh in ((2048, 20, 5), (2048, 32, 8)):
        k, v, cap = bf16(1, kvh, n, 128), bf16(1, kvh, n, 128), n
        q16, qf = bf16(n, nh, 128), torch.randn(n, nh, 128, device="cuda")
        o16, of, posd = bf16(n, nh * 128), torch.zeros(n, nh * 128, device="cuda"), torch.zeros(1, dtype=torch.int32, device="cuda")
        for win, keep in ((0, 0), (512, 4)):
            pairs = n * (n + 1) / 2 if not win else sum(min(i + 1, win + keep) for i in range(n))
            us = graph_us(torch, [lambda: chk(lib.lbk_attn_window(h, 0, q16.data_ptr(), k.data_ptr(), v.data_ptr(), posd.data_ptr(), n, 0, nh, kvh, 128, 128, 128,
                                                                  128, cap, 0.088, win, keep, 1, None, o16.data_ptr(), nh * 128, st()))] * 10)
            add("prompt attention", f"{n} rows, {nh}/{kvh} heads, window {win or 'none'}", "Pefolix", us, flops=4.0 * nh * 128 * pairs)
        us = graph_us(torch, [lambda: chk(lib.lbk_attn_prefill(h, qf.data_ptr(), k.data_ptr(), v.data_ptr(), posd.data_ptr(), n, nh, kvh, 128, cap, 0,
                                                               of.data_ptr(), st()))] * 10)
        add("prompt attention", f"{n} rows, {nh}/{kvh} heads, window none", "BitNet", us, flops=4.0 * nh * 128 * n * (n + 1) / 2)

    # norms of a prompt pass: (x += ..., norm, operand of the projection behind it)
    for n, W in ((2048, 2560), (2048, 4096)):
        sets = [(torch.randn(n, W, device="cuda"), torch.randn(n, W, device="cuda")) for _ in range(6)]
        w = torch.ones(W, device="cuda")
        o = bf16(n, W)
        calls = [(lambda x=x, y=y: chk(lib.lbk_sandwich_norm(h, x.data_ptr(), y.data_ptr(), w.data_ptr(), w.data_ptr(), n, W, 1e-6, None, o.data_ptr(), W, st())))
                 for x, y in sets]
        add("norm", f"{n} x {W}", "Pefolix", graph_us(torch, calls * 4), n * W * 14)
        q8, qs, qsum = torch.zeros(n, W, dtype=torch.int8, device="cuda"), torch.ones(n, device="cuda"), torch.zeros(n, dtype=torch.int32, device="cuda")
        calls = [(lambda x=x, y=y: ops.norm_quant(ops.PRE_ADD_RMS, x, y, w, 1e-6, q8, qs, qsum, ctx)) for x, y in sets]
        add("norm", f"{n} x {W}", "BitNet", graph_us(torch, calls * 4), n * W * 13)

    # experts of a prompt pass, sorted tokens (no counterpart in BitNet; its prompt projection is the like kernel)
    E, top, F, W, n = 64, 6, 1408, 4096, 2048
    offs = torch.arange(0, E + 1, device="cuda", dtype=torch.int32) * (n * top // E)
    for name, r, c in (("experts' up", F, W), ("experts' down", W, F)):
        w, x = bf16(E * r, c), bf16(n * top, c)
        out = bf16(n * top, r)
        us = graph_us(torch, [lambda: chk(lib.lbk_dense_linear(h, 0, x.data_ptr(), c, n * top, w.data_ptr(), c, E * r, c, 0, r, 1, out.data_ptr(), r, 0, offs.data_ptr(),
                                                               E, st()))] * 5)
        add("projection", f"{name} {c} -> {r}, {E} experts, {n * top} rows", "Pefolix", us, E * r * c * 2 + n * top * (r + c) * 2, 2.0 * n * top * r * c)
        del w
    ctx.check_device_error()
    return rows


def time_model(torch, net, vocab, batches=(1, 16)):
    rng = np.random.default_rng(1)
    out = {}
    toks = rng.integers(0, vocab, size=PROMPT).astype(np.uint32)
    c = net.new_cache(1, PROMPT + 64)
    best = 1e9
    for i in range(5):
        net.reset_cache(c)
        torch.cuda.synchronize()
        t0 = time.perf_counter()
        net.forward(toks, c)
        if i:
            best = min(best, time.perf_counter() - t0)
    out["prompt"] = {"tokens": PROMPT, "ms": round(best * 1e3, 3), "tok_per_s": round(PROMPT / best)}
    long = rng.integers(0, vocab, size=CONTEXT - 1).astype(np.uint32)
    for b in batches:
        c = net.new_cache(b, CONTEXT + 128)
        if b == 1:
            net.forward(long, c)
        else:
            for s in range(b):
                net.forward_rows(long, c, [], seq=s)
        tk = torch.from_numpy(rng.integers(0, vocab, size=b).astype(np.int32)).cuda()
        for _ in range(4):
            net.decode(tk, c)
        e0, e1, n = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True), 40
        torch.cuda.synchronize()
        e0.record()
        for _ in range(n):
            net.decode(tk, c)
        e1.record()
        torch.cuda.synchronize()
        ms = e0.elapsed_time(e1) / n
        out[f"decode_batch{b}"] = {"position": CONTEXT, "ms": round(ms, 4), "tok_per_s": round(b / ms * 1e3)}
        net.ctx.check_device_error()
    return out


def model_bytes(width, heads, kv, dim, ff, layers, vocab, window, keep, experts, batch):
    """HBM bytes of a decode step: weights once (the experts a batch can choose), the head, visible keys and values."""
    attn = 2 * width * dim * (2 * heads + 2 * kv)
    if experts:
        E, top, shared = experts
        hit = E * (1.0 - (1.0 - top / E) ** batch)
        mlp = 4 * width * (ff * hit + shared)
    else:
        mlp = 6 * width * ff
    seen = CONTEXT if not window else min(CONTEXT, window + keep)
    return layers * (attn + mlp) + 2 * vocab * width + layers * batch * seen * kv * dim * 4


def run(args, sampler_cls):
    import torch
    from lemonade_burn_b200 import model, pefolix, ternary
    torch.cuda.set_device(0)
    path = Path(__file__).resolve().parent / "MEASURED_PEAKS.json"  # a copy and a cuBLAS product on this pool's GPUs
    peaks = json.loads(path.read_text()) if path.exists() else {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}
    ctx = ternary.Context(0)
    sampler = sampler_cls(0)
    sampler.start()
    out = {"workload": "pefolix", "data": "synthetic", "dtype": "bf16", "context": CONTEXT, "hbm_gbs": peaks["hbm_gbs"], "bf16_tflops": peaks["bf16_tflops"],
           "models": {}, "kernels": []}
    parts = set(args.parts.split(","))
    if "kernels" in parts:
        out["kernels"] = kernels(torch, ctx, peaks)
    if "models" in parts:
        for name, (W, H, G, D, F, L, V, win, keep, ex) in MODELS.items():
            mlp = pefolix.moe_mlp(ex[0], ex[1], F, ex[2]) if ex else pefolix.dense_mlp(F)
            cfg = pefolix.make_config(V, W, [pefolix.attention_layer(H, G, D, D, win, keep, None, mlp)] * L)
            with tempfile.TemporaryDirectory() as d:
                pefolix.save_checkpoint(d, cfg, fast_checkpoint(pefolix, cfg, 3))
                net = pefolix.NativePefolix(d, ctx)
            r = time_model(torch, net, V)
            for b in (1, 16):
                nb = model_bytes(W, H, G, D, F, L, V, win, keep, ex, b)
                r[f"decode_batch{b}"]["fraction_of_hbm"] = round(nb / peaks["hbm_gbs"] / 1e6 / r[f"decode_batch{b}"]["ms"], 3)
            r["layers"] = L
            out["models"]["Pefolix " + name] = r
            net.close()
        for name, (W, H, G, F, L, V) in BITNET.items():
            cfg = model.Config(W, F, H, G, L, V, 1e-5, 500000.0, CONTEXT + 128)
            with tempfile.TemporaryDirectory() as d:
                model.save_checkpoint(d, cfg, model.random_checkpoint(cfg, 3))
                net = model.NativeBitNet(d, ctx)
            r = time_model(torch, net, V)
            for b in (1, 16):
                nb = L * (W * 128 * (2 * H + 2 * G) / 4 + 3 * W * F / 4) + 2 * V * W + L * b * CONTEXT * G * 128 * 4
                r[f"decode_batch{b}"]["fraction_of_hbm"] = round(nb / peaks["hbm_gbs"] / 1e6 / r[f"decode_batch{b}"]["ms"], 3)
            r["layers"] = L
            out["models"]["BitNet " + name] = r
            net.close()
    out["clocks"] = sampler.stop()
    print(json.dumps(out))
    return 0
