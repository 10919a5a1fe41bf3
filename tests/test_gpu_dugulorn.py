"""The Dugulorn family through the runtime (lbk_model_*, lbk_batcher_*) against the plain oracle: whole prompts, token by
token, portions of any size, several sequences in one cache, slots that are used again, long decoding, greedy generation
through the batcher. Small configurations of their own with every size different from every other, and one whose sizes
are all equal or 1."""
import json

import numpy as np
import pytest

pytestmark = pytest.mark.gpu


def configs():
    from lemonade_burn_b200 import dugulorn as p
    lat, lin, dlt = p.latent_layer, p.lightning_layer, p.delta_layer
    return {
        # every mixer with and without a feed-forward, latents read by later layers, sizes that are multiples of nothing
        "mixed": p.make_config(203, 104, [
            dlt(6, 3, 24, 20, 4, 72),
            lat(6, 24, 10, 40, 72, 56, 0.5, 5000.0, p.yarn(3.0, 64, 8.0, 1.0), None, 96),
            lin(3, 18, 44, [0.2, 0.95, 0.9995], None),
            lat(5, 40, 10, 17, 33, 56, 0.4, 300.0, None, 1, None),
            lat(3, 33, 22, 24, 40, 70, 0.45, 50.0, None, None, 40),
            dlt(2, 1, 40, 33, 3, None),
            lat(2, 16, 22, 48, 24, 70, 0.5, 50.0, p.yarn(8.0, 20, 4.0, 0.5), 4, 88),
            lat(4, 20, 10, 16, 48, 56, 0.6, 5000.0, None, 1, None)], eps=3e-4),
        # wide enough for every kernel's tiles, more than 16 heads, several 64-position chunks
        "wide": p.make_config(520, 320, [
            lin(4, 128, 64, [0.4, 0.9, 0.99, 1.0], 448),
            lat(20, 128, 64, 128, 200, 256, 0.3, 1e4, p.yarn(4.0, 64), None, 200),
            dlt(4, 2, 128, 96, 4, None),
            lat(17, 32, 64, 64, 100, 256, 0.25, 1e4, p.yarn(4.0, 64), 1, 128)], eps=1e-5),
        # one head, one tap, no decay, everything the same size, and a width of no whole unit
        "ones": p.make_config(65, 66, [lat(1, 16, 16, 16, 16, 16, 1.0, 100.0, None, None, 16), dlt(1, 1, 16, 16, 1, None), lin(1, 16, 16, [1.0], 18)], eps=1e-6),
        # value heads and keys that the prompt attention on tcgen05 does not take
        "tall": p.make_config(90, 48, [lat(2, 200, 8, 160, 30, 130, 0.2, 1e3, None, None, 24), lin(2, 200, 24, [0.5, 0.97], None), dlt(2, 2, 16, 150, 6, 20)], eps=1e-5),
    }


NAMES = ["mixed", "wide", "ones", "tall"]
TOL = {"float32": 3e-5, "bfloat16": 6e-2}


@pytest.fixture(scope="module")
def nets(ctx, tmp_path_factory):
    """name -> (config, float64 weights, {dtype: model}), loaded once."""
    from lemonade_burn_b200 import dugulorn, runtime
    from oracle import pefolix_oracle as po
    out = {}
    for i, (name, cfg) in enumerate(configs().items()):
        d = tmp_path_factory.mktemp(name)
        dugulorn.save_checkpoint(d, cfg, dugulorn.random_checkpoint(cfg, 60 + i, low_rank=7 + 10 * i))
        _, w = po.load(d)
        out[name] = (cfg, w, {t: runtime.load_model(d, ctx, t) for t in TOL})
    return out


def tokens(seed, n, vocab):
    return np.random.default_rng(seed).integers(0, vocab, size=n).astype(np.uint32)


def close(got, want, dtype):
    """Root mean square over the vocabulary (mean taken off), against the spread of the logits."""
    d = np.asarray(got, dtype=np.float64) - want
    d -= d.mean(-1, keepdims=True)
    err = np.atleast_1d(np.sqrt((d * d).mean(-1)) / want.std(-1))
    if dtype == "bfloat16":
        # a head whose read-out is nearly zero is scaled up by its norm, rounding and all, and a sharp row may turn: a
        # numpy model with the same roundings has the same rows. All but a tenth of the rows (a quarter of a few) have to
        # be close; the 32-bit runs of the same tests have no such allowance.
        spare = len(err) // (10 if len(err) > 40 else 4)
        assert np.sort(err)[len(err) - 1 - spare] < TOL[dtype] and err.max() < 0.4, (int(err.argmax()), np.sort(err)[-5:])
    else:
        assert err.max() < TOL[dtype], (int(err.argmax()), float(err.max()))


_memo = {}


def logits(nets, name, toks):
    from oracle import dugulorn_oracle as do
    key = (name, toks.tobytes())
    if key not in _memo:
        cfg, w, _ = nets[name]
        _memo[key] = do.forward(cfg, w, toks)
    return _memo[key]


@pytest.mark.parametrize("dtype", list(TOL))
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompts(nets, name, dtype):
    cfg, _, models = nets[name]
    net = models[dtype]
    assert net.architecture == "Dugulorn" and net.cfg.vocab_size == cfg["vocab"] and net.cfg.hidden_size == cfg["width"]
    want = logits(nets, name, tokens(7, 260, cfg["vocab"]))
    for n in (1, 2, 5, 8, 31, 32, 33, 129, 260):
        got = net.forward(tokens(7, 260, cfg["vocab"])[:n], net.new_cache(1, 300), all_logits=True)
        close(got, want[:n], dtype)     # a decoder: the front of a sequence does not know its rest
    net.ctx.check_device_error()


@pytest.mark.parametrize("dtype", list(TOL))
@pytest.mark.parametrize("name", NAMES)
def test_token_by_token_and_long_decoding(nets, name, dtype):
    """The recorded decode step from position 0 to 260, and the same tokens as a prompt of 200 followed by single ones (the
    step is recorded in between: that must not move any state)."""
    cfg, _, models = nets[name]
    net = models[dtype]
    t = tokens(7, 260, cfg["vocab"])
    want = logits(nets, name, t)
    c = net.new_cache(1, 300)
    close(np.stack([net.forward(t[i:i + 1], c) for i in range(len(t))]), want, dtype)
    net.reset_cache(c)
    got = [net.forward(t[:200], c)] + [net.forward(t[i:i + 1], c) for i in range(200, 230)]
    close(np.stack(got), want[199:230], dtype)
    c = net.new_cache(1, 300)
    got = [net.forward(t[:200], c)] + [net.forward(t[i:i + 1], c) for i in range(200, 260)]
    close(np.stack(got), want[199:], dtype)
    net.ctx.check_device_error()


@pytest.mark.parametrize("dtype", list(TOL))
@pytest.mark.parametrize("name", NAMES)
@pytest.mark.parametrize("portions", [[2] * 30, [3, 64, 1, 2, 17, 16, 100, 5, 1, 1, 40], [7, 8, 9, 31, 32, 33, 2, 128], [1, 2, 3, 4, 5, 6, 7, 8, 9, 10]])
def test_portions(nets, name, dtype, portions):
    """A prompt in portions gives each position the logits it has in one piece."""
    cfg, _, models = nets[name]
    net = models[dtype]
    n = sum(portions)
    t = tokens(7, 260, cfg["vocab"])[:n]
    c, at, got = net.new_cache(1, n), 0, []
    for k in portions:
        got.append(net.forward(t[at:at + k], c, all_logits=True))
        at += k
    close(np.concatenate(got), logits(nets, name, tokens(7, 260, cfg["vocab"]))[:n], dtype)
    net.ctx.check_device_error()


@pytest.mark.parametrize("dtype", list(TOL))
def test_passes_of_a_limited_number_of_rows(nets, dtype):
    """A prompt longer than a pass goes through in several, the last one ragged; wanted places in any order."""
    cfg, _, models = nets["mixed"]
    net = models[dtype]
    t = tokens(7, 260, cfg["vocab"])
    want = [149, 0, 64, 63, 65, 128, 2, 259]
    net.set_prefill_rows(64)
    try:
        got = net.forward_rows(t, net.new_cache(1, 260), want)
    finally:
        net.set_prefill_rows(4096)
    close(got, logits(nets, "mixed", t)[want], dtype)


@pytest.mark.parametrize("dtype", list(TOL))
def test_prompts_longer_than_a_run_of_records(nets, dtype):
    """More rows than a recurrence keeps records of at a time, and expanded keys that have to grow between passes."""
    cfg, _, models = nets["ones"]
    net = models[dtype]
    t = tokens(9, 2300, cfg["vocab"])
    c = net.new_cache(1, 2400)
    got = [net.forward_rows(t[:2100], c, [0, 1023, 1024, 2047, 2048, 2099]), net.forward_rows(t[2100:], c, [0, 199])]
    close(np.concatenate(got), logits(nets, "ones", t)[[0, 1023, 1024, 2047, 2048, 2099, 2100, 2299]], dtype)


@pytest.mark.parametrize("dtype", list(TOL))
@pytest.mark.parametrize("name", NAMES)
def test_unequal_requests_share_a_cache(nets, name, dtype):
    """Sequences of lengths 1, 37, 90 and 161 in one cache, decoded together, each as if alone; then one of them is
    given back and another request takes its place while the others go on."""
    import torch
    cfg, _, models = nets[name]
    net = models[dtype]
    V, lens, more = cfg["vocab"], [1, 37, 90, 161], 12
    seqs = [tokens(100 + i, n + 2 * more, V) for i, n in enumerate(lens)]
    c = net.new_cache(4, 220)
    at = list(lens)
    for s, n in enumerate(lens):
        close(net.forward_rows(seqs[s][:n], c, [n - 1], seq=s), logits(nets, name, seqs[s])[n - 1:n], dtype)

    def together(steps):
        got = [[] for _ in seqs]
        for _ in range(steps):
            tk = torch.tensor([int(seqs[s][at[s]]) for s in range(4)], dtype=torch.int32, device="cuda")
            lg, _ = net.decode(tk, c)
            lg = lg.cpu().numpy()
            for s in range(4):
                got[s].append(lg[s])
                at[s] += 1
        for s in range(4):
            close(np.stack(got[s]), logits(nets, name, seqs[s])[at[s] - steps:at[s]], dtype)

    together(more)
    seqs[2] = tokens(200, 55 + more, V)
    net.reset_seq(c, 2)
    close(net.forward_rows(seqs[2][:54], c, [0, 53], seq=2), logits(nets, name, seqs[2])[[0, 53]], dtype)
    close(net.forward_rows(seqs[2][54:55], c, [0], seq=2), logits(nets, name, seqs[2])[[54]], dtype)
    at[2] = 55
    together(more)
    net.ctx.check_device_error()


@pytest.mark.parametrize("dtype", list(TOL))
@pytest.mark.parametrize("b", [2, 9, 16])
def test_batches(nets, dtype, b):
    """Two, nine and sixteen sequences (different projection kernels), every position different."""
    import torch
    cfg, _, models = nets["wide"]
    net = models[dtype]
    seqs = [tokens(400 + s, 3 + 11 * s + 4, cfg["vocab"]) for s in range(b)]
    c = net.new_cache(b, 190)
    for s in range(b):
        net.forward_rows(seqs[s][:-4], c, [], seq=s)
    got = [[] for _ in range(b)]
    for i in range(4):
        lg, _ = net.decode(torch.tensor([int(q[len(q) - 4 + i]) for q in seqs], dtype=torch.int32, device="cuda"), c)
        for s, r in enumerate(lg.cpu().numpy()):
            got[s].append(r)
    close(np.concatenate([np.stack(r) for r in got]), np.concatenate([logits(nets, "wide", q)[-4:] for q in seqs]), dtype)
    net.ctx.check_device_error()


@pytest.mark.parametrize("dtype", list(TOL))
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_a_used_cache_is_as_good_as_a_new_one(nets, name, dtype):
    """The same request in a fresh cache and in one that a longer request has left, in a prompt and decoded: the same bits."""
    cfg, _, models = nets[name]
    net = models[dtype]
    t = tokens(5, 120, cfg["vocab"])

    def run(c):
        return np.concatenate([net.forward(t[:100], c, all_logits=True)] + [net.forward(t[i:i + 1], c)[None] for i in range(100, 120)])

    fresh = run(net.new_cache(1, 400))
    c = net.new_cache(1, 400)
    net.forward(tokens(6, 350, cfg["vocab"]), c)
    for i in range(3):
        net.forward(t[i:i + 1], c)
    net.reset_cache(c)
    assert np.array_equal(run(c), fresh)


def single(tmp_path, ctx, layers, edit, dtype="bfloat16", vocab=80, width=64, seed=9):
    from lemonade_burn_b200 import dugulorn, runtime
    from oracle import pefolix_oracle as po
    cfg = dugulorn.make_config(vocab, width, layers, eps=1e-6)
    t = {k: dugulorn.bf16_values(v).copy() for k, v in dugulorn.random_checkpoint(cfg, seed).items()}
    edit(t)
    dugulorn.save_checkpoint(tmp_path, cfg, {k: dugulorn.bf16_bits(v) for k, v in t.items()})
    return po.load(tmp_path) + (runtime.load_model(tmp_path, ctx, dtype),)


@pytest.mark.parametrize("shared", [False, True])
def test_one_far_token_decides(tmp_path, ctx, shared):
    """Latent attention whose queries single out one token, wherever it stands: the answer moves when that token is another
    one and not when it comes after the question; also in a layer that reads an earlier layer's latents."""
    from lemonade_burn_b200 import dugulorn
    from oracle import dugulorn_oracle as do
    layers = [dugulorn.latent_layer(2, 32, 8, 24, 40, 48, 1.0, 1e6)] * (1 + shared)
    if shared:
        layers = [layers[0], dugulorn.latent_layer(2, 32, 8, 24, 40, 48, 1.0, 1e6, None, 0)]
    last = len(layers) - 1

    def edit(t):
        t["embed"][:, 40:] = 0.0
        t["embed"][7, 40], t["embed"][9, 41] = 12.0, 12.0     # token 7 is the key, token 9 asks for it
        for i in range(len(layers)):
            p = f"l{i}.mix."
            for n in ("dq", "uq", "uk"):
                t[p + n][:] *= 0.05
            t[p + "dq"][0, 41] = 4.0                            # query latent 0: the question
            t[p + "uk"][0::32, :] = 0.0
            t[p + "uk"][0::32, 0] = 6.0                         # unrotated key dimension 0 of every head: latent 0
            if i == last:
                t[p + "uq"][0::40, 0] = 6.0
            t[f"l{i}.norm1"][:] = 0.5
            if shared and i == 0:
                t[p + "o"][:] *= 0.01                          # the second layer has to do it
        t["l0.mix.dkv"][0, :] = 0.0
        t["l0.mix.dkv"][0, 40] = 4.0                            # latent 0: the marked token

    cfg, w, net = single(tmp_path, ctx, layers, edit)
    rng = np.random.default_rng(3)
    for key_at, ask_at in ((0, 300), (30, 50), (63, 64), (64, 64 + 128), (128, 200), (5, 6), (199, 231), (100, 40)):
        toks = rng.integers(10, 80, size=max(key_at, ask_at) + 1).astype(np.uint32)
        toks[key_at], toks[ask_at] = 7, 9
        want = do.forward(cfg, w, toks)[ask_at]
        other = toks.copy()
        other[key_at] = 33
        moved = np.abs(do.forward(cfg, w, other)[ask_at] - want).max() / want.std()
        assert moved > 0.3 if key_at < ask_at else moved < 1e-9   # the input really asks the question
        close(net.forward_rows(toks, net.new_cache(1, 310), [ask_at])[0], want, "bfloat16")
        c = net.new_cache(1, 310)
        net.forward(toks[:ask_at], c)
        close(net.forward(toks[ask_at:ask_at + 1], c), want, "bfloat16")


@pytest.mark.parametrize("dtype", list(TOL))
def test_states_remember_the_first_token(tmp_path, ctx, dtype):
    """Recurrences that forget little: 300 tokens later the first token still shows in the logits, in prompts, portions
    and decoding."""
    from lemonade_burn_b200 import dugulorn
    from oracle import dugulorn_oracle as do

    def edit(t):
        t["l0.mix.A_log"][:] = -9.0
        t["l0.mix.b"][:, :] = 0.0
        t["embed"][7] *= 30.0

    cfg, w, net = single(tmp_path, ctx, [dugulorn.delta_layer(2, 1, 48, 32, 4, None), dugulorn.lightning_layer(2, 24, 32, [0.999, 1.0], None)], edit, dtype)
    toks = np.random.default_rng(3).integers(10, 80, size=301).astype(np.uint32)
    other = toks.copy()
    toks[0], other[0] = 7, 33
    want = do.forward(cfg, w, toks)
    assert np.abs(do.forward(cfg, w, other)[-1] - want[-1]).max() / want[-1].std() > 0.2
    close(net.forward(toks, net.new_cache(1, 310), all_logits=True), want, dtype)
    c = net.new_cache(1, 310)
    net.forward(toks[:1], c)
    net.forward(toks[1:150], c)
    got = [net.forward(toks[150:290], c)] + [net.forward(toks[i:i + 1], c) for i in range(290, 301)]
    close(np.stack(got), want[289:], dtype)


@pytest.mark.parametrize("name", NAMES)
def test_greedy_generation(nets, name):
    """generate() (batcher, prompt passes, recorded steps): in 32-bit the tokens are the oracle's greedy ones; in bf16
    they do not depend on who shares the batch. More requests than slots, so slots are used again."""
    from lemonade_burn_b200.generate import generate
    from oracle import dugulorn_oracle as do
    cfg, w, models = nets[name]
    prompts = [tokens(300 + i, n, cfg["vocab"]) for i, n in enumerate((1, 9, 40, 3, 70))]
    new = 10
    got = generate(models["float32"], prompts, new, slots=2)
    for p, g in zip(prompts, got):
        assert len(g) == new
        lg = do.forward(cfg, w, np.concatenate([p, np.array(g[:-1], dtype=np.uint32)]))[len(p) - 1:]
        top = np.sort(lg, -1)
        clear = top[:, -1] - top[:, -2] > 1e-3 * lg.std(-1)
        assert clear.mean() > 0.7 and (lg.argmax(-1)[clear] == np.array(g)[clear]).all()
    together = generate(models["bfloat16"], prompts, new, slots=3)
    alone = [generate(models["bfloat16"], [p], new, slots=3, capacity=90)[0] for p in prompts]
    same = [a == b for a, b in zip(together, alone)]
    assert sum(same) >= len(same) - 1, (together, alone)   # another kernel at another batch size may turn one near-tie


def test_trace_replay(nets, tmp_path):
    """The replay program's loop: logits of the wanted places per step, caches taken over by later requests."""
    from lemonade_burn_b200 import trace
    cfg, _, models = nets["mixed"]
    net = models["float32"]
    a, b = tokens(1, 50, cfg["vocab"]), tokens(2, 33, cfg["vocab"])
    steps = [("a", a[:20], [0, 19], []), ("a", a[20:22], [], []), ("a", a[22:23], [0], []), ("a", a[23:], [26, 3], ["a"]),
             ("b", b[:2], [1], []), ("b", b[2:], [30], ["b"])]
    lines = [json.dumps({"step": i, "entries": [{"id": r, "tokens": [int(x) for x in t], "want": w}], "end": e}) for i, (r, t, w, e) in enumerate(steps)]
    done = []
    trace.replay(net, lines, tmp_path, 64, done.append)
    assert done == list(range(len(steps))) and not (tmp_path / "1.f32").exists()
    la, lb = logits(nets, "mixed", a), logits(nets, "mixed", b)
    for i, want in ((0, la[[0, 19]]), (2, la[[22]]), (3, la[[49, 26]]), (4, lb[[1]]), (5, lb[[32]])):
        close(np.fromfile(tmp_path / f"{i}.f32", dtype="<f4").reshape(-1, cfg["vocab"]), want, "float32")


def test_loader_errors(ctx, tmp_path):
    """Missing tensors, wrong shapes, unknown mixers and feed-forwards, inconsistent sizes, sources and rotations: errors
    with a message, never a crash; refused calls leave the model usable."""
    from lemonade_burn_b200 import _lib, dugulorn as p, runtime
    cfg = p.make_config(40, 32, [p.latent_layer(2, 16, 4, 16, 24, 20, 0.25, 100.0, None, None, 24), p.lightning_layer(2, 8, 8, [0.5, 0.9]),
                                 p.delta_layer(2, 1, 8, 8, 3), p.latent_layer(2, 16, 4, 16, 24, 20, 0.25, 100.0, None, 0)])
    t = p.random_checkpoint(cfg, 1)

    def load(c, tensors, dtype="bfloat16"):
        p.save_checkpoint(tmp_path, c, tensors)
        return runtime.NativeModel(tmp_path, ctx, dtype)

    net = load(cfg, t)
    c = net.new_cache(1, 8)
    with pytest.raises(_lib.LbkError, match="do not fit"):
        net.forward(np.zeros(9, np.uint32), c)
    with pytest.raises(_lib.LbkError, match="outside the vocabulary"):
        net.forward(np.array([40], np.uint32), c)
    assert net.forward(np.zeros(8, np.uint32), c).shape == (40,)
    for missing in ("l0.mix.dkv", "l0.mix.dq.norm", "l1.mix.g", "l2.mix.A_log", "l2.mix.v.conv", "l0.mlp.up.b", "embed.norm"):
        with pytest.raises(_lib.LbkError, match=missing + " is missing"):
            load(cfg, {k: v for k, v in t.items() if k != missing})
    with pytest.raises(_lib.LbkError, match="l3.mix.uk has dtype"):
        load(cfg, {**t, "l3.mix.uk": t["l3.mix.uk"][:8]})
    mixer = lambda i, **kw: lambda l: l[i]["mixer"].update(kw)
    for edit, text in ((lambda l: l[1].update(type="other"), "unknown mixer"), (lambda l: l[0]["mlp"].update(kind="other"), "unknown feed-forward"),
                       (lambda l: l[0]["mixer"].pop("vdim"), "vdim"), (mixer(1, decay=[0.5]), "decay"), (mixer(2, kv_heads=3), "kv_heads"), (mixer(2, conv=4), "conv"),
                       (mixer(3, kv_from=3), "earlier layer"), (mixer(3, kv_from=1), "latent of the same sizes"), (mixer(3, kv_rank=21), "latent of the same sizes"),
                       (lambda l: l[0]["mixer"]["rot"].update(dims=6), "mixer.rot"), (lambda l: l[0]["mixer"]["rot"].update(scaling={"factor": 2.0}), "scaling")):
        bad = json.loads(json.dumps(cfg))
        edit(bad["layers"])
        with pytest.raises(_lib.LbkError, match=text):
            load(bad, t)
    with pytest.raises(_lib.LbkError, match="not sharded"):
        load(cfg, t)
        _lib.check(ctx._lib.lbk_model_load_shard(ctx.handle, str(tmp_path).encode(), 0, 2, _lib.ptr_array([0])[0]))
