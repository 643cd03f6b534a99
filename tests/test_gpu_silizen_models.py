"""Whole Silizen models on the GPU engine against the plain oracle of tests/silizen_oracle.py, under every way of feeding them: whole
prompts, portions down to two tokens, decoding, mixed batches, pages and slots used again, loops, generation."""
import copy
import random

import pytest
import torch

import silizen_oracle as O

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module", autouse=True)
def _one_thread():
    """The oracle is thousands of small products: threads would only wait for one another."""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)

F32_TOL, BF16_TOL = 2e-4, 0.1
PAGE = 32
FIRST = 8


def _wkv(heads=3, dim=20):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}}


def _parallel(heads=6, kv_heads=3, dim=24, vdim=40, rot=16, base=10000.0, scale=0.3, softcap=12.0, scaling=(4.0, 1.0, 4.0, 128), rheads=2, rdim=28, rvdim=16,
              tau=9.0, scales=(0.8, 1.1), rank=7):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": softcap, "rot": {"base": base, "dims": rot}}
    if scaling:
        left["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"type": "parallel", "mixer": {"left": left, "right": {"heads": rheads, "dim": rdim, "vdim": rvdim, "tau": tau, "rank": rank},
                                          "left_scale": scales[0], "right_scale": scales[1]}}


def _parallel_2(heads=4, kv_heads=2, dim=32, vdim=32, window=40, scale=0.4, rheads=4, rkv=2, rdim=20, rvdim=24, conv=3, rank=6):
    return {"type": "parallel_2", "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": window}},
        "right": {"heads": rheads, "kv_heads": rkv, "dim": rdim, "vdim": rvdim, "conv": conv, "rank": rank}}}


def _ff(layer, ff):
    return dict(layer, mlp={"kind": "dense", "ff": ff} if ff else None)


def _model(layers, loop=None, width=88, vocab=277, eps=1e-5, logit_scale=0.7):
    c = {"architecture": "Silizen", "width": width, "vocab": vocab, "norm": {"eps": eps}, "logit_scale": logit_scale, "layers": layers}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


def _cfg_a():
    """Sizes unlike powers of two and layers of every kind, three of them run three times: a layer without a feed-forward in
    the loop, head sizes that differ between q / k and v, one key/value head per query head in one layer, all heads on one in another."""
    return _model([_ff(_wkv(), 120), _ff(_parallel(), 96), _ff(_parallel_2(), 0), _ff(_wkv(2, 16), 40),
                   _ff(_parallel_2(3, 1, 16, 24, window=70, rheads=3, rkv=3, rdim=32, rvdim=8, conv=4), 64),
                   _ff(_parallel(4, 4, 16, 16, 4, scaling=None, softcap=5.0, rheads=1, rdim=8, rvdim=36, tau=16.0, scales=(1.3, -0.6)), 0)], loop=(1, 4, 3))


@pytest.fixture(scope="module")
def model_a(tmp_path_factory):
    from dllama_b200.models.layered import write_random_model
    d = str(tmp_path_factory.mktemp("silizen") / "a")
    cfg = _cfg_a()
    tensors = write_random_model(d, cfg, seed=3)
    g = torch.Generator().manual_seed(4)
    reqs = [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in (170, 70, 5, 33)]
    want = [O.model_logits(tensors, cfg, r) for r in reqs]
    return d, cfg, tensors, reqs, want


def _engine(path, dtype="float32", max_rows=256, n_slots=4, seq=256, n_pages=None, **kw):
    from dllama_b200.models import registry
    return registry.engine_for_dir(path, max_rows=max_rows, n_slots=n_slots, max_seq_len=seq, n_pages=n_pages, dtype=dtype, **kw)


def _replay(eng, reqs, steps):
    fed, slot, got = {}, {}, {i: [] for i in range(len(reqs))}
    for step in steps:
        toks, pos, slots, owner = [], [], [], []
        for i, n in step:
            if i not in slot:
                slot[i], fed[i] = eng.alloc_slot(), 0
            toks += reqs[i][fed[i]:fed[i] + n]
            pos += list(range(fed[i], fed[i] + n))
            slots += [slot[i]] * n
            owner += [i] * n
            fed[i] += n
        lg = eng.forward(toks, pos, slots).cpu()
        for r, i in enumerate(owner):
            got[i].append(lg[r])
        for i, _ in step:
            if fed[i] == len(reqs[i]) and i in slot:
                eng.free_slot(slot.pop(i))
    return {i: torch.stack(v) for i, v in got.items() if v}


def _close(got, want, tol, what=""):
    """Every row within tol.  A bf16 run against the exact oracle (tol >= BF16_TOL): a quarter of it in the median, a few rows may lie
    outside, and the first FIRST rows are left out -- a recurrence's head holds next to nothing there, o = (q . k) v for the very first
    token, and the norm per head turns that into +- v / rms(v): where q . k is near zero the rounding of q and k decides the sign.
    Those rows are held row by row to the other bf16 runs, and to the oracle in f32."""
    err = O.logit_error(got, want[:got.shape[0]])
    if tol >= BF16_TOL:
        assert bool(torch.isfinite(err).all()), what
        err = err[FIRST:]
        if len(err):
            over = int((err > tol).sum())
            assert float(err.median()) < tol / 4 and over <= max(1, len(err) // 30), f"{what}: median {float(err.median()):.3e}, {over} of {len(err)} rows over {tol}"
        return
    assert float(err.max()) < tol, f"{what}: worst row {int(err.argmax())} error {float(err.max()):.3e}"


def _whole(reqs):
    return [[(i, len(r))] for i, r in enumerate(reqs)]


DTYPES = [("float32", F32_TOL, 1e-4), ("bfloat16", BF16_TOL, 0.04)]


@pytest.mark.parametrize("dtype,tol,same", DTYPES)
def test_whole_prompts_match_the_oracle(model_a, dtype, tol, same):
    path, cfg, tensors, reqs, want = model_a
    eng = _engine(path, dtype)
    assert len(eng.layers) == 6 + 2 * 3
    first, again = eng.layers[1].mixer, eng.layers[4].mixer
    assert again.right.w_in is first.right.w_in and again.right.state is not first.right.state and again.left.cache is not first.left.cache
    assert eng.layers[6].mixer.shift_state is not eng.layers[3].mixer.shift_state and eng.layers[5].mixer.right.conv_state is not eng.layers[2].mixer.right.conv_state
    if dtype == "bfloat16":          # the tile kernels and the operand images are the ones that run
        assert first.left.tc_talk and eng.layers[2].mixer.left.tc_talk and eng.tc and eng.image("h", 64) is not None
    got = _replay(eng, reqs, _whole(reqs))
    assert eng.gated_chunks == 0 and eng._gated_scratch is not None
    for i in got:
        _close(got[i], want[i], tol, f"request {i}")


def test_residual_stream_after_every_layer(model_a):
    path, cfg, tensors, reqs, want = model_a
    eng = _engine(path)
    for i in (0, 3):                 # a prompt in chunks, a short one
        res = []
        O.model_logits(tensors, cfg, reqs[i], residual_out=res)
        eng.layer_probe = []
        s = eng.alloc_slot()
        lg = eng.forward(reqs[i], list(range(len(reqs[i]))), [s] * len(reqs[i])).cpu()
        assert len(eng.layer_probe) == len(res) == 12
        for k, (a, b) in enumerate(zip(eng.layer_probe, res)):
            err = ((a.double().cpu() - b).abs().amax(1) / b.abs().amax(1)).max()
            assert float(err) < 3e-4, f"after layer run {k}: {float(err)}"
        _close(lg, want[i], F32_TOL, "probed run")
        eng.free_slot(s)


@pytest.mark.parametrize("dtype,tol,same", DTYPES)
def test_prefill_then_token_by_token(model_a, dtype, tol, same):
    path, cfg, tensors, reqs, want = model_a
    eng = _engine(path, dtype)
    got = _replay(eng, reqs, [[(0, 135)]] + [[(0, 1)]] * 35 + [[(1, 1)]] * 70)          # request 1 is decoded from its first token
    _close(got[0], want[0], tol, "prompt + decoded")
    _close(got[1], want[1], tol, "decoded from the start")
    assert not eng.use_graphs or eng._graphs               # decoding replays a captured graph


@pytest.mark.parametrize("dtype,tol,same", DTYPES)
def test_portions_of_every_size(model_a, dtype, tol, same):
    path, cfg, tensors, reqs, want = model_a
    eng = _engine(path, dtype)
    whole = _replay(eng, reqs, [[(0, 170)], [(1, 70)]])
    sizes = [2, 30, 1, 31, 2, 2, 33, 3, 32, 5, 2, 27]                 # cuts before, at and after page borders
    assert sum(sizes) == 170
    for what, i, steps in (("portions", 0, [[(0, n)] for n in sizes]), ("two tokens at a time", 1, [[(1, 2)]] * 35),
                           ("a long portion after a short one", 0, [[(0, 3)], [(0, 130)], [(0, 37)]]), ("chunk borders", 0, [[(0, 64)], [(0, 65)], [(0, 41)]]),
                           ("the first token alone", 0, [[(0, 1)], [(0, 169)]]), ("the last token alone", 0, [[(0, 169)], [(0, 1)]])):
        got = _replay(eng, reqs, steps)
        _close(got[i], want[i], tol, what)
        _close(got[i], whole[i], same, what + " against whole")


@pytest.mark.parametrize("dtype,tol,same", DTYPES)
def test_mixed_batches_equal_each_request_alone(model_a, dtype, tol, same):
    path, cfg, tensors, reqs, want = model_a
    eng = _engine(path, dtype)
    steps = [[(0, 3), (2, 1)], [(0, 40), (1, 2), (2, 1)], [(1, 30), (0, 1), (2, 2)], [(0, 1), (1, 1), (2, 1), (3, 20)],
             [(3, 13), (0, 64), (1, 5)], [(0, 1), (1, 32)], [(0, 60)]]
    got = _replay(eng, reqs, steps)
    assert [got[i].shape[0] for i in range(4)] == [170, 70, 5, 33]
    whole = _replay(eng, reqs, _whole(reqs))
    for i in got:
        _close(got[i], want[i], tol, f"request {i} in mixed batches")
        _close(got[i], whole[i], same, f"request {i} in mixed batches against alone")
    # a long portion (chunk-parallel scans) beside decoding rows
    got = _replay(eng, reqs, [[(1, 20)], [(0, 150), (1, 1), (3, 2)], [(0, 1), (1, 49), (3, 31)], [(0, 19), (2, 5)]])
    for i in got:
        _close(got[i], want[i], tol, f"request {i} beside a long portion")


def test_pages_and_slots_are_reused_cleanly(model_a):
    path, cfg, tensors, reqs, want = model_a
    eng = _engine(path, max_rows=192, n_slots=1, seq=192, n_pages=6)
    for order in ([0, 2, 1, 3, 0], [3, 1]):
        for i in order:
            n = len(reqs[i])
            got = _replay(eng, reqs, [[(i, n // 2)], [(i, n - n // 2)]])
            _close(got[i], want[i], F32_TOL, f"request {i} after reuse")
    assert len(eng.pages.free_pages) == 6 and len(eng.pages.free_slots) == 1
    eng2 = _engine(path, "bfloat16", max_rows=160, n_slots=2, seq=192, n_pages=6)       # two live requests share a small pool
    got = _replay(eng2, reqs, [[(1, 20), (3, 33)], [(1, 50)], [(0, 140)], [(0, 29)], [(0, 1)], [(2, 5)]])
    for i in got:
        _close(got[i], want[i], BF16_TOL, f"request {i} in the shared pool")


def test_long_decoding_and_long_portions(model_a):
    path, cfg, tensors, reqs, want = model_a
    g = torch.Generator().manual_seed(21)
    seq = torch.randint(0, cfg["vocab"], (430,), generator=g).tolist()
    ref = O.model_logits(tensors, cfg, seq)
    for dtype, tol, same in DTYPES:
        eng = _engine(path, dtype, max_rows=512, seq=512)
        got = _replay(eng, [seq], [[(0, 6)]] + [[(0, 1)]] * 224 + [[(0, 200)]])
        _close(got[0], ref, tol, "224 decoded tokens, then a long portion")
        got2 = _replay(eng, [seq], [[(0, 300)], [(0, 130)]])
        _close(got2[0], ref, tol, "two long portions")
        _close(got[0], got2[0], same, "decoded against portions")


@pytest.mark.parametrize("kind", ["wkv", "left", "right", "delta"])
def test_a_far_token_reaches_the_end(tmp_path, kind):
    """One early token is changed; the only path to the last logits is one mixer's state or cache.  Its decays are set so that it
    keeps what it read (or the attention so that it looks back), and the last logits move in the engine as in the oracle: by
    prompt, and with the tail decoded."""
    from dllama_b200.formats.safetensors import write_safetensors
    from dllama_b200.models.layered import write_random_model
    layer = {"wkv": _wkv(2, 16), "left": _parallel(4, 2, 16, 24, 8, scales=(1.5, 0.0)), "right": _parallel(4, 2, 16, 24, 8, scales=(0.0, 1.5)),
             "delta": _parallel_2(4, 2, 16, 16, window=9, rdim=40)}[kind]
    cfg = _model([_ff(layer, 48)], width=64, vocab=97)
    d = str(tmp_path / kind)
    t = write_random_model(d, cfg, seed=5)
    if kind == "wkv":
        t["l0.mix.w0"] = torch.full_like(t["l0.mix.w0"], -8.0)
    elif kind == "left":
        t["l0.mix.left.q"] = t["l0.mix.left.q"] * 0.25
    elif kind == "right":
        t["l0.mix.right.a2.b"] = torch.full_like(t["l0.mix.right.a2.b"], 9.0)
    else:
        t["l0.mix.right.dt_bias"] = torch.full_like(t["l0.mix.right.dt_bias"], -12.0)
        t["l0.mix.right.b"] = t["l0.mix.right.b"] * 0.1
    write_safetensors(f"{d}/model.safetensors", t)
    g = torch.Generator().manual_seed(6)
    a = torch.randint(0, 97, (190,), generator=g).tolist()
    b = list(a)
    b[3] = (a[3] + 1) % 97
    eng = _engine(d)
    wa, wb = O.model_logits(t, cfg, a), O.model_logits(t, cfg, b)
    ga, gb = _replay(eng, [a], [[(0, 190)]])[0], _replay(eng, [b], [[(0, 150)]] + [[(0, 1)]] * 40)[0]
    _close(ga, wa, F32_TOL, "a")
    _close(gb, wb, F32_TOL, "b")
    moved = float((wa[-1] - wb[-1]).abs().max())
    assert torch.equal(ga[:3].argmax(1), gb[:3].argmax(1)) and moved > 1e-3
    assert float(((ga[-1] - gb[-1]).double() - (wa[-1] - wb[-1])).abs().max()) < 0.2 * moved


def test_window_edges_in_prompts_and_in_decoding(tmp_path):
    """A windowed layer alone, its recurrent branch silenced, distances nearly free: a changed token moves the logits up to the last
    position whose window holds it and not one further."""
    from dllama_b200.formats.safetensors import write_safetensors
    from dllama_b200.models.layered import write_random_model
    window = 37
    cfg = _model([_ff(_parallel_2(8, 2, 16, 16, window=window, scale=0.1), 0)], width=64, vocab=97)
    d = str(tmp_path / "w")
    t = write_random_model(d, cfg, seed=15)
    t["l0.mix.right.out"] = torch.zeros_like(t["l0.mix.right.out"])
    write_safetensors(f"{d}/model.safetensors", t)
    a = torch.randint(0, 97, (150,), generator=torch.Generator().manual_seed(16)).tolist()
    eng = _engine(d)
    for at in (0, 31, 32, 70):
        b = list(a)
        b[at] = (a[at] + 1) % 97
        for steps in ([[(0, 150)]], [[(0, at + 1)]] + [[(0, 1)]] * (149 - at), [[(0, at + 20)], [(0, 2)], [(0, 128 - at)]]):
            ga, gb = _replay(eng, [a], steps)[0], _replay(eng, [b], steps)[0]
            diff = (ga - gb).abs().amax(1)
            last = at + window - 1
            assert float(diff[last]) > 1e-5 and float(diff[last + 1:].max()) < 1e-6 and float(diff[:at].max() if at else 0.0) < 1e-6, (at, len(steps))


@pytest.mark.parametrize("loop", [None, (0, 1, 1), (0, 3, 2), (2, 3, 4), (1, 2, 3)])
def test_loops(tmp_path, loop):
    """No loop, a loop of one pass, over the whole list, over the last layer, over one layer in the middle -- prompt and decoding."""
    from dllama_b200.models.layered import write_random_model
    cfg = _model([_ff(_wkv(2, 12), 0), _ff(_parallel(2, 1, 16, 16, 16, rheads=1, rdim=12, rvdim=20), 40), _ff(_parallel_2(2, 2, 8, 24, window=17, rheads=2, rkv=1), 24)],
                 loop, width=52, vocab=83, logit_scale=1.0)
    d = str(tmp_path / "m")
    tensors = write_random_model(d, cfg, seed=8)
    toks = torch.randint(0, 83, (60,), generator=torch.Generator().manual_seed(9)).tolist()
    res = []
    want = O.model_logits(tensors, cfg, toks, res)
    for dtype, tol, same in DTYPES:
        eng = _engine(d, dtype, max_rows=64, seq=64, n_slots=2)
        assert len(eng.layers) == len(res)
        got = _replay(eng, [toks, toks], [[(0, 60)], [(1, 37)], [(1, 2)]] + [[(1, 1)]] * 21)
        _close(got[0], want, tol, f"{dtype} whole")
        _close(got[1], want, tol, f"{dtype} parts")


def test_greedy_generation_through_the_batching_loop(model_a, tmp_path):
    """The framework's own entry point: requests submitted to BatchEngine, batches formed by the C++ scheduler (prompt
    portions of 16 rows beside decoding rows), device greedy pick."""
    from dllama_b200.formats import tfile
    from dllama_b200.serving.batch_engine import BatchEngine, GenerationRequest
    from dllama_b200.text import native as T
    path, cfg, tensors, reqs, want = model_a
    tp = str(tmp_path / "t.t")
    tfile.write_synthetic_tokenizer(tp, cfg["vocab"])
    tok = T.Tokenizer(tp)
    eng = _engine(path, max_rows=32, n_slots=3, seq=128)
    be = BatchEngine(eng, tok, prefill_chunk=16)
    prompts = [reqs[1][:40], reqs[2], reqs[3][:20], reqs[0][:7], reqs[0][50:53]]
    n_new = 6
    rs = [be.submit(GenerationRequest(prompt_tokens=p, max_tokens=n_new, temperature=0.0)) for p in prompts]
    be.start()
    for r in rs:
        r.result(timeout=120)
    be.stop()
    assert be.n_errors == 0
    for r, p in zip(rs, prompts):
        seq = list(p)
        for _ in range(len(r.tokens)):
            seq.append(int(O.model_logits(tensors, cfg, seq)[-1].argmax()))
        assert r.tokens == seq[len(p):], (p, r.tokens, seq[len(p):])
        assert len(r.tokens) == n_new or tok.is_eos(r.tokens[-1])
    assert be.sched.stats()["free_slots"] == 3


def test_the_command_line_serves_the_model_directory(model_a):
    from dllama_b200.cli.app import build_engine
    from dllama_b200.ops import quant
    path, cfg, tensors, reqs, want = model_a
    eng = build_engine(path, 0, 1, 64, 2, 128, quant.F32, "cuda", dtype="float32")
    assert type(eng).__name__ == "LayerListEngine" and eng.h.vocab_size == cfg["vocab"] and eng.cfg.residual == "parallel"
    s = eng.alloc_slot()
    lg = eng.prefill(s, reqs[2])
    _close(lg.cpu(), want[2][-1:], F32_TOL, "prefill() of the engine surface")


# ---------------------------------------------------------------------------------------------------------------------
# random configurations: sizes, layer lists, loops and schedules drawn from a seed
# ---------------------------------------------------------------------------------------------------------------------
def _random_config(rng):
    layers = []
    for _ in range(rng.randint(1, 4)):
        r = rng.random()
        G, rep = rng.choice([1, 2, 3, 4, 5]), rng.choice([1, 2, 3, 5, 8])
        dim = rng.choice([16, 24, 36, 64, 128])
        if r < 0.3:
            l = _wkv(rng.choice([1, 2, 3, 5]), rng.choice([8, 17, 32, 64, 128]))
        elif r < 0.65:
            l = _parallel(G * rep, G, dim, rng.choice([dim, dim, 8, 20, 40, 128]), rng.choice([dim, dim // 2, 4, 8]), rng.choice([100.0, 10000.0, 500000.0]),
                          rng.choice([0.05, 0.2, 1.0]), rng.choice([3.0, 20.0, 50.0]), rng.choice([None, (8.0, 1.0, 4.0, 64), (2.0, 1.0, 32.0, 1024)]),
                          rng.choice([1, 2, 4]), rng.choice([8, 28, 32, 64]), rng.choice([8, 16, 40, 128]), rng.choice([1.0, 16.0]), (rng.uniform(0.3, 1.5), rng.uniform(0.3, 1.5)),
                          rng.choice([1, 5, 16]))
        else:
            rkv = rng.choice([1, 2, 3])
            l = _parallel_2(G * rep, G, dim, rng.choice([dim, dim, 8, 20, 40, 128]), rng.choice([1, 2, 31, 32, 33, 64, 500]), rng.choice([0.05, 0.2, 1.0]),
                            rkv * rng.choice([1, 2, 4]), rkv, rng.choice([8, 28, 32, 64, 100]), rng.choice([8, 16, 40, 128]), rng.choice([1, 2, 4, 7]), rng.choice([1, 6, 16]))
        layers.append(_ff(copy.deepcopy(l), rng.choice([0, 24, 100, 128, 256])))
    loop = None
    if rng.random() < 0.6:
        start = rng.randrange(len(layers))
        loop = (start, rng.randint(start + 1, len(layers)), rng.randint(1, 3))
    return _model(layers, loop, rng.choice([64, 90, 100, 136, 192]), rng.choice([97, 300, 513]), rng.choice([1e-5, 1e-6, 1e-3]), rng.choice([1.0, 0.25, 3.0]))


def _random_schedule(rng, lens):
    left, steps, live, pending = list(lens), [], [], list(range(len(lens)))
    while pending or live:
        while pending and len(live) < 3 and (not live or rng.random() < 0.7):
            live.append(pending.pop(0))
        step = []
        for i in list(live):
            if rng.random() < 0.2 and len(live) > 1:
                continue                                                # a request sits a step out
            n = min(left[i], rng.choice([1, 1, 1, 2, 3, 17, 32, 33, 64, 90, 150]))
            step.append((i, n))
            left[i] -= n
            if left[i] == 0:
                live.remove(i)
        if step:
            steps.append(step)
    return steps


@pytest.mark.parametrize("seed", range(10))
def test_random_configurations_and_schedules(tmp_path, seed):
    from dllama_b200.models.layered import write_random_model
    rng = random.Random(seed)
    cfg = _random_config(rng)
    tensors = write_random_model(str(tmp_path / "m"), cfg, seed=seed)
    g = torch.Generator().manual_seed(seed)
    lens = [rng.choice([1, 5, 40, 70, 130, 160]) for _ in range(4)]
    reqs = [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in lens]
    want = [O.model_logits(tensors, cfg, r) for r in reqs]
    n_pages = 3 * (max(lens) + 64) // PAGE
    for dtype, tol in (("float32", F32_TOL), ("bfloat16", BF16_TOL)):
        eng = _engine(str(tmp_path / "m"), dtype, max_rows=n_pages * PAGE, n_slots=3, seq=n_pages * PAGE, n_pages=n_pages)
        got = _replay(eng, reqs, _random_schedule(random.Random(seed + 100), lens))
        for i in got:
            assert got[i].shape[0] == lens[i]
            _close(got[i], want[i], tol, f"seed {seed}, {dtype}, request {i}: {cfg['layers']}, loop {cfg.get('loop')}")
        assert len(eng.pages.free_pages) == n_pages and len(eng.pages.free_slots) == 3
        eng.close()
