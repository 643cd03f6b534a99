#!/usr/bin/env python3
"""Workloads for launch lists and counter captures of the layer-list models (one GPU).

  python scripts/profile_layered.py steps --design sunesun --size w2048
      one 2048-token prompt per slot, then decode steps of 1 and of 32 rows, launched eagerly (no CUDA graphs) so that
      every kernel shows in a launch list:
        ncu --metrics gpu__time_duration.sum --clock-control none --csv --log-file out.csv python scripts/profile_layered.py steps ...
  python scripts/profile_layered.py window-attention
      the windowed-attention tile kernel alone (2048 rows of one sequence, 16 / 8 heads of 128, 64 rotated dims, window
      1024, soft cap 50), timed with CUDA events; small enough for a full counter capture:
        ncu --set full --clock-control none -k regex:window_attention_mma -s 1 -c 2 -o out python scripts/profile_layered.py window-attention
  python scripts/profile_layered.py lightning-scan
      the chunk-parallel linear-attention scan alone (2048 rows of one sequence, 16 heads of 128 x 128), timed with CUDA
      events, then the token-by-token kernel on 32 sequences of one row:
        ncu --set full --clock-control none -k regex:lightning_chunk_out -s 1 -c 2 -o out python scripts/profile_layered.py lightning-scan
  python scripts/profile_layered.py talk-attention
      the head-mixed attention tile kernel alone (2048 rows of one sequence, 16 / 4 heads, keys and values of 128, 64
      rotated dims, the head mix folded into queries of 4 x 128), timed with CUDA events:
        ncu --set full --clock-control none -k regex:talk_attention_mma -s 1 -c 1 -o out python scripts/profile_layered.py talk-attention
  python scripts/profile_layered.py gated-scan
      the chunk-parallel scans with data-dependent gates alone (2048 rows of one sequence; matrix memory with 8 heads of
      128 x 256, HGRN2 with 16 heads of 128 x 128), then both token by token on 1 and 32 sequences of one row:
        ncu --set full --clock-control none -k regex:gated_chunk_out -s 1 -c 2 -o out python scripts/profile_layered.py gated-scan
  python scripts/profile_layered.py delta-scan
      the recurrences with keys of their own alone (2048 rows of one sequence; gated linear attention and the gated delta rule with
      16 heads of 128 x 128, time mixing with 32 heads of 64 x 64), then token by token on 1 and 32 sequences of one row:
        ncu --set full --clock-control none -k regex:delta_chunk_ -s 2 -c 2 -o out python scripts/profile_layered.py delta-scan
  python scripts/profile_layered.py biased-attention
      the attention tile kernel with values of its own (2048 rows of one sequence, 16 / 4 heads of 128, sink, head gates), soft-capped
      over all earlier positions, then with a distance bias in a window of 1024:
        ncu --set full --clock-control none -k regex:window_attention_mma -s 1 -c 1 -o out python scripts/profile_layered.py biased-attention
  python scripts/profile_layered.py selective-scan
      the selective scan alone (4096 channels of 16 state entries; 2048 rows of one sequence, then 32 sequences of one row):
        ncu --set full --clock-control none -k regex:selective_scan -s 1 -c 1 -o out python scripts/profile_layered.py selective-scan
  python scripts/profile_layered.py wide-attention
      attention whose softmax weights are mixed across heads (2048 rows of one sequence, 16 / 4 heads of 128) and the mix alone:
        ncu --set full --clock-control none -k regex:talk_attention_mma -s 1 -c 1 -o out python scripts/profile_layered.py wide-attention
Run the plain command first; capture only if it exits 0.
"""
import argparse
import math
import os
import sys

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))


def steps(a):
    os.environ["DLLAMA_LAYERS_GRAPHS"] = "0"
    import numpy as np
    import torch
    import bench
    from dllama_b200.models import registry
    from dllama_b200.models.layered import write_random_model
    T, users, vocab, nl = a.prompt, 32, 32768, a.layers
    d = os.path.join(a.model_dir, f"dllama_b200_{'layered' if a.design == 'ribivik' else a.design}_{a.size}_l{nl}")
    if not os.path.exists(os.path.join(d, "model.safetensors")):
        cfg = {"ribivik": lambda: bench.layered_config(bench.LAYERED_SIZES[a.size], nl, vocab), "sunesun": lambda: bench.sunesun_config(a.size, nl, vocab),
               "venadra": lambda: bench.venadra_config(a.size, nl, vocab), "darusun": lambda: bench.darusun_config(a.size, nl, vocab),
               "vopedra": lambda: bench.vopedra_config(a.size, nl, vocab), "silizen": lambda: bench.silizen_config(a.size, nl, vocab)}[a.design]()
        write_random_model(d, cfg, seed=1)
    torch.cuda.set_device(0)
    eng = registry.engine_for_dir(d, max_rows=T, n_slots=users, max_seq_len=T + 64, dtype="bfloat16")
    prompt = np.random.default_rng(0).integers(1, vocab, T).tolist()
    slots = [eng.alloc_slot() for _ in range(users)]
    for s in slots:
        eng.forward(prompt, list(range(T)), [s] * T, logits_from=T - 1)
    torch.cuda.synchronize()
    print("prompts done: %d forwards of %d rows" % (users, T))
    for i in range(3):
        eng.decode_step_greedy([1], [T + i], [slots[0]])
    torch.cuda.synchronize()
    print("3 decode steps of 1 row done")
    for i in range(2):
        eng.decode_step_greedy([1] * users, [T + 3 + i] + [T + i] * (users - 1), slots)
    torch.cuda.synchronize()
    print("2 decode steps of %d rows done" % users)


def window_attention(a):
    import torch
    from dllama_b200.models.layered import interpolated_rotary
    from dllama_b200.ops import layers as L
    H, G, d, rd, window, cap, n = 16, 8, 128, 64, 1024, 50.0, 2048
    f, mag = interpolated_rotary(10000.0, rd, None)
    n_pages = n // 32
    bt = torch.arange(n_pages, dtype=torch.int32).view(1, -1).cuda()
    cache = torch.zeros(n_pages, G, 32, d + rd, dtype=torch.bfloat16, device="cuda")
    g = torch.Generator().manual_seed(1)
    k, q = torch.randn(n, G * d, generator=g).cuda(), torch.randn(n, H * d, generator=g).cuda()
    pos, slot = torch.arange(n, dtype=torch.int32).cuda(), torch.zeros(n, dtype=torch.int32).cuda()
    L.window_kv_write(k, n, G, d, rd, f.cuda(), mag, pos, slot, bt, cache, q=q, q_heads=H)
    out = torch.zeros(n, H * d, device="cuda")
    rq = L.window_tc_rows(H, G)
    tiles = torch.arange(n, dtype=torch.int32).view(-1, rq).cuda()
    ev0, ev1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    for _ in range(4):
        ev0.record()
        L.window_attention_tc(q, out, H, G, d, rd, 1 / math.sqrt(d), cap, window, pos, slot, bt, cache, tiles, n // rq, rq)
        ev1.record()
        torch.cuda.synchronize()
        print("window attention: %.1f us" % (ev0.elapsed_time(ev1) * 1e3))
    keys = sum(min(i + 1, window) for i in range(n))
    print("GFLOP over the visible keys: %.2f" % (keys * H * d * 4 / 1e9))


def talk_attention(a):
    import torch
    from dllama_b200.models.layered import rotary_frequencies
    from dllama_b200.ops import layers as L
    H, G, d, dv, rd, n = 16, 4, 128, 128, 64, 2048
    n_pages = n // 32
    bt = torch.arange(n_pages, dtype=torch.int32).view(1, -1).cuda()
    cache = torch.zeros(n_pages, G, 32, d + dv, dtype=torch.bfloat16, device="cuda")
    g = torch.Generator().manual_seed(1)
    q, k, v = (torch.randn(n, w, generator=g).cuda() for w in (H * d, G * d, G * dv))
    talk = (torch.eye(H) + torch.randn(H, H, generator=g) * 0.3).cuda()
    qm = torch.zeros(n, H * G * d, device="cuda")
    pos, slot = torch.arange(n, dtype=torch.int32).cuda(), torch.zeros(n, dtype=torch.int32).cuda()
    ev0, ev1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    freqs = rotary_frequencies(500000.0, rd).cuda()
    for _ in range(3):
        ev0.record()
        L.window_kv_write(k, n, G, d, rd, freqs, 1.0, pos, slot, bt, cache, q=q, q_heads=H, v=v, vdim=dv,
                          qk_norm=True, eps=1e-5, rope_half=True, talk=talk, q_mixed=qm)
        ev1.record()
        torch.cuda.synchronize()
        print("cache writer (rotary, unit norms, head mix): %.1f us" % (ev0.elapsed_time(ev1) * 1e3))
    out = torch.zeros(n, H * dv, device="cuda")
    rq = L.talk_tc_rows(H, G, d, dv, G, n)
    tiles = torch.arange(n, dtype=torch.int32).view(-1, rq).cuda()
    for n_splits in (1, 4):
        part = torch.zeros(L.talk_tc_partial_floats(n // rq, G, n_splits, dv, rq, H), device="cuda") if n_splits > 1 else None
        for _ in range(4):
            ev0.record()
            L.talk_attention_tc(qm, out, H, G, d, dv, 0.1, 0, pos, slot, bt, cache, tiles, n // rq, rq, n_splits, part, key_heads=G)
            ev1.record()
            torch.cuda.synchronize()
            print("head-mixed attention, tiles of %d rows, %d page shares: %.1f us" % (rq, n_splits, ev0.elapsed_time(ev1) * 1e3))
    pairs = n * (n + 1) // 2
    print("FLOPs per launch (visible pairs, folded form 2 * (4 * 128 + 128) per head): %.1f G" % (pairs * H * 2 * (G * d + dv) / 1e9))


def lightning_scan(a):
    import torch
    from dllama_b200.ops import layers as L
    H, d, dv, n, users = 16, 128, 128, 2048, 32
    g = torch.Generator().manual_seed(1)
    qkv = (torch.randn(n, H * (2 * d + dv), generator=g) * 0.3).cuda()
    decay = torch.linspace(0.6, 0.999, H).cuda()
    y = torch.zeros(n, H * dv, device="cuda")
    state = torch.zeros(users, H, d, dv, device="cuda")
    scratch = torch.zeros(L.lightning_chunk_floats(n, 1, H, d, dv), device="cuda")
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    keep = [i32(list(range(n))), i32([0] * n), i32([0, n]), i32(list(range(n))), i32([0]), i32([0])]
    b = L.mamba_batch(*keep)
    ev0, ev1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    for _ in range(4):
        ev0.record()
        L.lightning_scan(b, 1, qkv, qkv[:, H * d:], qkv[:, 2 * H * d:], decay, y, state, H, d, dv, max_chunks=n // L.LIGHTNING_CHUNK, scratch=scratch)
        ev1.record()
        torch.cuda.synchronize()
        print("chunked scan, %d rows: %.1f us" % (n, ev0.elapsed_time(ev1) * 1e3))
    print("GFLOP (state update and read-out, 4 dim vdim per row and head): %.2f" % (n * H * 4 * d * dv / 1e9))
    keep2 = [i32([5] * users), i32(list(range(users))), i32(list(range(users + 1))), i32(list(range(users))), i32(list(range(users))), i32([5] * users)]
    b2 = L.mamba_batch(*keep2)
    for m in (1, users):
        for _ in range(3):
            ev0.record()
            L.lightning_scan(b2, m, qkv, qkv[:, H * d:], qkv[:, 2 * H * d:], decay, y, state, H, d, dv)
            ev1.record()
            torch.cuda.synchronize()
            print("token-by-token scan, %d sequences of one row: %.1f us for %.1f MB of state read and written" % (m, ev0.elapsed_time(ev1) * 1e3, 2 * m * H * d * dv * 4 / 1e6))


def _sequences(n_rows, n_seq):
    """Batch descriptor of n_seq sequences of n_rows consecutive rows each (fresh if a sequence has more than one row)."""
    import torch
    from dllama_b200.ops import layers as L
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    M, p0 = n_rows * n_seq, 0 if n_rows > 1 else 5
    keep = [i32([p0 + i % n_rows for i in range(M)]), i32([i // n_rows for i in range(M)]), i32([i * n_rows for i in range(n_seq + 1)]),
            i32(list(range(M))), i32(list(range(n_seq))), i32([p0] * n_seq)]
    return L.mamba_batch(*keep), keep


def _timed(what, fn, repeats=4):
    import torch
    ev0, ev1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    for _ in range(repeats):
        ev0.record()
        fn()
        ev1.record()
        torch.cuda.synchronize()
        print("%s: %.1f us" % (what, ev0.elapsed_time(ev1) * 1e3))


def gated_scan(a):
    import torch
    from dllama_b200.ops import layers as L
    n, users = 2048, 32
    g = torch.Generator().manual_seed(1)
    for name, H, d, dv in (("matrix memory", 8, 128, 256), ("HGRN2", 16, 128, 128)):
        x = torch.randn(n, H * (2 * d + dv), generator=g).cuda()
        y, den = torch.zeros(n, H * dv, device="cuda"), torch.zeros(n * H, device="cuda")
        state, n_state, u = torch.zeros(users, H, d, dv, device="cuda"), torch.zeros(users, H, d, device="cuda"), torch.zeros(users, H, device="cuda")
        z, bias = torch.randn(n, 2 * H, generator=g).cuda(), torch.full((H * d,), 2.0, device="cuda")
        keep, put, floor = (torch.zeros(n * H, device="cuda") for _ in range(3))
        slots = n // L.GATED_CHUNK + users
        scratch = torch.zeros(L.gated_chunk_floats(n, users, H, d, dv), device="cuda")

        def scan(b, n_seq, **kw):
            if name == "HGRN2":
                L.gated_scan(b, n_seq, x, x[:, 2 * H * d:], y, state, H, d, dv, q_silu=True, f=x[:, H * d:], f_bias=bias, lower=bias * 0.1, **kw)
            else:
                L.mlstm_gates(b, n_seq, z, z[:, H:], bias, bias, 15.0, u, keep, put, floor, H, n if n_seq == 1 and kw else 1)
                L.gated_scan(b, n_seq, x, x[:, 2 * H * d:], y, state, H, d, dv, q_scale=d ** -0.5, k=x[:, H * d:], log_keep=keep, put=put,
                             den=den, n_state=n_state, **kw)

        b, hold = _sequences(n, 1)
        _timed(f"{name}, chunked, {n} rows", lambda: scan(b, 1, max_chunks=n // L.GATED_CHUNK, scratch=scratch, chunk_slots=slots))
        print("GFLOP (state update and read-out, 4 dim vdim per row and head): %.2f" % (n * H * 4 * d * dv / 1e9))
        for m in (1, users):
            b1, hold1 = _sequences(1, m)
            _timed(f"{name}, token by token, {m} sequences of one row ({2 * m * H * d * dv * 4 / 1e6:.1f} MB of state)", lambda: scan(b1, m), 3)


def delta_scan(a):
    import torch
    from dllama_b200.ops import layers as L
    n, users = 2048, 32
    g = torch.Generator().manual_seed(1)
    for name, H, d, dv in (("gated linear attention", 16, 128, 128), ("time mixing", 32, 64, 64), ("gated delta rule", 16, 128, 128)):
        x = torch.randn(n, H * (3 * d + dv + 1), generator=g).cuda()
        x[:, :2 * H * d] *= d ** -0.5
        y, u, state, vec = torch.zeros(n, H * dv, device="cuda"), torch.zeros(n, H * dv, device="cuda"), torch.zeros(users, H, d, dv, device="cuda"), torch.zeros(H * d, device="cuda")
        slots, z0 = n // L.GATED_CHUNK + users, H * (2 * d + dv)
        kw = {"gated linear attention": dict(gate=L.GATE_ROOT_SIGMOID, tau=16.0), "time mixing": dict(gate=L.GATE_EXP_EXP, bonus=vec),
              "gated delta rule": dict(gate=L.GATE_SOFTPLUS, rate=torch.ones(H, device="cuda"), beta=x[:, z0 + H * d:])}[name]
        scratch = torch.zeros((L.delta_chunk_floats if "beta" in kw else L.gated_chunk_floats)(n, users, H, d, dv), device="cuda")

        def scan(b, n_seq, **more):
            L.gated_scan(b, n_seq, x, x[:, 2 * H * d:], y, state, H, d, dv, k=x[:, H * d:], f=x[:, z0:], f_bias=vec - 2, **kw, **more)

        b, hold = _sequences(n, 1)
        more = dict(u=u) if "beta" in kw else {}
        _timed(f"{name}, chunked, {n} rows", lambda: scan(b, 1, max_chunks=n // L.GATED_CHUNK, scratch=scratch, chunk_slots=slots, **more))
        for m in (1, users):
            b1, hold1 = _sequences(1, m)
            _timed(f"{name}, token by token, {m} sequences of one row ({2 * m * H * d * dv * 4 / 1e6:.1f} MB of state)", lambda: scan(b1, m), 3)


def biased_attention(a):
    import torch
    from dllama_b200.ops import layers as L
    H, G, d, n = 16, 4, 128, 2048
    n_pages = n // 32
    bt = torch.arange(n_pages, dtype=torch.int32).view(1, -1).cuda()
    cache = torch.randn(n_pages, G, 32, 2 * d, device="cuda").to(torch.bfloat16)
    g = torch.Generator().manual_seed(1)
    q, gate = torch.randn(n, H * d, generator=g).cuda(), torch.randn(n, H, generator=g).cuda()
    pos, slot = torch.arange(n, dtype=torch.int32).cuda(), torch.zeros(n, dtype=torch.int32).cuda()
    out, sink, slope = torch.zeros(n, H * d, device="cuda"), torch.zeros(H, device="cuda"), torch.full((H,), 0.01, device="cuda")
    rq = L.window_tc_rows(H, G)
    tiles = torch.arange(n, dtype=torch.int32).view(-1, rq).cuda()
    rq2 = L.talk_tc_rows(H, G, d, d, 0, n)
    tiles2 = torch.arange(n, dtype=torch.int32).view(-1, rq2).cuda()
    for what, cap, window, sl in (("soft-capped", 50.0, 0, None), ("distance bias, window 1024", 0.0, 1024, slope)):
        _timed(f"windowed-attention kernel, {what}", lambda: L.window_attention_tc(q, out, H, G, d, 0, 0.09, cap, window, pos, slot, bt, cache, tiles, n // rq, rq,
                                                                                  vdim=d, sink=sink, slope=sl, gate=gate))
        _timed(f"own-width kernel, {what}", lambda: L.talk_attention_tc(q, out, H, G, d, d, 0.09, window, pos, slot, bt, cache, tiles2, n // rq2, rq2,
                                                                       sink=sink, softcap=cap, slope=sl, gate=gate))
        pairs = sum(min(i + 1, window or n) for i in range(n))
        print("FLOPs per launch (visible pairs): %.1f G" % (pairs * H * 4 * d / 1e9))


def selective_scan(a):
    import torch
    from dllama_b200.ops import layers as L
    n, users, inner, N, r = 2048, 32, 4096, 16, 128
    g = torch.Generator().manual_seed(1)
    x, dt, z = (torch.randn(n, inner, generator=g).cuda() for _ in range(3))
    dbc = torch.randn(n, r + 2 * N, generator=g).cuda()
    A2, bias, D = -torch.exp(torch.randn(inner, N, generator=g) * 0.5).cuda(), torch.full((inner,), -3.0, device="cuda"), torch.ones(inner, device="cuda")
    state, y = torch.zeros(users, inner, N, device="cuda"), torch.zeros(n, inner, device="cuda")
    slots = n // L.SELECTIVE_CHUNK + 1
    scratch = torch.zeros(slots * inner * (N + 1), device="cuda")
    for rows, n_seq, chunked in ((n, 1, True), (n, 1, False), (1, users, False)):
        b, hold = _sequences(rows, n_seq)
        kw = dict(max_chunks=n // L.SELECTIVE_CHUNK, scratch=scratch, chunk_slots=slots) if chunked else {}
        _timed(f"selective scan, {n_seq} sequences of {rows} rows{', chunked' if chunked else ''}",
               lambda: L.selective_scan(b, n_seq, x, dt, dbc[:, r:], dbc[:, r + N:], bias, A2, D, state, y, inner, N, rows, z=z, **kw))


def wide_attention(a):
    import torch
    from dllama_b200.ops import layers as L
    H, G, d, dv, n = 16, 4, 128, 128, 2048
    n_pages = n // 32
    bt = torch.arange(n_pages, dtype=torch.int32).view(1, -1).cuda()
    cache = torch.randn(n_pages, G, 32, d + dv, device="cuda").to(torch.bfloat16)
    g = torch.Generator().manual_seed(1)
    q, talk = torch.randn(n, H * d, generator=g).cuda(), (torch.eye(H) + torch.randn(H, H, generator=g) * 0.3).cuda()
    pos, slot = torch.arange(n, dtype=torch.int32).cuda(), torch.zeros(n, dtype=torch.int32).cuda()
    wide, out = torch.zeros(n, H * G * dv, device="cuda"), torch.zeros(n, H * dv, device="cuda")
    rq = L.talk_tc_rows(H, G, d, dv, 0, n, G)
    tiles = torch.arange(n, dtype=torch.int32).view(-1, rq).cuda()
    _timed("attention, weights against all value heads, tiles of %d rows" % rq,
           lambda: L.talk_attention_tc(q, wide, H, G, d, dv, 0.1, 0, pos, slot, bt, cache, tiles, n // rq, rq, 1, None, value_heads=G))
    _timed("mix of the heads' outputs", lambda: L.talk_mix(wide, talk, n, H, G, dv, out))
    pairs = n * (n + 1) // 2
    print("FLOPs per launch (visible pairs, 2 * (128 + 4 * 128) per head): %.1f G" % (pairs * H * 2 * (d + G * dv) / 1e9))


if __name__ == "__main__":
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("what", choices=("steps", "window-attention", "lightning-scan", "talk-attention", "gated-scan", "delta-scan", "selective-scan", "wide-attention", "biased-attention"))
    ap.add_argument("--design", default="sunesun", choices=("ribivik", "sunesun", "venadra", "darusun", "vopedra", "silizen"))
    ap.add_argument("--size", default="w2048")
    ap.add_argument("--layers", type=int, default=4)
    ap.add_argument("--prompt", type=int, default=2048)
    ap.add_argument("--model-dir", default="/tmp")
    a = ap.parse_args()
    {"steps": steps, "window-attention": window_attention, "lightning-scan": lightning_scan, "talk-attention": talk_attention,
     "gated-scan": gated_scan, "delta-scan": delta_scan, "biased-attention": biased_attention, "selective-scan": selective_scan, "wide-attention": wide_attention}[a.what](a)
