"""Ranilix on the GPU against the plain implementation: each mechanism alone, then the model through the engine
(whole prompts, the stream after every layer, token by token, unequal batches, reused slots and pages, keys far away and
at the edges of windows and pages, old tokens in a decaying state, the first tokens, long decoding, greedy generation,
the command line, trace replay)."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_ranilix as plain
import trapetum_b200 as tb
from conftest import ROOT, rel_l2, within
from ranilix_util import (CONFIGS, attention, config, doubles, parallel, position_errors, prompts, random_weights, tolerance,
                          worst_ratio, write_folder)

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}
F = torch.float64
PAGE = 64


@pytest.fixture(scope="module")
def weights():
    return {name: random_weights(cfg, 17 + ord(name)) for name, cfg in CONFIGS.items()}


@pytest.fixture(scope="module")
def folders(tmp_path_factory, weights):
    return {name: write_folder(str(tmp_path_factory.mktemp("ranilix" + name)), cfg, weights[name]) for name, cfg in CONFIGS.items()}


@pytest.fixture(scope="module")
def oracles(weights):
    return {name: (cfg, doubles(weights[name])) for name, cfg in CONFIGS.items()}


_MODELS = {}


def model_of(folders, name, dtype):
    if (name, dtype) not in _MODELS:
        _MODELS[(name, dtype)] = tb.load_model(folders[name], dtype, DEV)
    return _MODELS[(name, dtype)]


def close(got, want, tol, what, dtype):
    within(worst_ratio(got, want, tol), 1.0, dtype, what + " (error / tolerance)")


def near(got, want, dtype, what, rel32=2e-5, rel16=2e-2):
    got, want = got.double().cpu(), want.double().cpu()
    err = float((got - want).abs().max() / want.abs().max().clamp_min(1e-30))
    assert err <= (rel32 if dtype == "float32" else rel16), f"{what} [{dtype}]: {err:.3e}"


def dev(t, dt=None):
    return t.to(device=DEV, dtype=dt) if dt is not None else t.to(DEV)


def rounded(t, dtype):
    """What the kernel gets: the values as the dtype stores them, in 64-bit for the oracle."""
    return t.to(DTYPES[dtype]).to(F)


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def split_up(x, n, g):
    """``n`` partial sums (float32, on the device) that add up to x."""
    parts = torch.randn((n,) + tuple(x.shape), generator=g, dtype=F)
    parts[-1] = x - parts[:-1].sum(0)
    return dev(parts, torch.float32)


def starts_of(lens):
    return [0] + torch.tensor(lens).cumsum(0).tolist()


def seq_of(lens):
    return [i for i, n in enumerate(lens) for _ in range(n)]


# ---------------------------------------------------------------------------
# mechanisms alone
# ---------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width, rows", [(48, 5), (50, 3), (2048, 9), (12288, 2)])
def test_terms_added_with_scales_and_two_norms_of_the_sum(width, rows, dtype):
    from trapetum_b200.csrc import ops
    g = torch.Generator().manual_seed(width)
    h = torch.randn(rows, width, generator=g, dtype=F)
    branches = [(torch.randn(rows, width, generator=g, dtype=F), s) for s in (0.75, -1.5, 1.0)]
    w1, w2 = (torch.randn(width, generator=g, dtype=F).float() for _ in range(2))
    for n in range(4):
        x = h + sum((s * b for b, s in branches[:n]), torch.zeros_like(h))
        hd = dev(h, torch.float32)
        terms = [(split_up(b, k + 1, g) if k else dev(b, torch.float32), s) for k, (b, s) in enumerate(branches[:n])]
        a, b = ops.add_terms_rmsnorm(hd, terms, [dev(w1), dev(w2)], 1e-3, 0.0, DTYPES[dtype])
        near(hd, x, "float32", f"sum of {n} terms")
        near(a, plain.norm(x, w1.double(), 1e-3), dtype, "first norm")
        near(b, plain.norm(x, w2.double(), 1e-3), dtype, "second norm")
        hd = dev(h, torch.float32)
        ops.add_terms_rmsnorm(hd, terms)
        near(hd, x, "float32", f"sum of {n} terms alone")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H, G, dim, vdim, pad, R", [(3, 1, 8, 12, 12, 4), (4, 4, 64, 48, 64, 64), (6, 2, 10, 7, 16, 2),
                                                    (16, 4, 128, 128, 128, 32), (2, 1, 48, 96, 128, 0)])
@pytest.mark.parametrize("mix", [False, True])
def test_head_norms_biases_rotation_and_mixed_values_in_one_kernel(H, G, dim, vdim, pad, R, mix, dtype):
    """Also the cache write: pages out of order, and a ring that keeps the last 64 rows."""
    from trapetum_b200.csrc import ops
    g = torch.Generator().manual_seed(H * 10 + dim)
    lens, T = [70, 3], 73
    width = (H + G) * dim + G * vdim
    x, bias = torch.randn(T, width, generator=g, dtype=F) * 2, torch.randn((width + 3) // 4 * 4, generator=g).float()
    wq, wk = torch.randn(dim, generator=g).float(), torch.randn(dim, generator=g).float()
    first = torch.randn(T, G * vdim, generator=g).float()
    full = torch.cat([x, torch.randn(T, -width % 16, generator=g, dtype=F)], dim=1)
    part = split_up(full, 3, g)
    pos = torch.cat([torch.arange(n) + 5 for n in lens])
    base, eps, lam = 50.0, 1e-4, 0.3
    freq = dev(plain.frequencies(R, base), torch.float32) if R else None
    y = x + bias[:width].double()
    q = plain.turn(plain.norm(y[:, :H * dim].view(T, H, dim), wq.double(), eps), pos, R, base, False)
    k = plain.turn(plain.norm(y[:, H * dim:(H + G) * dim].view(T, G, dim), wk.double(), eps), pos, R, base, False)
    v = y[:, (H + G) * dim:].view(T, G, vdim)
    vm = (1 - lam) * v + lam * first.double().view(T, G, vdim) if mix else v
    for ring in (0, 64):
        pool = [torch.zeros(8, G, PAGE, pad, dtype=DTYPES[dtype], device=DEV) for _ in range(2)]
        table = i32([[5, 2], [3, 0]])
        keep = torch.empty(T, G * vdim, dtype=torch.float32, device=DEV)
        out, _ = ops.projnorm_kv(part, H, G, dim, vdim, pad, DTYPES[dtype], dev(wq), dev(wk), eps, None, R, freq, False, i32(pos.tolist()),
                                 i32(seq_of(lens)), i32([n + 5 for n in lens]), pool[0], pool[1], table, ring, dev(bias), True,
                                 dev(first) if mix else None, lam, keep)
        out = out.view(T, H + 2 * G, pad).double().cpu()
        near(out[:, :H, :dim], q, dtype, "q")
        near(out[:, H:H + G, :dim], k, dtype, "k")
        near(out[:, H + G:, :vdim], vm, dtype, "v")
        assert float(out[:, :H + G, dim:].abs().max() if pad > dim else 0.0) == 0.0
        near(keep.view(T, G, vdim), v, "float32", "kept values")
        for t, (b, p) in enumerate(zip(seq_of(lens), pos.tolist())):
            if ring and p < lens[b] + 5 - ring:
                continue
            r = p % ring if ring else p
            page = int(table[b, r // PAGE])
            assert torch.equal(pool[0][page, :, r % PAGE].double().cpu(), out[t, H:H + G]) and \
                torch.equal(pool[1][page, :, r % PAGE].double().cpu(), out[t, H + G:])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T, H, D, V, splits", [(3, 4, 64, 48, 2), (70, 3, 12, 7, 1), (1, 16, 128, 128, 4), (5, 2, 16, 16, 9)])
def test_the_gate_of_every_output_number(T, H, D, V, splits, dtype):
    from trapetum_b200.csrc import ops
    g = torch.Generator().manual_seed(T)
    o = rounded(torch.randn(T, H, D, generator=g), dtype)
    z = torch.randn(T, H * V, generator=g, dtype=F) * 3
    wide = split_up(torch.cat([torch.randn(T, 8, generator=g, dtype=F), z], dim=1), splits, g)
    got = ops.value_gate(dev(o.reshape(T, H * D), DTYPES[dtype]), wide[:, :, 8:], H, V)
    near(got, o[..., :V].reshape(T, H * V) * torch.sigmoid(z), dtype, "gate")


SINK_SHAPES = [(3, 1, 12, 5), (4, 4, 64, 64), (8, 2, 64, 65), (2, 1, 128, 0), (16, 2, 128, 100), (6, 6, 48, 7), (4, 1, 256, 0), (8, 8, 32, 33)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H, G, D, window", SINK_SHAPES)
def test_softmax_with_a_sink_in_prompts(H, G, D, window, dtype):
    from trapetum_b200.csrc import ops
    g = torch.Generator().manual_seed(H + D)
    lens = [1, 130, 37]
    T = sum(lens)
    sink = torch.tensor([(-30.0, 0.5, 2.0, 80.0, 4.0)[h % 5] for h in range(H)])
    x = rounded(torch.randn(T, H + 2 * G, D, generator=g), dtype)
    want, st = [], starts_of(lens)
    for a, b in zip(st, st[1:]):
        want.append(plain.attend(x[a:b, :H], x[a:b, H:H + G], x[a:b, H + G:], torch.arange(b - a), 0.3, window or None, sink.double()))
    qkv = dev(x.reshape(T, -1), DTYPES[dtype])
    got = ops.attn_prefill_sink(qkv[:, :H * D], qkv[:, H * D:(H + G) * D], qkv[:, (H + G) * D:], i32(st), i32(seq_of(lens)), H, D, 0.3,
                                dev(sink), max(lens), lens, window, n_kv_heads=G)
    got = got.view(T, H, D)
    for h in range(H):
        if sink[h] < 50:                                  # (a head whose sink takes everything leaves nothing to compare)
            near(got[:, h], torch.cat(want)[:, h], dtype, f"head {h}, sink {float(sink[h])}", rel16=1.5e-2)
        else:
            assert float(got[:, h].abs().max()) < 1e-5


@pytest.mark.parametrize("partition", ["split", "stream", None])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H, G, D, window", SINK_SHAPES)
def test_softmax_with_a_sink_over_the_cache(H, G, D, window, dtype, partition):
    """One piece and several, lengths around the edges of pages, windows and rings that have wrapped, pages out of order."""
    from trapetum_b200.csrc import ops
    if partition is not None and dtype == "float32":
        pytest.skip("the float32 kernel has one partition")
    g = torch.Generator().manual_seed(H * 3 + D)
    lens = [1, 64, 65, 63, 300, 129]
    B = len(lens)
    ring = (window + 63) // 64 * 64 if window else 0
    sink = torch.tensor([(-30.0, 0.5, 2.0, 4.0)[h % 4] for h in range(H)])
    ks, vs = ([rounded(torch.randn(n, G, D, generator=g), dtype) for n in lens] for _ in range(2))
    order = torch.randperm(32, generator=g).tolist()
    pools = [torch.full((32, G, PAGE, D), float("nan")) for _ in range(2)]
    table, at = [], 0
    for b, n in enumerate(lens):
        held = min(n, ring) if ring else n
        mine = order[at:at + (held + PAGE - 1) // PAGE]
        at += len(mine)
        for p in range(max(0, n - ring) if ring else 0, n):
            r = p % ring if ring else p
            pools[0][mine[r // PAGE], :, r % PAGE] = ks[b][p].float()
            pools[1][mine[r // PAGE], :, r % PAGE] = vs[b][p].float()
        table.append(mine + [0] * (8 - len(mine)))
    kp, vp = (dev(p, DTYPES[dtype]).contiguous() for p in pools)         # rows that hold no key stay NaN
    q = rounded(torch.randn(B, H, D, generator=g), dtype)
    want = torch.cat([plain.attend(q[b:b + 1], ks[b], vs[b], torch.tensor([n - 1]), 0.3, window or None, sink.double()) for b, n in enumerate(lens)])
    was = ops.set_decode_partition(partition)
    try:
        for bucket in (512, 8192):                                       # the second cuts every sequence into pieces
            got = ops.attn_decode(dev(q.reshape(B, -1), DTYPES[dtype]), kp, vp, i32(table), i32(lens), H, G, D, 0.3, 0.0, window, ring,
                                  bucket, sink=dev(sink))
            near(got.view(B, H, D), want, dtype, f"bucket {bucket}", rel16=1.5e-2)
    finally:
        ops.set_decode_partition(was)
    assert not ops.kernel_errors()


RETENTION_SHAPES = [(3, 12, 10, 6, (0.5, 0.9, 1.0)), (2, 64, 64, 64, (0.97, 0.999)), (4, 64, 96, 32, (0.9, 0.99, 0.999, 0.6)),
                    (2, 128, 160, 128, (0.95, 0.9995)), (1, 128, 256, 64, (0.998,)), (2, 256, 512, 256, (0.99, 0.9)),
                    (1, 10, 7, 0, (0.93,)), (5, 32, 48, 16, (0.99, 0.5, 0.8, 1.0, 0.2)), (2, 96, 32, 48, (0.98, 0.7)),
                    (2, 64, 40, 64, (0.98, 0.9)), (1, 80, 200, 80, (0.99,)), (1, 256, 48, 128, (0.995,))]


@pytest.mark.parametrize("generic", [False, True])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H, D, V, R, decay", RETENTION_SHAPES)
def test_retention_between_its_products(H, D, V, R, decay, dtype, generic):
    """Prompts of several lengths in one step (around the edges of chunks), then one token each, from states in slots out of
    order; what the slots of other sequences hold stays as it is."""
    from trapetum_b200.csrc import ops
    g = torch.Generator().manual_seed(H * 7 + D + V)
    base, eps, k_scale = 300.0, 1e-4, D ** -0.5
    HD, HV = H * D, H * V
    freq = dev(plain.frequencies(R, base), torch.float32) if R else None
    dec = torch.tensor(decay)

    def truth(x, pos, S):
        q = plain.turn(x[:, :HD].view(-1, H, D), pos, R, base, False)
        k = plain.turn(x[:, HD:2 * HD].view(-1, H, D), pos, R, base, False) * k_scale
        v = rounded(x[:, 2 * HD:2 * HD + HV], dtype).view(-1, H, V)
        o, S = plain.retain(q, k, v, dec.double().tolist(), S)
        return plain.unit(o, eps).reshape(-1, HV) * plain.silu(x[:, 2 * HD + HV:2 * HD + 2 * HV]), S

    for lens, longest in (([1, 2, 65, 130, 64], 130), ([700], 700), ([3, 300], 300), ([1100, 257, 128, 129], 1100)):
        B, T = len(lens), sum(lens)
        slots = [6, 1, 4, 0, 3][:B]
        state = torch.randn(8, HD * V, generator=g).float().to(DEV)
        untouched = state.clone()
        for s in slots:
            state[s] = 0
        x = torch.randn(T, 2 * HD + 2 * HV, generator=g, dtype=F).float().double()
        wide = torch.cat([x, torch.zeros(T, 16, dtype=F)], dim=1)
        st = starts_of(lens)
        pos = torch.cat([torch.arange(n) for n in lens])
        got = ops.retention(split_up(wide, 2, g), H, D, V, DTYPES[dtype], R, freq, k_scale, dev(dec), eps, state, i32(pos.tolist()), i32(st),
                            i32(seq_of(lens)), i32(slots), B, longest, generic=generic)
        S = []
        for a, b in zip(st, st[1:]):
            want, s = truth(x[a:b], pos[a:b], torch.zeros(H, D, V, dtype=F))
            # (the unit norm enlarges what rounding leaves of an output that almost cancels: a looser bound on single numbers)
            near(got[a:b], want, dtype, f"a prompt of {b - a} in {lens}", rel32=2e-4, rel16=0.1)
            assert rel_l2(got[a:b], want) <= (5e-5 if dtype == "float32" else 1.5e-2)
            S.append(s)
        for b, s in enumerate(slots):
            near(state[s].view(H, D, V), S[b], dtype, f"the state after {lens[b]} tokens", rel32=5e-5, rel16=6e-3)
            assert rel_l2(state[s].view(H, D, V), S[b]) <= (5e-5 if dtype == "float32" else 3e-3)
        for step in range(3):
            x = torch.randn(B, 2 * HD + 2 * HV, generator=g, dtype=F).float().double()
            pos = torch.tensor(lens) + step
            got = ops.retention(split_up(x, 3, g), H, D, V, DTYPES[dtype], R, freq, k_scale, dev(dec), eps, state, i32(pos.tolist()),
                                i32(list(range(B + 1))), i32(list(range(B))), i32(slots), B, generic=generic)
            for b in range(B):
                want, S[b] = truth(x[b:b + 1], pos[b:b + 1], S[b])
                near(got[b:b + 1], want, dtype, f"token {step} after {lens[b]}", rel32=2e-4, rel16=3e-2)
        for s in range(8):
            if s not in slots:
                assert torch.equal(state[s], untouched[s])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("decay", [0.9, 0.0])
def test_a_tokens_own_product_keeps_its_sign(dtype, decay):
    """A sequence's first token (and every token of a head that forgets at once) gives (q . k) v, of which the norm leaves
    the sign of q . k: products that nearly cancel, in a prompt and in a one-token step."""
    from trapetum_b200.csrc import ops
    g = torch.Generator().manual_seed(5)
    H, D, V, n = 4, 64, 64, 40
    q = torch.randn(n, H, D, generator=g, dtype=F)
    k = torch.randn(n, H, D, generator=g, dtype=F)
    k = k - q * ((q * k).sum(-1, keepdim=True) / (q * q).sum(-1, keepdim=True))       # orthogonal, then a little of q
    k = k + q * torch.where(torch.rand(n, H, 1, generator=g) < 0.5, -1e-4, 1e-4).double()
    v, z = torch.randn(n, H, V, generator=g, dtype=F), torch.full((n, H * V), 3.0, dtype=F)
    x = torch.cat([q.reshape(n, -1), k.reshape(n, -1), v.reshape(n, -1), z], dim=1).float()
    want = torch.sign((x[:, :H * D].double().view(n, H, D) * x[:, H * D:2 * H * D].double().view(n, H, D)).sum(-1))
    dec = torch.full((H,), decay, device=DEV)
    lens = [n] if decay == 0.0 else [1] * n
    pos = torch.zeros(n, dtype=torch.int32, device=DEV)
    for longest in (max(lens), 0):
        steps = [slice(0, n)] if longest or decay else [slice(i, i + 1) for i in range(n)]
        state = torch.zeros(len(lens), H * D * V, device=DEV)
        for sl in steps:
            L = lens if len(steps) == 1 else [1]
            got = ops.retention(dev(x[sl])[None].contiguous(), H, D, V, DTYPES[dtype], 0, None, 1.0, dec, 1e-12, state, pos[sl], i32(starts_of(L)),
                                i32(seq_of(L)), i32(list(range(len(L)))), len(L), longest)
            sign = torch.sign((got.double().cpu().view(-1, H, V) * v[sl]).sum(-1))
            assert torch.equal(sign, want[sl])


# ---------------------------------------------------------------------------
# the model through the engine
# ---------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompts(folders, oracles, name, dtype):
    cfg, w = oracles[name]
    eng = tb.Engine(model_of(folders, name, dtype), max_tokens=1024)
    for ids in prompts(cfg["vocab"], [1, 2, 64, 65, 150, 300], seed=1):
        s = eng.start(1)
        got = eng.step(s, [ids], [list(range(len(ids)))])
        eng.release(s)
        close(got, plain.forward(cfg, w, ids), tolerance(name, cfg, w, ids, dtype), f"{name}: whole prompt of {len(ids)}", dtype)
    eng.check_kernels()


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_the_residual_stream_after_every_layer(folders, oracles, name, monkeypatch):
    from trapetum_b200.parts.block import ParallelBlock
    cfg, w = oracles[name]
    ids = prompts(cfg["vocab"], [75], seed=2)[0]
    seq = plain.Sequence(cfg, w)
    seq.feed(ids)
    seen, orig = [], ParallelBlock.forward

    def spy(self, stream, ctx, cache):
        orig(self, stream, ctx, cache)
        seen.append(stream.value().clone())
    monkeypatch.setattr(ParallelBlock, "forward", spy)
    eng = tb.Engine(model_of(folders, name, "float32"), max_tokens=256)
    eng.step(eng.start(1), [ids], [[0]])
    assert len(seen) == len(seq.streams) == len(cfg["layers"])
    for r, x in enumerate(seen):
        near(x, seq.streams[r], "float32", f"{name}: the stream after layer {r} ({cfg['layers'][r]['type']})", rel32=2e-5)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name, first", [("A", 1), ("A", 2), ("B", 63), ("B", 64), ("B", 7), ("C", 65), ("C", 3)])
def test_prompt_then_token_by_token(folders, oracles, name, first, dtype):
    """Decoding runs across pages' borders (64, 128, 192), over every window's edge (windows of 3 to 100 pass over decoded
    tokens, and the rows of their rings are used again) and through the capture of the step's graph."""
    cfg, w = oracles[name]
    ids = prompts(cfg["vocab"], [215], seed=first)[0]
    truth = plain.forward(cfg, w, ids)
    eng = tb.Engine(model_of(folders, name, dtype), max_tokens=512)
    s = eng.start(1)
    got = [eng.step(s, [ids[:first]], [list(range(first))])] + [eng.step(s, [[t]], [[0]]).clone() for t in ids[first:]]
    eng.release(s)
    assert dtype == "float32" or eng.graphs_captured >= 1
    close(torch.cat(got), truth, tolerance(name, cfg, w, ids, dtype), f"{name}: {first} tokens, then one by one", dtype)
    eng.check_kernels()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(folders, oracles, dtype):
    """600 tokens one by one: the buckets of the captured step change on the way."""
    cfg, w = oracles["A"]
    ids = prompts(cfg["vocab"], [604], seed=21)[0]
    truth = plain.forward(cfg, w, ids)
    eng = tb.Engine(model_of(folders, "A", dtype), max_tokens=1024)
    s = eng.start(1)
    got = [eng.step(s, [ids[:4]], [[3]])] + [eng.step(s, [[t]], [[0]]).clone() for t in ids[4:]]
    eng.release(s)
    close(torch.cat(got), truth[3:], tolerance("Along", cfg, w, ids, dtype)[3:], "600 decoded tokens", dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_unequal_batch_equals_each_alone_and_slots_are_reused(folders, oracles, name, dtype):
    cfg, w = oracles[name]
    eng = tb.Engine(model_of(folders, name, dtype), max_tokens=1024, max_slots=4)
    rounds = [prompts(cfg["vocab"], [1, 90, 33], seed=4), prompts(cfg["vocab"], [70, 2, 129], seed=5)]
    for ps in rounds:                                            # the second round takes the first one's slots and pages
        n_new = 6
        full = [p + q for p, q in zip(ps, prompts(cfg["vocab"], [n_new] * 3, seed=6))]
        truth = [plain.forward(cfg, w, f) for f in full]
        s = eng.start(3)
        got = [[] for _ in ps]
        out = eng.step(s, ps, [[len(p) - 1] for p in ps])
        for i in range(3):
            got[i].append(out[i:i + 1].clone())
        live = [0, 1, 2]
        for j in range(n_new):
            if j == 3:
                eng.release([s[1]])                              # the middle one ends early; the others go on
                live = [0, 2]
            out = eng.step([s[i] for i in live], [[full[i][len(ps[i]) + j]] for i in live], [[0]] * len(live))
            for r, i in enumerate(live):
                got[i].append(out[r:r + 1].clone())
        eng.release([s[i] for i in live])
        eng.cache.check()
        for i in range(3):
            g = torch.cat(got[i])
            lo = len(ps[i]) - 1
            close(g, truth[i][lo:lo + g.shape[0]], tolerance(name + "u", cfg, w, full[i], dtype)[lo:lo + g.shape[0]],
                  f"{name}: request {i} of an unequal batch", dtype)
    eng.check_kernels()


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_decoding_in_a_large_batch(folders, oracles, name):
    """More tokens in a step than the split products take, through the same kernels."""
    cfg, w = oracles[name]
    ps = prompts(cfg["vocab"], [3 + i % 9 for i in range(140)], seed=31)
    nxt = prompts(cfg["vocab"], [2] * 140, seed=32)
    eng = tb.Engine(model_of(folders, name, "bfloat16"), max_tokens=140 * 64, max_slots=140)
    s = eng.start(140)
    eng.step(s, ps, [[]] * 140)
    got = [eng.step(s, [[t[j]] for t in nxt], [[0]] * 140).clone() for j in range(2)]
    for i in (0, 5, 77, 139):
        full = ps[i] + nxt[i]
        close(torch.stack([got[0][i], got[1][i]]), plain.forward(cfg, w, full)[-2:], tolerance(name, cfg, w, full, "bfloat16")[-2:],
              f"{name}: request {i} of 140", "bfloat16")


def _layer(kind, size):
    if kind == "attention":
        return attention(2, 1, 16, 24, 0.5, size=size, rot=(8, 10000.0))
    return parallel((2, 1, 16, 24, 0.25, (8, 10000.0)), (16, 16, (16, 10000.0), (0.999, 0.9999)), 0.0 if kind == "retention" else 1.0,
                    1.0 if kind == "retention" else 0.0)


def _needle(tmp_path, kind, size, key_pos, n, probe, least=0.05):
    """A one-layer model without feed-forward whose scores are sharpened, and a prompt of one repeated token with a single
    other token at ``key_pos``, chosen (with the plain implementation) as the one that the query at ``probe`` singles
    out most."""
    cfg = config(50, 32, [(_layer(kind, size), None)])
    w = random_weights(cfg, 5, sharp=4.0)
    if kind == "attention":
        w["l0.mix.q.b"] *= 0                                     # the needle's own content decides
    wd = doubles(w)
    base = [3] * n
    without = plain.forward(cfg, wd, base)[probe:probe + 1]
    best, ids = -1.0, None
    for cand in range(4, 24):
        trial = list(base)
        trial[key_pos] = cand
        e = float(position_errors(plain.forward(cfg, wd, trial)[probe:probe + 1], without))
        if e > best:
            best, ids = e, trial
    assert best > least, best
    folder = write_folder(str(tmp_path / f"needle_{kind}_{size}_{key_pos}_{n}"), cfg, w)
    return cfg, wd, ids, folder


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["attention", "left"])
@pytest.mark.parametrize("key_pos, n", [(0, 200), (63, 130), (64, 130), (5, 700)])
def test_a_far_key_is_found_in_prompts_and_in_decoding(tmp_path, kind, key_pos, n, dtype):
    """No mask: every earlier token is seen, also the first one and those at a page's edge, hundreds of tokens back."""
    cfg, w, ids, folder = _needle(tmp_path, kind, None, key_pos, n, n - 1)
    truth = plain.forward(cfg, w, ids)
    tol = tolerance(("far", kind, key_pos, n), cfg, w, ids, dtype)
    eng = tb.Engine(tb.load_model(folder, dtype, DEV), max_tokens=1024)
    s = eng.start(1)
    close(eng.step(s, [ids], [[n - 1]]), truth[-1:], tol[-1:], f"{kind}: needle at {key_pos} of {n}, prompt", dtype)
    eng.release(s)
    s = eng.start(1)
    eng.step(s, [ids[:n - 3]], [[]])
    got = torch.cat([eng.step(s, [[t]], [[0]]).clone() for t in ids[n - 3:]])
    close(got, truth[-3:], tol[-3:], f"{kind}: needle at {key_pos} of {n}, decoded", dtype)
    eng.check_kernels()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("size, key_pos", [(48, 1), (48, 30), (64, 0), (64, 63), (64, 70), (65, 63), (65, 64), (130, 2), (2, 77), (1, 50), (100, 127)])
def test_a_key_at_a_windows_edge_in_prompts_and_in_decoding(tmp_path, size, key_pos, dtype):
    """The key is seen by the queries up to ``size - 1`` behind it and by none after them: the logits of the last query that
    sees it and of the first that does not, in a prompt and decoded."""
    last = key_pos + size - 1
    n = last + 3
    cfg, w, ids, folder = _needle(tmp_path, "attention", size, key_pos, n, last)
    truth = plain.forward(cfg, w, ids)
    blind = plain.forward(cfg, w, [3] * n)
    assert float(position_errors(truth[last:last + 1], blind[last:last + 1])) > 0.05
    assert float((truth[last + 1:] - blind[last + 1:]).abs().max()) == 0.0
    first = max(1, last - 2)
    tol = tolerance(("edge", size, key_pos), cfg, w, ids, dtype)
    eng = tb.Engine(tb.load_model(folder, dtype, DEV), max_tokens=512)
    s = eng.start(1)
    close(eng.step(s, [ids], [list(range(n))]), truth, tol, f"window {size}, key at {key_pos}: prompt", dtype)
    eng.release(s)
    s = eng.start(1)
    got = [eng.step(s, [ids[:first]], [[first - 1]])] + [eng.step(s, [[t]], [[0]]).clone() for t in ids[first:]]
    close(torch.cat(got), truth[first - 1:], tol[first - 1:], f"window {size}, key at {key_pos}: decoded", dtype)
    eng.release(s)
    eng.check_kernels()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key_pos, n, first", [(0, 150, 1), (63, 150, 64), (64, 150, 100), (127, 400, 128), (0, 400, 399)])
def test_an_old_token_stays_in_the_state(tmp_path, key_pos, n, first, dtype):
    """Slow decays: the first token and those at the edges of a chunk still show in the last logits, whether they were read
    in the prompt or decoded."""
    cfg, w, ids, folder = _needle(tmp_path, "retention", None, key_pos, n, n - 1, least=0.003)
    truth = plain.forward(cfg, w, ids)
    blind = plain.forward(cfg, w, [3] * n)
    eng = tb.Engine(tb.load_model(folder, dtype, DEV), max_tokens=512)
    s = eng.start(1)
    got = [eng.step(s, [ids[:first]], [list(range(first))])] + [eng.step(s, [[t]], [[0]]).clone() for t in ids[first:]]
    eng.release(s)
    got = torch.cat(got)
    close(got, truth, tolerance(("old", key_pos, n), cfg, w, ids, dtype), f"token {key_pos} of {n} in the state, {first} first", dtype)
    # and it is this token that shows: the engine follows the truth more closely than the prompt without it
    if dtype == "float32":
        assert float(position_errors(got[-1:], truth[-1:])) < 0.05 * float(position_errors(blind[-1:], truth[-1:]))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_what_the_design_adds_would_show(tmp_path, dtype):
    """The engine follows the plain implementation, and the plain implementation without the sinks, biases, head norms'
    weights, mixed values, gates or with other norms is far away."""
    cfg = config(60, 40, [(attention(2, 2, 8, 12, 0.5, size=9, rot=(8, 100.0), v_mix=True), 24),
                          (parallel((2, 1, 8, 12, 0.5, (8, 100.0)), (8, 12, (8, 100.0), (0.9, 0.8)), 0.7, 1.4), 24),
                          (attention(2, 2, 8, 12, 0.5, size=6, rot=(4, 100.0), v_mix=True), None)], scale=2.0)
    w = {k: v.float() for k, v in random_weights(cfg, 9).items()}
    w["l0.mix.sink"] += 1.0
    w["l2.mix.vmix"] = torch.tensor(0.7)
    w = {k: v.to(torch.bfloat16) for k, v in w.items()}
    wd = doubles(w)
    ids = prompts(60, [40], seed=3)[0]
    truth = plain.forward(cfg, wd, ids)
    for name, value in (("l0.mix.sink", torch.full((2,), -50.0, dtype=F)), ("l0.mix.q.b", torch.zeros(16, dtype=F)),
                        ("l2.mix.vmix", torch.zeros((), dtype=F)), ("l2.mix.g", torch.zeros(24, 40, dtype=F)),
                        ("l0.mix.k.norm", torch.ones(8, dtype=F)), ("l0.norm2", wd["l0.norm1"]), ("l1.mix.right.g", wd["l1.mix.right.v"])):
        other = dict(wd)
        other[name] = value
        assert float(position_errors(plain.forward(cfg, other, ids), truth).median()) > 0.03, name
    eng = tb.Engine(tb.load_model(write_folder(str(tmp_path / "adds"), cfg, w), dtype, DEV), max_tokens=256)
    s = eng.start(1)
    got = [eng.step(s, [ids[:30]], [list(range(30))])] + [eng.step(s, [[t]], [[0]]).clone() for t in ids[30:]]
    close(torch.cat(got), truth, tolerance("adds", cfg, wd, ids, dtype), "everything together: prompt then decoding", dtype)


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_greedy_generation_through_the_library(folders, oracles, name):
    cfg, w = oracles[name]
    ps = prompts(cfg["vocab"], [5, 1, 70, 12], seed=9)
    want = [plain.generate_greedy(cfg, w, p, 10) for p in ps]
    model = model_of(folders, name, "float32")
    assert tb.generate(model, ps, max_tokens=10, stop_ids=[]) == want
    assert tb.generate(model, ps, max_tokens=10, stop_ids=[], max_batch=2) == want      # two batches, slots used again
    got16 = tb.generate(model_of(folders, name, "bfloat16"), ps, max_tokens=10, stop_ids=[])
    assert all(len(o) == 10 for o in got16)


def test_command_line_runs_the_model(folders, oracles):
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "gemma_run"), folders["A"], "--prompt_ids", "5,17,3",
                           "--max_tokens", "5", "--dtype", "float32"], capture_output=True, text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-3000:]
    cfg, w = oracles["A"]
    assert f"continuation ids: {plain.generate_greedy(cfg, w, [5, 17, 3], 5)}" in proc.stdout


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay(folders, oracles, tmp_path, dtype):
    """Two requests start together, are decoded together, one ends early; a third starts from one token later and
    takes the freed slot and pages."""
    cfg, w = oracles["B"]
    a, b, c = prompts(cfg["vocab"], [70, 9, 1], seed=11)
    tail = prompts(cfg["vocab"], [3, 2, 66], seed=12)
    steps = []

    def add(entries, end=()):
        steps.append({"step": len(steps), "entries": entries, "end": list(end)})
    add([{"id": "a", "tokens": a, "want": [0, 69]}, {"id": "b", "tokens": b, "want": [8]}])
    for j in range(2):
        add([{"id": "a", "tokens": [tail[0][j]], "want": [0]}, {"id": "b", "tokens": [tail[1][j]], "want": [0] if j else []}],
            end=["b"] if j else [])
    add([{"id": "a", "tokens": [tail[0][2]], "want": [0]}], end=["a"])
    add([{"id": "c", "tokens": c, "want": [0]}])
    for j in range(66):
        add([{"id": "c", "tokens": [tail[2][j]], "want": [0] if j >= 60 else []}])
    out = tmp_path / "out"
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folders["B"], "--dtype", dtype,
                           "--out", str(out), "--max-tokens", "512"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                          capture_output=True, text=True, timeout=1200)
    assert proc.returncode == 0, proc.stderr[-3000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(len(steps))]
    full = {"a": a + tail[0], "b": b + tail[1], "c": c + tail[2]}
    truth = {k: plain.forward(cfg, w, v) for k, v in full.items()}
    at = {k: 0 for k in full}
    for st in steps:
        rows = []
        for e in st["entries"]:
            rows += [(e["id"], at[e["id"]] + p) for p in e["want"]]
            at[e["id"]] += len(e["tokens"])
        path = out / f"{st['step']}.f32"
        if not rows:
            assert not path.exists()
            continue
        got = torch.from_numpy(np.fromfile(path, dtype="<f4").reshape(len(rows), cfg["vocab"]))
        for r, (i, p) in enumerate(rows):
            tol = tolerance("trace" + i, cfg, w, full[i], dtype)[p:p + 1]
            close(got[r:r + 1], truth[i][p:p + 1], tol, f"trace: request {i}, position {p}", dtype)
