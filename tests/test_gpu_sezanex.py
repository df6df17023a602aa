"""Sezanex on the GPU against the plain implementation: each mechanism alone, then the model through the engine
(whole prompts, the stream after every layer call, token by token, unequal batches, reused slots and pages, keys far away
and at the edges of windows and pages, old tokens in a decaying state, the first tokens, long decoding, greedy
generation, the command line, trace replay)."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_sezanex as plain
import trapetum_b200 as tb
from conftest import ROOT, rel_l2, within
from sezanex_util import (CONFIGS, attention, config, dense, doubles, mamba2, moe, position_errors, prompts, random_weights, tolerance,
                          worst_ratio, write_folder)

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}
F = torch.float64
PAGE = 64
_route = plain.route


@pytest.fixture(scope="module")
def weights():
    return {name: random_weights(cfg, 23 + ord(name)) for name, cfg in CONFIGS.items()}


@pytest.fixture(scope="module")
def folders(tmp_path_factory, weights):
    return {name: write_folder(str(tmp_path_factory.mktemp("sezanex" + name)), cfg, weights[name]) for name, cfg in CONFIGS.items()}


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
@pytest.mark.parametrize("rows, width, splits", [(1, 48, 1), (3, 50, 2), (9, 2048, 9), (300, 128, 1), (261, 50, 1), (258, 260, 3)])
def test_the_dynamic_tanh_norm_around_the_residual_sum(rows, width, splits, dtype):
    """Every form: the norm alone, of a branch, of the sum, of a product that replaces the stream, and copies of the stream
    into a part of a wider matrix whose other part stays."""
    from trapetum_b200.csrc import ops
    g = torch.Generator().manual_seed(rows + width)
    dt = DTYPES[dtype]

    def norm(alpha):
        return alpha, torch.randn(width, generator=g), torch.randn(width, generator=g)

    def applied(n, x):
        return plain.dyt(x, n[0], n[1].double(), n[2].double())

    def on(n):
        return n[0], dev(n[1]), dev(n[2])
    na, nb = norm(0.37), norm(1.6)
    h, a = torch.randn(rows, width, generator=g, dtype=F).float().double() * 2, torch.randn(rows, width, generator=g, dtype=F) * 2
    part = split_up(a, splits, g) if splits > 1 else dev(a, torch.float32)[None]
    total = h + applied(na, a)

    def stream():
        return dev(h, torch.float32)
    hd = stream()
    near(ops.dyt(hd, part, on(na), on(nb), dt), applied(nb, total), dtype, "sum and two norms", rel16=6e-3)
    near(hd, total, "float32", "the sum")
    hd = stream()
    assert ops.dyt(hd, part, on(na)) is None
    near(hd, total, "float32", "the sum alone")
    hd = stream()
    near(ops.dyt(hd, part, None, on(nb), dt, replace=True), applied(nb, a), dtype, "replaced", rel16=6e-3)
    near(hd, a, "float32", "the stream replaced")
    hd = stream()
    near(ops.dyt(hd, None, None, on(nb), dt), applied(nb, h), dtype, "the stream's norm", rel16=6e-3)
    assert torch.equal(hd, stream())
    branch = rounded(a, dtype)
    near(ops.dyt(None, dev(branch, dt), norm_b=on(nb), out_dtype=torch.float32), applied(nb, branch), "float32", "a matrix' norm")
    near(ops.dyt(stream(), dev(branch, dt), on(na), on(nb), dt), applied(nb, h + applied(na, branch)), dtype, "a branch of the dtype", rel16=6e-3)
    wide = torch.full((rows, 2 * width), 7.0, dtype=dt, device=DEV)
    hd = stream()
    ops.dyt(hd, part, on(na), out=wide[:, width:])
    assert torch.equal(wide[:, width:], hd.to(dt)) and bool((wide[:, :width] == 7.0).all())
    near(hd, total, "float32", "the sum beside a copy")
    ops.dyt(hd, out=wide[:, :width])
    assert torch.equal(wide[:, :width], hd.to(dt))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H, G, dim, vdim, pad, R", [(3, 1, 12, 16, 16, 4), (4, 4, 64, 48, 64, 64), (6, 2, 10, 7, 16, 2),
                                                    (16, 4, 128, 128, 128, 32), (2, 1, 48, 96, 128, 48)])
def test_projection_norms_and_a_rotation_with_a_factor(H, G, dim, vdim, pad, R, dtype):
    """Also the cache write: pages out of order, and a ring that keeps the last 64 rows."""
    from trapetum_b200.csrc import ops
    g = torch.Generator().manual_seed(H * 10 + dim)
    lens, T = [70, 3], 73
    width = (H + G) * dim + G * vdim
    x = torch.randn(T, width, generator=g, dtype=F) * 2
    wq, wk = torch.randn(H * dim, generator=g), torch.randn(G * dim, generator=g)
    part = split_up(torch.cat([x, torch.zeros(T, -width % 16, dtype=F)], dim=1), 3, g)
    pos = torch.cat([torch.arange(n) + 5 for n in lens])
    rot = {"dims": R, "base": 50.0, "scaling": {"factor": 6.0, "original": 40, "fast": 4.0, "slow": 0.5}}
    f, mult = plain.frequencies(rot)
    eps = 1e-4
    q, k = x[:, :H * dim], x[:, H * dim:(H + G) * dim]
    q = plain.turned((q / plain.rms(q, eps) * wq.double()).view(T, H, dim), pos, rot)
    k = plain.turned((k / plain.rms(k, eps) * wk.double()).view(T, G, dim), pos, rot)
    v = x[:, (H + G) * dim:].view(T, G, vdim)
    for ring in (0, 64):
        pool = [torch.zeros(8, G, PAGE, pad, dtype=DTYPES[dtype], device=DEV) for _ in range(2)]
        table = i32([[5, 2], [3, 0]])
        out, _ = ops.projnorm_kv(part, H, G, dim, vdim, pad, DTYPES[dtype], dev(wq), dev(wk), eps, None, R, dev(f, torch.float32), False,
                                 i32(pos.tolist()), i32(seq_of(lens)), i32([n + 5 for n in lens]), pool[0], pool[1], table, ring, rot_mult=mult)
        out = out.view(T, H + 2 * G, pad).double().cpu()
        near(out[:, :H, :dim], q, dtype, "q")
        near(out[:, H:H + G, :dim], k, dtype, "k")
        near(out[:, H + G:, :vdim], v, dtype, "v")
        for t, (b, p) in enumerate(zip(seq_of(lens), pos.tolist())):
            if ring and p < lens[b] + 5 - ring:
                continue
            r = p % ring if ring else p
            page = int(table[b, r // PAGE])
            assert torch.equal(pool[0][page, :, r % PAGE].double().cpu(), out[t, H:H + G]) and \
                torch.equal(pool[1][page, :, r % PAGE].double().cpu(), out[t, H + G:])


SINK_SHAPES = [(3, 1, 12, 5), (4, 4, 64, 64), (8, 2, 64, 65), (2, 1, 128, 0), (12, 2, 128, 100), (6, 6, 48, 7), (9, 1, 64, 33)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H, G, D, window", SINK_SHAPES)
def test_one_added_to_the_softmax_denominator(H, G, D, window, dtype):
    """Scores far below zero (the one takes nearly all), around it and far above (it takes nothing), in prompts and over the
    cache: a sink of 0 for every head."""
    from trapetum_b200.csrc import ops
    g = torch.Generator().manual_seed(H + D)
    lens = [1, 130, 37]
    sink = torch.zeros(H, device=DEV)
    for shift in (-4.0, 0.0, 6.0):
        x = torch.randn(sum(lens), H + 2 * G, D, generator=g)
        x[:, :H, 0], x[:, H:H + G, 0] = 4.0, shift                        # a product that every score shares
        x = rounded(x, dtype)
        st = starts_of(lens)
        want = torch.cat([plain.attend(x[a:b, :H], x[a:b, H:H + G], x[a:b, H + G:], torch.arange(b - a), 0.3, window or None)
                          for a, b in zip(st, st[1:])])
        qkv = dev(x.reshape(sum(lens), -1), DTYPES[dtype])
        got = ops.attn_prefill_sink(qkv[:, :H * D], qkv[:, H * D:(H + G) * D], qkv[:, (H + G) * D:], i32(st), i32(seq_of(lens)), H, D, 0.3,
                                    sink, max(lens), lens, window, n_kv_heads=G).view(-1, H, D)
        near(got, want, dtype, f"prompt, scores around {1.2 * shift}", rel16=1.5e-2)
        # the last token of every sequence over pages in another order
        ring = (window + 63) // 64 * 64 if window else 0
        pools = [torch.full((8, G, PAGE, D), float("nan")) for _ in range(2)]
        table = [[6, 0, 0], [1, 7, 3], [2, 0, 0]]
        for b, n in enumerate(lens):
            for p in range(max(0, n - ring) if ring else 0, n):
                r = p % ring if ring else p
                for pool, lo in zip(pools, (H, H + G)):
                    pool[table[b][r // PAGE], :, r % PAGE] = x[st[b] + p, lo:lo + G].float()
        last = [s - 1 for s in st[1:]]
        got = ops.attn_decode(qkv[last, :H * D].contiguous(), dev(pools[0], DTYPES[dtype]), dev(pools[1], DTYPES[dtype]), i32(table), i32(lens),
                              H, G, D, 0.3, 0.0, window, ring, 512, sink=sink)
        near(got.view(-1, H, D), want[last], dtype, f"decoded, scores around {1.2 * shift}", rel16=1.5e-2)
    assert not ops.kernel_errors()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H, P, N, G, K, parts", [(4, 6, 16, 4, 5, 3), (6, 40, 48, 2, 4, 6), (1, 9, 3, 1, 1, 3), (8, 64, 128, 4, 2, 2)])
def test_state_space_mixer_between_its_products(H, P, N, G, K, parts, dtype):
    """Prompts that are one chunk and several, in slots out of order, then single tokens; a slot of nobody stays."""
    from trapetum_b200.csrc import ops
    g = torch.Generator().manual_seed(H + P + N)
    inner, ch = H * P, H * P + 2 * G * N
    lens, slots = [1, 290, 33], [4, 0, 2]
    m = {"heads": H, "vdim": P, "state": N, "groups": G, "conv": K, "norm_groups": parts}
    t = {"in": torch.eye(inner + ch + H), "o": torch.eye(inner), "conv": torch.randn(ch, K, generator=g) * 0.5,
         "conv.b": torch.randn(ch, generator=g) * 0.2, "dt_bias": torch.randn(H, generator=g) - 1, "A_log": torch.rand(H, generator=g) * 3 - 2.5,
         "D": torch.randn(H, generator=g), "norm": 1 + 0.2 * torch.randn(inner, generator=g)}
    d = {k: dev(v).float().contiguous() for k, v in t.items()}
    state = torch.zeros(6, ops.mamba2_state_size(H, P, N, G, K), device=DEV)
    state[1] = 7.0
    past = [{} for _ in lens]
    rnd = plain.to_bf16 if dtype == "bfloat16" else plain.same
    for step in range(4):
        n = lens if step == 0 else [1] * 3
        st = starts_of(n)
        rows = torch.randn(st[-1], inner + ch + H, generator=g)
        rows[:, :inner + ch] = rows[:, :inner + ch].to(DTYPES[dtype]).float()
        got = ops.mamba2(dev(rows[:, :inner + ch], DTYPES[dtype]), dev(rows[:, inner + ch:]).contiguous(), H, P, N, G, K, parts, d["conv"],
                         d["conv.b"], d["dt_bias"], d["A_log"], d["D"], d["norm"], 1e-4, state, i32(st), i32(seq_of(n)), i32(slots), 3, step > 0,
                         max_seq_len=0 if step else max(n))
        for b in range(3):
            want = plain.mamba2(rows[st[b]:st[b + 1]].double(), m, t, "", 1e-4, past[b], rnd)
            assert rel_l2(got[st[b]:st[b + 1]], want) <= (2e-5 if dtype == "float32" else 2e-2), (step, b)
    for b, s in enumerate(slots):
        S = state[s, :H * P * N].view(H, P, N).transpose(1, 2)
        assert rel_l2(S.reshape(1, -1), past[b]["S"].reshape(1, -1)) <= (2e-5 if dtype == "float32" else 2e-2)
    assert bool((state[1] == 7.0).all()) and bool((state[3] == 0).all()) and bool((state[5] == 0).all())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_exact_gelu_in_its_kernel_and_in_the_products_epilogue(dtype):
    """Where the tanh form differs by up to 5e-4, far out on both sides, and after a product of many tokens."""
    from trapetum_b200.csrc import ops
    g = torch.Generator().manual_seed(3)
    u = torch.cat([torch.linspace(-14, 14, 4001, dtype=F), torch.randn(999, generator=g, dtype=F)]).view(10, 500)
    part = split_up(u, 3, g)
    exact = part.double().cpu().sum(0)
    got = ops.unary_act(part, "gelu", DTYPES[dtype], 4, 490)
    want = plain.gelu(exact[:, 4:494])
    assert float((got.double().cpu() - want).abs().sub(want.abs() * (0 if dtype == "float32" else 2 ** -8)).max()) < 3e-6
    if dtype == "bfloat16":
        for T, N, K in ((129, 100, 64), (300, 384, 128), (600, 50, 72)):
            x, w = torch.randn(T, K, generator=g).to(torch.bfloat16), (torch.randn(N, K, generator=g) * 0.3).to(torch.bfloat16)
            want = plain.gelu(x.double() @ w.double().T)
            near(ops.gemm_tc(dev(x), dev(w), torch.float32, unary_act="gelu"), want, "float32", f"product of {T} x {N} x {K}", rel32=3e-6)
            near(ops.gemm_tc(dev(x), dev(w), torch.bfloat16, unary_act="gelu"), want, "bfloat16", f"product of {T} x {N} x {K}", rel16=4e-3)


@pytest.mark.parametrize("E, top", [(5, 2), (4, 4), (11, 1), (1, 1), (64, 6), (40, 33)])
def test_scores_as_weights(E, top):
    from trapetum_b200.csrc import ops
    g = torch.Generator().manual_seed(E * top)
    z = torch.randn(57, E + 3, generator=g, dtype=F) * 3
    z[0, :E] = -30.0 + torch.arange(E)      # scores close to nothing are not blown up by their sum; close to one they keep an order
    idx, wt, _ = ops.moe_route(split_up(z, 2, g), E, None, False, top, 1, 1, 1, 0.0, renormalize=False)
    wi, ww = plain.route(z[:, :E], torch.eye(E, dtype=F), top)
    assert torch.equal(idx.cpu().long(), wi)
    near(wt, ww, "float32", "weights")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T, W, E, ff, top", [(1, 50, 3, 11, 1), (21, 72, 5, 24, 2), (150, 72, 5, 24, 2), (333, 128, 16, 200, 3), (70, 40, 3, 8, 3),
                                              (400, 128, 6, 48, 3), (700, 256, 5, 256, 2), (1100, 64, 7, 32, 1)])
def test_experts_whose_weights_multiply_what_they_read(T, W, E, ff, top, dtype):
    """One by one, grouped on mma.sync and on tcgen05 (tiles that are not full, experts that nobody chose), with weights
    beyond one; weights on the output of the same experts give something else."""
    from trapetum_b200.csrc import ops
    dt = DTYPES[dtype]
    g = torch.Generator().manual_seed(8)
    x = torch.randn(T, W, generator=g).to(dt)
    gw, uw, dw = (torch.randn(E, a, b, generator=g).to(dt) / 5 for a, b in ((ff, W), (ff, W), (W, ff)))
    idx = torch.stack([torch.randperm(max(1, E - 1) if top < E else E, generator=g)[:top] for _ in range(T)]).int()
    wt = 0.05 + 1.5 * torch.rand(T, top, generator=g)
    gu = None
    if dtype == "bfloat16" and ff % 16 == 0:
        gu = torch.stack([ops.interleave_gate_up(dev(gw[e]), dev(uw[e])) for e in range(E)]).contiguous()
    out = ops.moe_experts(dev(x), dev(gw), dev(uw), dev(dw), dev(idx), dev(wt), gate_up_w=gu, weight_on="input")
    other = ops.moe_experts(dev(x), dev(gw), dev(uw), dev(dw), dev(idx), dev(wt), gate_up_w=gu)
    rnd = plain.to_bf16 if dtype == "bfloat16" else plain.same
    t = {f"e{e}.{k}": m[e] for e in range(E) for k, m in (("gate", gw), ("up", uw), ("down", dw))}
    want = torch.zeros(T, W, dtype=F)
    for n in range(T):
        for j in range(top):
            want[n] += plain.expert(wt[n, j].double() * x[n:n + 1].double(), t, f"e{int(idx[n, j])}.", rnd)[0]
    near(out, want, dtype, "experts", rel16=1e-2)
    assert T < 20 or rel_l2(other, want) > 0.1             # (one token's weight may lie near one)


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
def test_the_residual_stream_after_every_layer_call(folders, oracles, name, monkeypatch):
    from trapetum_b200.parts.block import SandwichBlock
    cfg, w = oracles[name]
    ids = prompts(cfg["vocab"], [75], seed=2)[0]
    seq = plain.Sequence(cfg, w)
    seq.feed(ids)
    seen, orig = [], SandwichBlock.forward

    def spy(self, stream, ctx, cache):
        orig(self, stream, ctx, cache)
        seen.append(stream.value().clone())
    monkeypatch.setattr(SandwichBlock, "forward", spy)
    eng = tb.Engine(model_of(folders, name, "float32"), max_tokens=256)
    eng.step(eng.start(1), [ids], [[0]])
    assert len(seen) == len(seq.streams) == len(plain.calls(cfg))
    for r, (x, (layer, _)) in enumerate(zip(seen, plain.calls(cfg))):
        near(x, seq.streams[r], "float32", f"{name}: the stream after call {r} (layer {layer}, {cfg['layers'][layer]['type']})", rel32=2e-5)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name, first", [("A", 1), ("A", 2), ("B", 63), ("B", 64), ("B", 7), ("C", 65), ("C", 3)])
def test_prompt_then_token_by_token(folders, oracles, name, first, dtype):
    """Decoding runs across pages' borders (64, 128, 192), over every window's edge (windows of 3 to 100 pass over decoded
    tokens, and the rows of their rings are used again), from first tokens fewer than a convolution's taps, and through the
    capture of the step's graph."""
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
    """More tokens in a step than the split products take, and experts grouped in a decode step."""
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


def _needle(tmp_path, kind, size, key_pos, n, probe, least):
    """A one-layer model without feed-forward whose scores are sharpened (or whose state decays slowly), and a prompt of one
    repeated token with a single other token at ``key_pos``, chosen (with the plain implementation) as the one that the query
    at ``probe`` singles out most."""
    layer = attention(2, 1, 16, 24, 0.25, size=size, rot=(8, 10000.0), scaling=(2.0, 512, 8.0, 1.0)) if kind == "attention" \
        else mamba2(2, 16, 16, groups=2, conv=3)
    cfg = config(50, 32, [(layer, None)])
    w = random_weights(cfg, 5, sharp=8.0)
    if kind == "mamba2":
        w["l0.mix.A_log"] = torch.tensor([-7.0, -8.0]).to(torch.bfloat16)
        w["l0.mix.dt_bias"] = torch.tensor([-3.0, -4.0]).to(torch.bfloat16)
        w["l0.mix.in"][-2:] *= 6.0                                # a step size that hangs on the token
    wd = doubles(w)
    few = 3
    if kind == "mamba2":                                          # the repeated token is the one that writes least into the state
        few = int((plain.named_norm(wd["embed"], wd, "l0.norm1") @ wd["l0.mix.in"][-2:].T).max(-1).values.argmin())
    base = [few] * n
    without = plain.forward(cfg, wd, base)[probe:probe + 1]
    best, ids = -1.0, None
    for cand in set(range(30)) - {few}:
        trial = list(base)
        trial[key_pos] = cand
        e = float(position_errors(plain.forward(cfg, wd, trial)[probe:probe + 1], without))
        if e > best:
            best, ids = e, trial
    assert best > least, best
    folder = write_folder(str(tmp_path / f"needle_{kind}_{size}_{key_pos}_{n}"), cfg, w)
    return cfg, wd, base, ids, folder


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key_pos, n", [(0, 200), (63, 130), (64, 130), (5, 700)])
def test_a_far_key_is_found_in_prompts_and_in_decoding(tmp_path, key_pos, n, dtype):
    """No mask: every earlier token is seen, also the first one and those at a page's edge, hundreds of tokens back."""
    cfg, w, base, ids, folder = _needle(tmp_path, "attention", None, key_pos, n, n - 1, 0.05)
    truth = plain.forward(cfg, w, ids)
    tol = tolerance(("far", key_pos, n), cfg, w, ids, dtype)
    eng = tb.Engine(tb.load_model(folder, dtype, DEV), max_tokens=1024)
    s = eng.start(1)
    close(eng.step(s, [ids], [[n - 1]]), truth[-1:], tol[-1:], f"needle at {key_pos} of {n}, prompt", dtype)
    eng.release(s)
    s = eng.start(1)
    eng.step(s, [ids[:n - 3]], [[]])
    got = torch.cat([eng.step(s, [[t]], [[0]]).clone() for t in ids[n - 3:]])
    close(got, truth[-3:], tol[-3:], f"needle at {key_pos} of {n}, decoded", dtype)
    eng.check_kernels()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("size, key_pos", [(48, 1), (48, 30), (64, 0), (64, 63), (64, 70), (65, 63), (65, 64), (130, 2), (2, 77), (1, 50), (100, 127)])
def test_a_key_at_a_windows_edge_in_prompts_and_in_decoding(tmp_path, size, key_pos, dtype):
    """The key is seen by the queries up to ``size - 1`` behind it and by none after them: the logits of the last query that
    sees it and of the first that does not, in a prompt and decoded."""
    last = key_pos + size - 1
    n = last + 3
    cfg, w, base, ids, folder = _needle(tmp_path, "attention", size, key_pos, n, last, 0.05)
    truth = plain.forward(cfg, w, ids)
    blind = plain.forward(cfg, w, base)
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
@pytest.mark.parametrize("key_pos, n, first", [(0, 150, 1), (63, 150, 64), (127, 400, 128), (0, 600, 599), (130, 600, 600)])
def test_an_old_token_stays_in_the_state(tmp_path, key_pos, n, first, dtype):
    """Slow decays: the first token and those at the edges of a chunk still show in the last logits, whether they were read
    in the prompt (one chunk or several) or decoded."""
    cfg, w, base, ids, folder = _needle(tmp_path, "mamba2", None, key_pos, n, n - 1, 0.05)
    truth = plain.forward(cfg, w, ids)
    blind = plain.forward(cfg, w, base)
    eng = tb.Engine(tb.load_model(folder, dtype, DEV), max_tokens=1024)
    s = eng.start(1)
    got = [eng.step(s, [ids[:first]], [list(range(first))])] + [eng.step(s, [[t]], [[0]]).clone() for t in ids[first:]]
    eng.release(s)
    got = torch.cat(got)
    close(got, truth, tolerance(("old", key_pos, n), cfg, w, ids, dtype), f"token {key_pos} of {n} in the state, {first} first", dtype)
    # and it is this token that shows: the engine follows the truth more closely than the prompt without it
    if dtype == "float32":
        assert float(position_errors(got[-1:], truth[-1:])) < 0.05 * float(position_errors(blind[-1:], truth[-1:]))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_what_the_design_adds_would_show(tmp_path, dtype, monkeypatch):
    """The engine follows the plain implementation; the plain implementation with a mistake planted in it (no one in the
    softmax denominator, no factor on the rotation or no blend, norms without their number or shift, another activation,
    weights renormalised or on the experts' outputs, a pass fewer or its product with the two halves exchanged) is far
    away."""
    cfg = config(60, 48, [(attention(2, 2, 8, 12, 0.4, size=9, rot=(8, 100.0), scaling=(4.0, 32, 4.0, 0.5)), moe(4, 2, 24)),
                          (mamba2(2, 12, 8, groups=1, conv=3, norm_groups=2), dense(32)),
                          (attention(2, 1, 8, 12, 0.4, size=6), moe(3, 1, 24))], loop=(0, 2, 2))
    w = random_weights(cfg, 9)
    wd = doubles(w)
    ids = prompts(60, [40], seed=3)[0]
    truth = plain.forward(cfg, wd, ids)

    def far(what, least=0.03, weights=None, **planted):
        with monkeypatch.context() as m:
            for name, f in planted.items():
                m.setattr(plain, name, f)
            e = float(position_errors(plain.forward(cfg, weights or wd, ids), truth).median())
        assert e > least, (what, e)
    with monkeypatch.context() as m:
        m.setattr(plain, "weights", lambda s, ok: torch.softmax(s.masked_fill(~ok, float("-inf")), -1))
        assert float(position_errors(plain.forward(cfg, wd, ids), truth).median()) > 0.03, "no one in the denominator"
    freq = plain.frequencies
    far("no factor on the rotation", frequencies=lambda rot: (freq(rot)[0], 1.0), least=0.01)
    far("no blend", frequencies=lambda rot: (freq({k: v for k, v in rot.items() if k != "scaling"})[0], freq(rot)[1]), least=0.01)
    far("norms without their number", dyt=lambda x, a, k, b: torch.tanh(x) * k + b)
    far("norms without their shift", dyt=lambda x, a, k, b: torch.tanh(a * x) * k)
    far("silu in the dense feed-forward", gelu=plain.silu)
    far("weights on the outputs", routed=_weights_on_outputs)
    far("renormalised weights", route=_renormalised)
    far("one expert fewer", route=lambda h, r, top: tuple(x[:, :max(1, top - 1)] for x in _route(h, r, top)))
    swapped = dict(wd)
    swapped["loop.in"] = torch.cat([wd["loop.in"][:, 48:], wd["loop.in"][:, :48]], dim=1)
    far("the halves of the pass's product exchanged", weights=swapped)
    once = dict(cfg, loop=dict(cfg["loop"], times=1))
    assert float(position_errors(plain.forward(once, wd, ids), truth).median()) > 0.03
    eng = tb.Engine(tb.load_model(write_folder(str(tmp_path / "adds"), cfg, w), dtype, DEV), max_tokens=256)
    s = eng.start(1)
    got = [eng.step(s, [ids[:30]], [list(range(30))])] + [eng.step(s, [[t]], [[0]]).clone() for t in ids[30:]]
    close(torch.cat(got), truth, tolerance("adds", cfg, wd, ids, dtype), "everything together: prompt then decoding", dtype)




def _renormalised(h, router, top):
    idx, s = _route(h, router, top)
    return idx, s / s.sum(-1, keepdim=True)


def _weights_on_outputs(h, ml, t, p, rnd=plain.same):
    idx, s = _route(h, t[p + "router"].double(), ml["router"]["top"])
    y = torch.zeros_like(h)
    for n in range(h.shape[0]):
        for e, x in zip(idx[n].tolist(), s[n]):
            y[n] += x * plain.expert(h[n][None], t, f"{p}e{e}.", rnd)[0]
    return y


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_first_tokens_of_a_sequence(folders, oracles, dtype):
    """Where a convolution reads zeros, the state is empty, a softmax has one key beside its one, and a window is not full:
    prompts of 1 to 6 tokens side by side, each then decoded for a few."""
    for name, (cfg, w) in oracles.items():
        full = prompts(cfg["vocab"], [9] * 6, seed=41)
        eng = tb.Engine(model_of(folders, name, dtype), max_tokens=512)
        s = eng.start(6)
        out = eng.step(s, [f[:i + 1] for i, f in enumerate(full)], [list(range(i + 1)) for i in range(6)])
        got, at = [], 0
        for i in range(6):
            got.append([out[at:at + i + 1].clone()])
            at += i + 1
        for j in range(3):
            out = eng.step(s, [[f[i + 1 + j]] for i, f in enumerate(full)], [[0]] * 6)
            for i in range(6):
                got[i].append(out[i:i + 1].clone())
        eng.release(s)
        for i, f in enumerate(full):
            ids = f[:i + 4]
            close(torch.cat(got[i]), plain.forward(cfg, w, ids), tolerance(name + "first", cfg, w, ids, dtype), f"{name}: the first {i + 4} tokens", dtype)


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
