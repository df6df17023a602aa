"""Shared pieces of the Sezanex tests: small configurations made up here, model folders with random weights drawn
here (not by the library), and tolerances taken from the plain implementation alone."""
import math

import torch

import plain_sezanex as plain
from lofirax_util import position_errors, prompts, worst_ratio, write_folder  # noqa: F401  (the tests import them from here)


def attention(heads, kv_heads, dim, vdim, scale, size=None, rot=None, scaling=None):
    """``rot`` (dims, base), ``scaling`` (factor, original, fast, slow)."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if size:
        m["mask"] = {"size": size}
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
        if scaling:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return "attention", m


def mamba2(heads, vdim, state, groups=1, conv=4, norm_groups=1):
    return "mamba2", {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def config(vocab, width, layers, loop=None, eps=1e-5):
    """``layers``: (mixer, feed-forward or None); ``loop`` (start, stop, times)."""
    cfg = {"architecture": "Sezanex", "vocab": vocab, "width": width, "norm": {"eps": eps},
           "layers": [{"type": t, "mixer": m, "mlp": f} for (t, m), f in layers]}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


# A: small and odd-shaped.  Two layers in the middle run three times; windows of 5 and 33; one and two kv heads; values wider
#    and narrower than keys; a third of a head and whole heads rotated, with blends whose ramp lies inside; experts of which
#    two of five and all four are chosen; as many groups as state-space heads; 3 and 5 taps; a layer without feed-forward.
CFG_A = config(150, 48, [
    (attention(3, 1, 12, 16, 0.5, size=5, rot=(4, 100.0), scaling=(4.0, 64, 4.0, 0.5)), moe(5, 2, 24)),
    (mamba2(3, 8, 10, groups=1, conv=3, norm_groups=1), dense(40)),
    (mamba2(4, 15, 16, groups=4, conv=5, norm_groups=3), None),
    (attention(4, 2, 12, 8, 0.4, size=33, rot=(12, 1000.0), scaling=(3.0, 128, 8.0, 1.0)), moe(4, 4, 20)),
], loop=(1, 3, 3))
# B: sizes that the tensor-core kernels take in bfloat16; the whole model runs twice; windows of 64 (a page) and 100; keys of
#    48 with values of 96; a blend and a plain rotation; one expert of four and two of eight.
CFG_B = config(384, 128, [
    (mamba2(4, 32, 64, groups=2, conv=4, norm_groups=4), moe(8, 2, 64)),
    (attention(8, 2, 64, 64, 0.15, size=64, rot=(64, 10000.0), scaling=(2.5, 1024, 32.0, 1.0)), dense(256)),
    (attention(4, 4, 48, 96, 0.15, size=100, rot=(16, 500.0)), moe(4, 1, 32)),
    (mamba2(2, 64, 128, groups=1, conv=4, norm_groups=2), dense(192)),
], loop=(0, 4, 2), eps=1e-6)
# C: sizes that fit no fast path and no vector load (a width of 50, a vocabulary of 77, heads of 6 and 10, values of 7, experts
#    of 11 and 14); no repeated span; an attention without window and rotation; a convolution of one tap.
CFG_C = config(77, 50, [
    (attention(3, 3, 6, 7, 0.7, size=3, rot=(2, 20.0), scaling=(8.0, 16, 4.0, 0.5)), moe(3, 1, 14)),
    (mamba2(2, 5, 7, groups=2, conv=2, norm_groups=1), moe(5, 3, 11)),
    (attention(1, 1, 10, 9, 0.6), dense(30)),
    (mamba2(1, 21, 3, groups=1, conv=1, norm_groups=3), None),
], eps=1e-3)

CONFIGS = {"A": CFG_A, "B": CFG_B, "C": CFG_C}


def random_weights(cfg: dict, seed: int, sharp: float = 2.0) -> dict:
    """bfloat16 weights, drawn here: matrices N(0, 1/fan_in), q norm weights around ``sharp`` (so that the scores single keys
    out), the other gains around 1, every norm with a number and a shift of its own.

    Which experts win must not hang on a rounding, or a 16-bit run could not be compared at all.  So the first columns of
    the stream carry a code of the token, one number per expert, all numbers of a token far apart; the norms after the
    sublayers hardly touch these columns, the product at the start of a pass hands them on, and the router reads little
    else.  Two more columns, one that varies from token to token and one that does not, place the scores around a half."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]
    C = max([L["mlp"]["router"]["experts"] for L in cfg["layers"] if (L["mlp"] or {}).get("kind") == "moe"], default=0)
    coded = slice(0, C + 2 if C else 0)
    out = {}

    def mat(o, i, scale=1.0):
        return torch.randn(o, i, generator=g) * (scale / math.sqrt(i))

    def gain(n, s=0.2):
        return 1.0 + s * torch.randn(n, generator=g)

    def small(n, s=0.2):
        return s * torch.randn(n, generator=g)

    def norm(name, after=False):
        w, b = gain(W), small(W)
        alpha = 0.4 + 0.5 * torch.rand((), generator=g)
        if after:
            w[coded], b[coded] = small(C + 2 if C else 0, 0.004), 0.0
        elif name.endswith("norm2"):
            w[coded], b[coded], alpha = gain(C + 2 if C else 0, 0.02), 0.0, 0.7 + 0.05 * torch.rand((), generator=g)
        out[name], out[name + ".b"], out[name + ".alpha"] = w, b, alpha

    E = torch.randn(V, W, generator=g)
    if C:
        levels = torch.atanh(0.8 - 0.1 * torch.arange(C)) / 0.72          # evenly spaced behind the norm's tanh
        E[:, :C] = torch.stack([levels[torch.randperm(C, generator=g)] for _ in range(V)])
        E[:, C], E[:, C + 1] = 3.0 * torch.rand(V, generator=g) - 1.5, 1.5
    out["embed"] = E
    if cfg.get("loop"):
        L = mat(W, 2 * W)
        L[coded] = 0.0
        L[coded, coded] = torch.eye(C + 2 if C else 0)
        out["loop.in"] = L
    for i, L in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", L["mixer"], L["mlp"]
        norm(p + "norm1")
        norm(p + "norm1b", after=True)
        if L["type"] == "attention":
            H, G, D, Vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            out[p + "mix.q"], out[p + "mix.k"], out[p + "mix.v"] = mat(H * D, W), mat(G * D, W), mat(G * Vd, W, 1.5)
            out[p + "mix.q.norm"], out[p + "mix.k.norm"] = sharp * gain(H * D), gain(G * D)
            out[p + "mix.o"] = mat(W, H * Vd, 2.0)
        else:
            H, P, N, G, K = m["heads"], m["vdim"], m["state"], m["groups"], m["conv"]
            inner = H * P
            ch = inner + 2 * G * N
            out[p + "mix.in"] = mat(inner + ch + H, W, 1.5)
            out[p + "mix.conv"], out[p + "mix.conv.b"] = 0.6 * torch.randn(ch, K, generator=g), small(ch)
            out[p + "mix.dt_bias"], out[p + "mix.A_log"] = torch.randn(H, generator=g) - 1.5, torch.rand(H, generator=g) * 3 - 2.5
            out[p + "mix.D"], out[p + "mix.norm"] = gain(H), gain(inner)
            out[p + "mix.o"] = mat(W, inner)
        if f is None:
            if i % 2 == 0:                           # a file may carry the norms that nothing follows
                norm(p + "norm2")
                norm(p + "norm2b", after=True)
            continue
        norm(p + "norm2")
        norm(p + "norm2b", after=True)
        if f["kind"] == "dense":
            out[p + "mlp.up"], out[p + "mlp.down"] = mat(f["ff"], W, 1.5), mat(W, f["ff"], 1.5)
        else:
            n, ff = f["router"]["experts"], f["expert"]["ff"]
            R = mat(n, W, 0.1)
            R[:, coded] = 0.0
            R[:, :n] = 14.0 * torch.eye(n)
            R[:, C], R[:, C + 1] = 2.0, -14.0
            out[p + "mlp.router"] = R
            for e in range(n):
                q = f"{p}mlp.e{e}."
                out[q + "gate"], out[q + "up"], out[q + "down"] = mat(ff, W, 2.0), mat(ff, W, 2.0), mat(W, ff, 1.5)
    norm("final.norm")
    return {k: v.to(torch.bfloat16).contiguous() for k, v in out.items()}


def doubles(w: dict) -> dict:
    return {k: v.double() for k, v in w.items()}


TOL32 = 3e-5
BF16_FLOOR, BF16_FACTOR = 2e-2, 3.0
_BUDGET = {}


def _dithered(seed: int):
    """Rounding to bfloat16 with other errors than :func:`plain.to_bf16`'s, of their size: numbers pushed by up to half a
    rounding step first."""
    g = torch.Generator().manual_seed(seed)

    def rnd(x):
        return plain.to_bf16(x * (1.0 + 2.0 ** -9 * (2.0 * torch.rand(x.shape, generator=g, dtype=plain.F) - 1.0)))
    return rnd


def tolerance(key, cfg, w, ids, dtype: str) -> torch.Tensor:
    """One tolerance per position.  float32: rounding only.  bfloat16: the larger of 2e-2 and three times what the plain
    implementation itself loses at that position when it rounds what a 16-bit engine stores, the larger of two ways to
    round (never taken from the library's output)."""
    if dtype == "float32":
        return torch.full((len(ids),), TOL32, dtype=torch.float64)
    k = (key, tuple(ids))
    if k not in _BUDGET:
        truth = plain.forward(cfg, w, ids)
        lost = torch.maximum(*(position_errors(plain.forward(cfg, w, ids, rnd=r), truth) for r in (plain.to_bf16, _dithered(1))))
        _BUDGET[k] = torch.clamp(BF16_FACTOR * lost, min=max(BF16_FLOOR, float(lost.median()) * BF16_FACTOR))
    return _BUDGET[k]
