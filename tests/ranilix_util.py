"""Shared pieces of the Ranilix tests: small configurations made up here, model folders with random weights drawn
here (not by the library), and tolerances taken from the plain implementation alone."""
import math

import torch

import plain_ranilix as plain
from lofirax_util import position_errors, prompts, worst_ratio, write_folder  # noqa: F401  (the tests import them from here)


def attention(heads, kv_heads, dim, vdim, scale, size=None, rot=None, v_mix=False):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix}
    if size:
        m["mask"] = {"size": size}
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    return "attention", m


def parallel(left, right, left_scale=1.0, right_scale=1.0):
    """``left`` (heads, kv_heads, dim, vdim, scale, rot), ``right`` (dim, vdim, rot, decays)."""
    h, g, d, v, s, r = left
    lm = {"heads": h, "kv_heads": g, "dim": d, "vdim": v, "scale": s}
    rd, rv, rr, decay = right
    rm = {"heads": len(decay), "dim": rd, "vdim": rv, "decay": list(decay)}
    if r:
        lm["rot"] = {"dims": r[0], "base": r[1]}
    if rr:
        rm["rot"] = {"dims": rr[0], "base": rr[1]}
    return "parallel", {"left": lm, "right": rm, "left_scale": left_scale, "right_scale": right_scale}


def config(vocab, width, layers, eps=1e-5, scale=None):
    """``layers``: (mixer, inner width of the feed-forward or None)."""
    cfg = {"architecture": "Ranilix", "vocab": vocab, "width": width, "norm": {"eps": eps},
           "layers": [{"type": t, "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}} for (t, m), ff in layers]}
    if scale is not None:
        cfg["embedding"] = {"scale": scale}
    return cfg


# A: small and odd-shaped.  A window of 5 and one of 33; fewer kv heads than heads; values wider and narrower than keys;
#    a quarter, half and all of a head rotated, two dims, nothing; a layer without feed-forward; the first layer mixes no
#    values, the first mixing layer comes later; decays from slow to fast, one of them 1.
CFG_A = config(150, 48, [
    (attention(3, 1, 8, 12, 0.5, size=5, rot=(4, 100.0)), 40),
    (parallel((4, 2, 8, 12, 0.4, (2, 50.0)), (12, 10, (6, 200.0), (0.5, 0.9, 0.99)), 0.6, 1.3), 24),
    (attention(4, 2, 12, 8, 0.4, size=33, rot=(12, 1000.0), v_mix=True), None),
    (attention(2, 2, 8, 8, 0.6, size=70, rot=(2, 30.0), v_mix=True), 56),
    (parallel((3, 3, 10, 6, 0.5, None), (6, 14, None, (1.0, 0.75)), 1.1, -0.4), 24),
    (attention(6, 2, 8, 8, 0.45, v_mix=True), 24),
], eps=1e-5, scale=3.0)
# B: sizes that the tensor-core kernels take in bfloat16 (heads of 64 and 128, retention with channels of 64 and 128 and
#    values of 64 to 160); windows of 64 (a page) and 65; one kv head; the parallel layer first.
CFG_B = config(512, 128, [
    (parallel((4, 2, 64, 64, 0.125, (32, 10000.0)), (64, 96, (64, 5000.0), (0.9, 0.95, 0.98, 0.995)), 0.9, 0.7), 256),
    (attention(4, 4, 64, 64, 0.15, size=64, rot=(64, 10000.0), v_mix=True), 256),
    (attention(8, 4, 48, 64, 0.2, size=65, rot=(16, 500.0), v_mix=True), 192),
    (parallel((2, 1, 128, 96, 0.09, (128, 250000.0)), (128, 160, (32, 10000.0), (0.97, 0.999)), 1.2, 0.5), None),
    (attention(2, 1, 128, 128, 0.1, size=100, rot=(64, 10000.0)), 256),
], eps=1e-6, scale=1.5)
# C: sizes that fit no fast path and no vector load (a width of 50, a vocabulary of 77, heads of 6 and 10, values of 7);
#    one head; no embedding scale; no layer mixes values.
CFG_C = config(77, 50, [
    (attention(3, 3, 6, 7, 0.7, size=3, rot=(2, 20.0)), 30),
    (parallel((1, 1, 10, 7, 0.5, (10, 40.0)), (10, 7, (2, 15.0), (0.93,)), 0.8, 0.9), 22),
    (attention(1, 1, 10, 9, 0.5, rot=(6, 200.0)), None),
], eps=1e-3)

CONFIGS = {"A": CFG_A, "B": CFG_B, "C": CFG_C}


def random_weights(cfg: dict, seed: int, sharp: float = 2.0) -> dict:
    """bfloat16 weights, drawn here: matrices N(0, 1/fan_in) (those of q and k of the attention without head norms
    ``sharp`` times larger, and head norm weights around ``sharp``, so that the scores single keys out), norm gains near 1,
    sinks around 1, mixing numbers between 0.2 and 0.8."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]
    out = {}

    def mat(o, i, scale=1.0):
        return torch.randn(o, i, generator=g) * (scale / math.sqrt(i))

    def small(n, s=0.2):
        return s * torch.randn(n, generator=g)
    out["embed"] = torch.randn(V, W, generator=g)
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        out[p + "norm1"] = 1.0 + small(W)
        if L["type"] == "attention":
            H, G, D, Vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            out[p + "mix.q"], out[p + "mix.k"], out[p + "mix.v"] = mat(H * D, W), mat(G * D, W), mat(G * Vd, W, 1.5)
            out[p + "mix.q.b"], out[p + "mix.k.b"], out[p + "mix.v.b"] = small(H * D, 0.5), small(G * D, 0.5), small(G * Vd, 0.5)
            out[p + "mix.q.norm"], out[p + "mix.k.norm"] = sharp * (1.0 + small(D)), 1.0 + small(D)
            if m["v_mix"]:
                out[p + "mix.vmix"] = 0.2 + 0.6 * torch.rand((), generator=g)
            out[p + "mix.sink"] = 1.0 + torch.randn(H, generator=g)
            out[p + "mix.g"] = mat(H * Vd, W, 2.0)
            out[p + "mix.o"] = mat(W, H * Vd, 2.0)
        else:
            l, r = m["left"], m["right"]
            H, G, D, Vd = l["heads"], l["kv_heads"], l["dim"], l["vdim"]
            q = p + "mix.left."
            out[q + "q"], out[q + "k"], out[q + "v"] = mat(H * D, W, sharp), mat(G * D, W, sharp), mat(G * Vd, W, 1.5)
            out[q + "o"] = mat(W, H * Vd, 1.5)
            H, D, Vd = r["heads"], r["dim"], r["vdim"]
            q = p + "mix.right."
            out[q + "q"], out[q + "k"], out[q + "v"] = mat(H * D, W, 1.5), mat(H * D, W, 1.5), mat(H * Vd, W, 1.5)
            out[q + "g"], out[q + "o"] = mat(H * Vd, W, 2.0), mat(W, H * Vd, 1.5)
        if L["mlp"] is not None:
            ff = L["mlp"]["ff"]
            out[p + "norm2"] = 1.0 + small(W)
            out[p + "mlp.up"], out[p + "mlp.down"] = mat(ff, W, 1.5), mat(W, ff)
    out["final.norm"] = 1.0 + small(W)
    out["head"] = mat(V, W)
    return {k: v.to(torch.bfloat16).contiguous() for k, v in out.items()}


def doubles(w: dict) -> dict:
    return {k: v.double() for k, v in w.items()}


TOL32 = 3e-5
BF16_FLOOR, BF16_FACTOR = 2e-2, 3.0
_BUDGET = {}


def tolerance(key, cfg, w, ids, dtype: str) -> torch.Tensor:
    """One tolerance per position.  float32: rounding only.  bfloat16: the larger of 2e-2 and three times what the plain
    implementation itself loses at that position when it rounds what a 16-bit engine stores (never taken from the
    library's output)."""
    if dtype == "float32":
        return torch.full((len(ids),), TOL32, dtype=torch.float64)
    k = (key, tuple(ids))
    if k not in _BUDGET:
        lost = position_errors(plain.forward(cfg, w, ids, rnd=plain.to_bf16), plain.forward(cfg, w, ids))
        _BUDGET[k] = torch.clamp(BF16_FACTOR * lost, min=max(BF16_FLOOR, float(lost.median()) * BF16_FACTOR))
    return _BUDGET[k]
