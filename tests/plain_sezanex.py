"""Sezanex, stated plainly: one slow function per mechanism, in 64-bit floats on the CPU.

This file is the tests' oracle.  It shares no code with the library: it reads a configuration dictionary (the
keys of config.json) and a dictionary of tensors by name, and keeps, per layer call, what the tokens it has seen
left behind (keys and values, a recurrent state, the convolution's last inputs), so that a sequence can be fed in
pieces.

Notation: ``W`` is the model's width, ``h`` a sublayer's input [tokens, W], matrices are stored [out, in].

    stream      x0 = E[token];   logits = E n(x_last)
    layer       x <- x + n1b(mix(n1(x)));  x <- x + n2b(ff(n2(x)));   n(x) = tanh(alpha x) w + b, alpha one number
    pass        a span of layers runs several times; before its first layer, each time: x <- L [x; x0]
    attention   q, k: u / rms(u) * w over the whole projection;  pairs (i, i + R/2) of the first R dims of a head turned
                by pos * f_i, lengthened by a factor m (f and m blended per frequency);  s_ij = scale q_i.k_j for
                0 <= i - j < window;  p = exp(s) / (1 + sum exp(s));  o_h = sum p v;  Wo o
    mamba2      [z | x B C | dt] = Wi h;  (x B C) <- silu(conv + b);  dt <- softplus(dt + c);
                S <- exp(-exp(A) dt) S + dt B x^T;  y = S^T C + D x;  y silu(z), each of the norm's parts / rms * w;  Wo y
    dense ff    Wd g(Wu h), g(z) = z Phi(z)
    routed ff   s = sigmoid(R h);  the top largest win;  sum over the winners of expert_e(s_e h),
                expert(u) = Wd (silu(Wg u) * (Wu u))
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F = torch.float64


def f64(t: torch.Tensor) -> torch.Tensor:
    return t.to(F)


def same(x):
    return x


def to_bf16(x: torch.Tensor) -> torch.Tensor:
    """What a 16-bit engine stores: the value rounded to bfloat16 (used only to size the tests' tolerances)."""
    return x.to(torch.bfloat16).to(F)


def rms(x, eps):
    return torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def dyt(x, alpha, w, b):
    return torch.tanh(alpha * x) * w + b


def named_norm(x, t, name):
    return dyt(x, f64(t[name + ".alpha"]), f64(t[name]), f64(t[name + ".b"]))


def silu(z):
    return z * torch.sigmoid(z)


def gelu(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


# ---------------------------------------------------------------------------
# positions
# ---------------------------------------------------------------------------

def frequencies(rot: dict):
    """(frequencies [dims / 2], the factor on cos and sin)."""
    R, base, sc = rot["dims"], float(rot["base"]), rot.get("scaling")
    out = []
    for i in range(R // 2):
        f = base ** (-2.0 * i / R)
        if sc:
            def turns_at(turns):
                return R * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
            lo = max(math.floor(turns_at(sc["fast"])), 0)
            hi = min(math.ceil(turns_at(sc["slow"])), R - 1)
            r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            f = f / sc["factor"] * r + f * (1.0 - r)
        out.append(f)
    return torch.tensor(out, dtype=F), (0.1 * math.log(sc["factor"]) + 1.0) if sc else 1.0


def turned(x, pos, rot: Optional[dict]):
    """x [tokens, heads, D] with the pairs (i, i + R/2) of the first R dims turned."""
    if not rot or not rot["dims"]:
        return x
    out, half = x.clone(), rot["dims"] // 2
    f, mult = frequencies(rot)
    for i in range(half):
        a = pos.to(F) * f[i]
        c, s = (mult * torch.cos(a))[:, None], (mult * torch.sin(a))[:, None]
        u, v = x[..., i], x[..., i + half]
        out[..., i], out[..., i + half] = u * c - v * s, v * c + u * s
    return out


# ---------------------------------------------------------------------------
# attention
# ---------------------------------------------------------------------------

def seen(qpos, kpos, window: Optional[int]):
    """[queries, keys]: key j is seen from query i iff 0 <= i - j (< window)."""
    d = qpos[:, None] - kpos[None, :]
    return (d >= 0) & (d < window) if window else d >= 0


def weights(s, ok):
    """exp(s) / (1 + sum of exp over the seen keys), row by row."""
    s = s.masked_fill(~ok, -math.inf)
    top = torch.clamp(s.max(-1, keepdim=True).values, min=0.0)
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(-top))


def attend(q, k, v, qpos, scale, window=None, rnd=same):
    """q [T, H, D] at positions ``qpos``, k [n, G, D] and v [n, G, V] at positions 0..n-1 -> [T, H, V].
    ``rnd``: tensor-core kernels round the weights that meet the values."""
    H, G = q.shape[1], k.shape[1]
    ok = seen(qpos, torch.arange(k.shape[0]), window)
    out = []
    for h in range(H):
        g = h // (H // G)
        out.append(rnd(weights((q[:, h] @ k[:, g].T) * scale, ok)) @ v[:, g])
    return torch.stack(out, dim=1)


def appended(past, key, x):
    """``x`` behind what ``past`` holds under ``key``; the whole is kept there."""
    if past is None:
        return x
    past[key] = torch.cat([past[key], x]) if key in past else x
    return past[key]


def attention(h, m, t, p, eps, first_pos=0, past=None, rnd=same):
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    pos = torch.arange(first_pos, first_pos + T)
    q, k = h @ f64(t[p + "q"]).T, h @ f64(t[p + "k"]).T
    v = (h @ f64(t[p + "v"]).T).view(T, G, V)
    q = turned((q / rms(q, eps) * f64(t[p + "q.norm"])).view(T, H, D), pos, m.get("rot"))
    k = turned((k / rms(k, eps) * f64(t[p + "k.norm"])).view(T, G, D), pos, m.get("rot"))
    k, v = appended(past, "k", rnd(k)), appended(past, "v", rnd(v))
    o = rnd(attend(rnd(q), k, v, pos, m["scale"], (m.get("mask") or {}).get("size"), rnd))
    return o.reshape(T, H * V) @ f64(t[p + "o"]).T


# ---------------------------------------------------------------------------
# the state-space mixer
# ---------------------------------------------------------------------------

def short_conv(u, w, b, before):
    """u [T, C], w [C, taps] whose last column meets the token itself, ``before`` [taps - 1, C] the inputs ahead of u."""
    full, taps = torch.cat([before, u]), w.shape[1]
    return b + sum(full[j:j + u.shape[0]] * w[:, j] for j in range(taps))


def recur(x, B, C, dt, A_log, D, S):
    """x [T, H, P], B and C [T, G, N], dt [T, H], S [H, N, P] -> (y [T, H, P], the state after the last token)."""
    H, G = x.shape[1], B.shape[1]
    of = torch.arange(H) // (H // G)
    y = []
    for n in range(x.shape[0]):
        decay = torch.exp(-torch.exp(A_log) * dt[n])
        S = decay[:, None, None] * S + dt[n][:, None, None] * B[n][of][:, :, None] * x[n][:, None, :]
        y.append((S * C[n][of][:, :, None]).sum(1) + D[:, None] * x[n])
    return torch.stack(y), S


def mamba2(h, m, t, p, eps, past=None, rnd=same):
    H, P, N, G, K, parts = m["heads"], m["vdim"], m["state"], m["groups"], m["conv"], m["norm_groups"]
    T, inner = h.shape[0], H * P
    proj = h @ f64(t[p + "in"]).T
    z, u, dt = rnd(proj[:, :inner]), rnd(proj[:, inner:2 * inner + 2 * G * N]), proj[:, 2 * inner + 2 * G * N:]
    before = past["conv"] if past else torch.zeros(K - 1, u.shape[1], dtype=F)
    c = rnd(silu(short_conv(u, f64(t[p + "conv"]), f64(t[p + "conv.b"]), before)))
    dt = torch.nn.functional.softplus(dt + f64(t[p + "dt_bias"]), threshold=50.0)
    x, B, C = c[:, :inner].view(T, H, P), c[:, inner:inner + G * N].view(T, G, N), c[:, inner + G * N:].view(T, G, N)
    S = past["S"] if past else torch.zeros(H, N, P, dtype=F)
    y, S = recur(x, B, C, dt, f64(t[p + "A_log"]), f64(t[p + "D"]), S)
    if past is not None:
        past["S"], past["conv"] = S, torch.cat([before, u])[u.shape[0]:]
    y = (y.reshape(T, inner) * silu(z)).view(T, parts, inner // parts)
    y = rnd((y / rms(y, eps)).reshape(T, inner) * f64(t[p + "norm"]))
    return y @ f64(t[p + "o"]).T


# ---------------------------------------------------------------------------
# feed-forwards
# ---------------------------------------------------------------------------

def dense(h, t, p, rnd=same):
    return rnd(gelu(h @ f64(t[p + "up"]).T)) @ f64(t[p + "down"]).T


MARGINS = None                   # a list while routing margins are collected


def route(h, router, top: int):
    """(winners [T, top], their scores [T, top])."""
    z = h @ router.T
    order = torch.sort(torch.sigmoid(z), dim=-1, descending=True, stable=True)
    if MARGINS is not None and top < z.shape[1]:
        ranked = torch.sort(z, dim=-1, descending=True).values
        MARGINS.append(ranked[:, top - 1] - ranked[:, top])
    return order.indices[:, :top], order.values[:, :top]


def expert(u, t, p, rnd=same):
    return rnd(silu(u @ f64(t[p + "gate"]).T) * (u @ f64(t[p + "up"]).T)) @ f64(t[p + "down"]).T


def routed(h, ml, t, p, rnd=same):
    idx, s = route(h, f64(t[p + "router"]), ml["router"]["top"])
    y = torch.zeros_like(h)
    for n in range(h.shape[0]):
        for e, w in zip(idx[n].tolist(), s[n]):
            y[n] += expert((w * h[n])[None], t, f"{p}e{e}.", rnd)[0]
    return y


def feed_forward(h, ml, t, p, rnd=same):
    if ml["kind"] == "dense":
        return dense(h, t, p, rnd)
    return routed(h, ml, t, p, rnd)


# ---------------------------------------------------------------------------
# the model
# ---------------------------------------------------------------------------

def calls(cfg: dict) -> list:
    """(layer, whether a pass begins right before it), in the order in which layers run."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, False) for i in range(n)]
    span = [(i, i == lp["start"]) for i in range(lp["start"], lp["stop"])]
    return [(i, False) for i in range(lp["start"])] + span * lp["times"] + [(i, False) for i in range(lp["stop"], n)]


class Sequence:
    """One sequence fed in pieces: ``feed(tokens)`` returns the logits of the piece's tokens [n, vocab]."""

    def __init__(self, cfg: dict, tensors: Dict[str, torch.Tensor], rnd=same):
        self.cfg, self.t, self.rnd = cfg, tensors, rnd
        self.n = 0
        self.past: List[dict] = [{} for _ in calls(cfg)]
        self.streams: List[torch.Tensor] = []          # after the last piece: the stream after every layer call

    def feed(self, tokens) -> torch.Tensor:
        cfg, t, rnd = self.cfg, self.t, self.rnd
        eps = cfg["norm"]["eps"]
        x = x0 = f64(t["embed"])[torch.as_tensor(tokens, dtype=torch.long)]
        self.streams = []
        for c, (i, begins) in enumerate(calls(cfg)):
            L = cfg["layers"][i]
            p, m, past = f"l{i}.", L["mixer"], self.past[c]
            if begins:
                x = torch.cat([rnd(x), rnd(x0)], dim=-1) @ f64(t["loop.in"]).T
            h = rnd(named_norm(x, t, p + "norm1"))
            if L["type"] == "attention":
                y = attention(h, m, t, p + "mix.", eps, self.n, past, rnd)
            elif L["type"] == "mamba2":
                y = mamba2(h, m, t, p + "mix.", eps, past, rnd)
            else:
                raise ValueError(L["type"])
            x = x + named_norm(y, t, p + "norm1b")
            if L.get("mlp") is not None:
                h = rnd(named_norm(x, t, p + "norm2"))
                x = x + named_norm(feed_forward(h, L["mlp"], t, p + "mlp.", rnd), t, p + "norm2b")
            self.streams.append(x.clone())
        self.n += len(tokens)
        return rnd(named_norm(x, t, "final.norm")) @ f64(t["embed"]).T


def logits(cfg, tensors, tokens, pieces=None, rnd=same) -> torch.Tensor:
    """Logits of every token of one sequence, fed whole or in the given pieces."""
    seq = Sequence(cfg, tensors, rnd)
    out, at = [], 0
    for n in (pieces or [len(tokens)]):
        out.append(seq.feed(tokens[at:at + n]))
        at += n
    return torch.cat(out)


def forward(cfg, tensors, tokens, rnd=same) -> torch.Tensor:
    return logits(cfg, tensors, tokens, None, rnd)


def routing_margin(cfg, tensors, tokens) -> float:
    """The smallest distance, in router logits, between a winner and a loser of any routing decision of the sequence."""
    global MARGINS
    MARGINS = []
    try:
        forward(cfg, tensors, tokens)
        return min((float(m.min()) for m in MARGINS), default=float("inf"))
    finally:
        MARGINS = None


def generate_greedy(cfg, tensors, prompt, n: int) -> List[int]:
    """``n`` tokens after ``prompt``, each the first of the largest logits."""
    seq = Sequence(cfg, tensors)
    nxt = int(torch.argmax(seq.feed(prompt)[-1]))
    out = [nxt]
    while len(out) < n:
        nxt = int(torch.argmax(seq.feed([nxt])[-1]))
        out.append(nxt)
    return out
