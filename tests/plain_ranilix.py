"""Ranilix, stated plainly: one slow function per mechanism, in 64-bit floats on the CPU.

This file is the tests' oracle.  It shares no code with the library: it reads a configuration dictionary (the
keys of config.json) and a dictionary of tensors by name, and keeps, per layer, what the tokens it has seen left
behind (keys and values, a recurrent state), so that a sequence can be fed in pieces.

Notation: ``W`` is the model's width, ``h`` a sublayer's input [tokens, W], matrices are stored [out, in].

    stream      x0 = E[token] * s_e;   logits = head n(x_last)
    layer       x <- x + mix(n1(x)) + ff(n2(x)), both branches of the same x;   n(x) = x / rms(x) * w
    ff          D relu(U h)^2
    attention   q, k, v with biases;  every head of q and of k: u / rms(u) * w;  pairs (2i, 2i + 1) of the first R dims
                turned by pos * base^(-2i/R);  v <- (1 - lam) v + lam v0, v0 the values of the first layer that
                mixes (same token);  s_ij = scale q_i.k_j for 0 <= i - j < window;
                p = exp(s) / (exp(sink_h) + sum exp(s));  o_h = sum p v;  Wo (o * sigmoid(G h))
    parallel    left_scale * left(h) + right_scale * right(h)
      left      attention without biases, norms, window, sink, mixing and gate
      right     retention: q and k turned in pairs (i, i + R/2);  k <- k / sqrt(D);  per head
                S <- decay_h S + k v^T;  o = S^T q;  o / rms(o);  Wo (o * silu(G h))
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


def norm(x, w, eps):
    return x / rms(x, eps) * w


def unit(x, eps):
    return x / rms(x, eps)


def silu(z):
    return z * torch.sigmoid(z)


# ---------------------------------------------------------------------------
# positions
# ---------------------------------------------------------------------------

def frequencies(dims: int, base: float) -> torch.Tensor:
    return torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F)


def turn(x, pos, dims: int, base: float, neighbours: bool):
    """x [tokens, heads, D]: the first ``dims`` numbers of every head in pairs, pair i turned by pos * base^(-2i/dims).
    ``neighbours``: the pairs are (2i, 2i + 1); else (i, i + dims/2)."""
    out = x.clone()
    f = frequencies(dims, base)
    for i in range(dims // 2):
        a, b = (2 * i, 2 * i + 1) if neighbours else (i, i + dims // 2)
        ang = pos.to(F) * f[i]
        c, s = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
        u, v = x[..., a], x[..., b]
        out[..., a], out[..., b] = u * c - v * s, v * c + u * s
    return out


def turned(x, pos, m: dict, neighbours: bool):
    rot = m.get("rot")
    return turn(x, pos, rot.get("dims", m["dim"]), rot["base"], neighbours) if rot else x


# ---------------------------------------------------------------------------
# softmax attention
# ---------------------------------------------------------------------------

def seen(qpos, kpos, window: Optional[int]):
    """[queries, keys]: key j is seen from query i iff 0 <= i - j (< window)."""
    d = qpos[:, None] - kpos[None, :]
    return (d >= 0) & (d < window) if window else d >= 0


def weights(s, ok, sink: Optional[float] = None):
    """Softmax over the seen keys of every row; ``sink``: the denominator also holds exp(sink)."""
    s = s.masked_fill(~ok, -math.inf)
    top = s.max(-1, keepdim=True).values
    if sink is not None:
        top = torch.clamp(top, min=sink)
    e = torch.exp(s - top)
    den = e.sum(-1, keepdim=True)
    if sink is not None:
        den = den + torch.exp(torch.tensor(sink, dtype=F) - top)
    return e / den


def attend(q, k, v, qpos, scale, window=None, sink=None, rnd=same):
    """q [T, H, D] at positions ``qpos``, k [n, G, D] and v [n, G, V] at positions 0..n-1 -> [T, H, V].
    ``rnd``: tensor-core kernels round the weights that meet the values."""
    H, G = q.shape[1], k.shape[1]
    ok = seen(qpos, torch.arange(k.shape[0]), window)
    out = []
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        out.append(rnd(weights(s, ok, None if sink is None else float(sink[h]))) @ v[:, g])
    return torch.stack(out, dim=1)


def appended(past, key, x):
    """``x`` behind what ``past`` holds under ``key``; the whole is kept there."""
    if past is None:
        return x
    past[key] = torch.cat([past[key], x]) if key in past else x
    return past[key]


def window_attention(h, m, t, p, eps, first_pos=0, past=None, first_values=None, rnd=same):
    """Returns (output, this layer's own values before mixing [T, G, V]).  ``first_values``: the first mixing layer's
    values of the same tokens, or None (this layer mixes nothing in)."""
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    pos = torch.arange(first_pos, first_pos + T)
    q = (h @ f64(t[p + "q"]).T + f64(t[p + "q.b"])).view(T, H, D)
    k = (h @ f64(t[p + "k"]).T + f64(t[p + "k.b"])).view(T, G, D)
    v = own = (h @ f64(t[p + "v"]).T + f64(t[p + "v.b"])).view(T, G, V)
    q = turned(norm(q, f64(t[p + "q.norm"]), eps), pos, m, True)
    k = turned(norm(k, f64(t[p + "k.norm"]), eps), pos, m, True)
    if first_values is not None:
        lam = float(t[p + "vmix"])
        v = (1.0 - lam) * v + lam * first_values
    k, v = appended(past, "k", rnd(k)), appended(past, "v", rnd(v))
    o = rnd(attend(rnd(q), k, v, pos, m["scale"], (m.get("mask") or {}).get("size"), f64(t[p + "sink"]), rnd))
    o = rnd(o.reshape(T, H * V) * torch.sigmoid(h @ f64(t[p + "g"]).T))
    return o @ f64(t[p + "o"]).T, own


def plain_attention(h, m, t, p, first_pos=0, past=None, rnd=same):
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    pos = torch.arange(first_pos, first_pos + T)
    q = turned((h @ f64(t[p + "q"]).T).view(T, H, D), pos, m, True)
    k = turned((h @ f64(t[p + "k"]).T).view(T, G, D), pos, m, True)
    v = (h @ f64(t[p + "v"]).T).view(T, G, V)
    k, v = appended(past, "k", rnd(k)), appended(past, "v", rnd(v))
    o = rnd(attend(rnd(q), k, v, pos, m["scale"], (m.get("mask") or {}).get("size"), None, rnd))
    return o.reshape(T, H * V) @ f64(t[p + "o"]).T


# ---------------------------------------------------------------------------
# retention
# ---------------------------------------------------------------------------

def retain(q, k, v, decay, S):
    """q, k [T, H, D], v [T, H, V], decay per head, S [H, D, V] -> (o [T, H, V], the state after the last token)."""
    d = torch.tensor(decay, dtype=F)[:, None, None]
    out = []
    for n in range(q.shape[0]):
        S = d * S + k[n][:, :, None] * v[n][:, None, :]
        out.append((S * q[n][:, :, None]).sum(1))
    return torch.stack(out), S


def retention(h, m, t, p, eps, first_pos=0, past=None, rnd=same):
    H, D, V = m["heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    pos = torch.arange(first_pos, first_pos + T)
    q = turned((h @ f64(t[p + "q"]).T).view(T, H, D), pos, m, False)
    k = turned((h @ f64(t[p + "k"]).T).view(T, H, D), pos, m, False) * D ** -0.5
    v = rnd(h @ f64(t[p + "v"]).T).view(T, H, V)
    S = past["S"] if past else torch.zeros(H, D, V, dtype=F)
    o, S = retain(q, k, v, m["decay"], S)
    if past is not None:
        past["S"] = S
    o = rnd(unit(o, eps).reshape(T, H * V) * silu(h @ f64(t[p + "g"]).T))
    return o @ f64(t[p + "o"]).T


# ---------------------------------------------------------------------------
# the model
# ---------------------------------------------------------------------------

def feed_forward(h, t, p, rnd=same):
    u = torch.clamp(h @ f64(t[p + "up"]).T, min=0.0)
    return rnd(u * u) @ f64(t[p + "down"]).T


class Sequence:
    """One sequence fed in pieces: ``feed(tokens)`` returns the logits of the piece's tokens [n, vocab]."""

    def __init__(self, cfg: dict, tensors: Dict[str, torch.Tensor], rnd=same):
        self.cfg, self.t, self.rnd = cfg, tensors, rnd
        self.n = 0
        self.past: List[dict] = [{"left": {}, "right": {}, "own": {}} for _ in cfg["layers"]]
        self.streams: List[torch.Tensor] = []          # after the last piece: the stream after every layer

    def feed(self, tokens) -> torch.Tensor:
        cfg, t, rnd = self.cfg, self.t, self.rnd
        eps = cfg["norm"]["eps"]
        x = f64(t["embed"])[torch.as_tensor(tokens, dtype=torch.long)] * (cfg.get("embedding") or {}).get("scale", 1.0)
        self.streams = []
        first = None                                   # the first mixing layer's values of these tokens
        for i, L in enumerate(cfg["layers"]):
            p, m, past = f"l{i}.", L["mixer"], self.past[i]
            h = rnd(norm(x, f64(t[p + "norm1"]), eps))
            if L["type"] == "attention":
                mixes = bool(m.get("v_mix"))
                y, own = window_attention(h, m, t, p + "mix.", eps, self.n, past["own"], first if mixes else None, rnd)
                if mixes and first is None:
                    first = own
            elif L["type"] == "parallel":
                y = m["left_scale"] * plain_attention(h, m["left"], t, p + "mix.left.", self.n, past["left"], rnd) \
                    + m["right_scale"] * retention(h, m["right"], t, p + "mix.right.", eps, self.n, past["right"], rnd)
            else:
                raise ValueError(L["type"])
            if L.get("mlp") is not None:
                y = y + feed_forward(rnd(norm(x, f64(t[p + "norm2"]), eps)), t, p + "mlp.", rnd)
            x = x + y
            self.streams.append(x.clone())
        self.n += len(tokens)
        return rnd(norm(x, f64(t["final.norm"]), eps)) @ f64(t["head"]).T


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


def generate_greedy(cfg, tensors, prompt, n: int) -> List[int]:
    """``n`` tokens after ``prompt``, each the first of the largest logits."""
    seq = Sequence(cfg, tensors)
    nxt = int(torch.argmax(seq.feed(prompt)[-1]))
    out = [nxt]
    while len(out) < n:
        nxt = int(torch.argmax(seq.feed([nxt])[-1]))
        out.append(nxt)
    return out
