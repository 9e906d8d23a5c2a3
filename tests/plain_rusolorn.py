"""Rusolorn, written out plainly: float64, one function per mechanism, whole sequences from their start,
explicit Python loops over tokens, heads and experts where a mechanism has them.  Shares no code with the
package; the tests compare the engine with it.

The design: x = embed[token] * scale; every layer norms the stream once, h = dyt(x) with
dyt(x) = tanh(alpha x) w + b, and adds the mixer's and the experts' output side by side,
x <- x + m (mixer(h) + experts(h)); then a second table's part for this token and layer is gated by the
stream and joined, x <- x + m norm(P (gelu(G x) * e)).  The mixer is half the sum of two normed outputs: a
windowed attention without positions whose values are the keys as projected, and a gated delta rule behind
short causal convolutions.  The experts are clamped gated units picked by a softmax router inside the best
groups, beside a shared one.  Logits: dyt(x) times the embedding table.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def dyt(x, alpha, w, b):
    return torch.tanh(alpha * x) * w + b


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


# ------------------------------------------------------------------ left: windowed attention on tied values

def attention(h, w, pre, mx, eps):
    n = h.shape[0]
    H, G, dk = mx["heads"], mx["kv_heads"], mx["dim"]
    raw_k = h @ w[pre + "k"].T
    q = (rms(h @ w[pre + "q"].T, eps) * w[pre + "q.norm"]).view(n, H, dk)
    k = (rms(raw_k, eps) * w[pre + "k.norm"]).view(n, G, dk)
    v = raw_k.view(n, G, dk)
    size = mx["mask"]["size"] if mx.get("mask") else 0
    out = torch.zeros((n, H, dk), dtype=F64)
    for i in range(n):
        lo = max(0, i - size + 1) if size else 0
        for hd in range(H):
            g = hd // (H // G)
            p = torch.softmax((k[lo:i + 1, g] @ q[i, hd]) * mx["scale"], 0)
            out[i, hd] = p @ v[lo:i + 1, g]
    return out.reshape(n, H * dk) @ w[pre + "o"].T


# ------------------------------------------------------------------ right: gated delta rule

def causal_conv_silu(x, taps):
    """x [n, c], taps [c, T]: the last column weighs the current token; zeros before the start."""
    n, T = x.shape[0], taps.shape[1]
    out = torch.zeros_like(x)
    for t in range(n):
        for j in range(T):
            s = t - (T - 1) + j
            if s >= 0:
                out[t] += taps[:, j] * x[s]
    return silu(out)


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_rule(q, k, v, beta, g):
    """q, k [n, H, dk], v [n, H, dv], beta, g [n, H] -> o [n, H, dv]: the literal recurrence."""
    n, H, dk = q.shape
    out = torch.zeros((n, H, v.shape[-1]), dtype=F64)
    for hd in range(H):
        S = torch.zeros((dk, v.shape[-1]), dtype=F64)
        for t in range(n):
            S = g[t, hd] * S
            u = beta[t, hd] * (v[t, hd] - S.T @ k[t, hd])
            S = S + torch.outer(k[t, hd], u)
            out[t, hd] = S.T @ q[t, hd]
    return out


def gated_delta(h, w, pre, mx, eps):
    n = h.shape[0]
    H, G, dk, dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    part = {s: causal_conv_silu(h @ w[pre + s].T, w[pre + s + ".conv"]) for s in "qkv"}
    rep = lambda t: t.view(n, G, dk).repeat_interleave(H // G, dim=1)
    q = unit(rep(part["q"])) * dk ** -0.5
    k = unit(rep(part["k"]))
    v = part["v"].view(n, H, dv)
    beta = torch.sigmoid(h @ w[pre + "b"].T)
    g = torch.exp(-torch.exp(w[pre + "A_log"]) * torch.nn.functional.softplus(h @ w[pre + "a"].T + w[pre + "dt_bias"]))
    o = rms(delta_rule(q, k, v, beta, g), eps) * w[pre + "norm"]
    o = o.reshape(n, H * dv) * silu(h @ w[pre + "g"].T)
    return o @ w[pre + "o"].T


def mixer(h, w, pre, mx, eps):
    left = rms(attention(h, w, pre + "left.", mx["left"], eps), eps) * w[pre + "left.out"]
    right = rms(gated_delta(h, w, pre + "right.", mx["right"], eps), eps) * w[pre + "right.out"]
    return 0.5 * (left + right)


# ------------------------------------------------------------------ experts

def clamped_unit(h, w, pre, limit):
    g = torch.clamp(h @ w[pre + "gate"].T, max=limit)
    u = torch.clamp(h @ w[pre + "up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[pre + "down"].T


def choose(s, top, count, keep):
    """(indices of one token's experts, how far the choice is from another one) from its scores s [E]."""
    E = s.shape[0]
    per = E // count
    best = [float(s[g * per:(g + 1) * per].max()) for g in range(count)]
    order = sorted(range(count), key=lambda g: (-best[g], g))
    kept = set(order[:keep])
    margin = best[order[keep - 1]] - best[order[keep]] if keep < count else math.inf
    pool = sorted((e for e in range(E) if e // per in kept), key=lambda e: (-float(s[e]), e))
    if top < len(pool):
        margin = min(margin, float(s[pool[top - 1]] - s[pool[top]]))
    return pool[:top], margin


def experts(h, w, pre, mlp, given=None, slack=0.0, margins=None):
    """`given` {token index: experts}: somebody else's choice is taken over for a token when moving every
    score by at most `slack` makes it this router's own.  `margins` (a list) takes the distances per token."""
    r = mlp["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    s = torch.softmax(h @ w[pre + "router"].T, -1)
    out = torch.zeros_like(h)
    far = []
    for t in range(h.shape[0]):
        idx, margin = choose(s[t], r["top"], groups["count"], groups["keep"])
        far.append(margin)
        cand = [int(c) for c in (given or {}).get(t, [])]
        if cand and sorted(cand) != sorted(idx) and len(set(cand)) == r["top"]:
            moved = s[t].clone() - slack
            moved[cand] += 2 * slack
            if sorted(choose(moved, r["top"], groups["count"], groups["keep"])[0]) == sorted(cand):
                idx = cand
        total = sum(float(s[t, e]) for e in idx) + 1e-20
        for e in idx:
            out[t] += s[t, e] / total * clamped_unit(h[t:t + 1], w, f"{pre}e{e}.", mlp["expert"]["limit"])[0]
    if margins is not None:
        margins.append(far)
    if mlp.get("shared"):
        out = out + clamped_unit(h, w, pre + "shared.", mlp["shared"]["limit"])
    return out


# ------------------------------------------------------------------ layer, model

def token_side(x, tokens, w, i, dim, eps):
    """The normed rows that layer i's token input adds (before the multiplier)."""
    e = w["side.embed"][torch.tensor(list(tokens), dtype=torch.long), i * dim:(i + 1) * dim]
    y = (gelu_tanh(x @ w[f"l{i}.side.gate"].T) * e) @ w[f"l{i}.side.proj"].T
    return rms(y, eps) * w[f"l{i}.side.norm"]


def layer(x, tokens, w, i, spec, cfg, given=None, slack=0.0, margins=None, coarse=None):
    """`coarse`, if given, is applied to what every sublayer reads and returns (operands of fewer bits)."""
    eps, m = cfg["norm"]["eps"], cfg.get("residual_mult", 1.0)
    see = coarse or (lambda t: t)
    p = f"l{i}."
    h = see(dyt(x, w[p + "norm1.alpha"], w[p + "norm1"], w[p + "norm1.b"]))
    y = see(mixer(h, w, p + "mix.", spec["mixer"], eps))
    if spec.get("mlp"):
        y = y + see(experts(h, w, p + "mlp.", spec["mlp"], (given or {}).get(i), slack, margins))
    x = x + m * y
    if cfg.get("token_side"):
        x = x + m * see(token_side(see(x), tokens, w, i, cfg["token_side"]["dim"], eps))
    return x


def forward(cfg, weights, tokens, streams=None, margins=None, given=None, slack=0.0, coarse=None):
    """Logits [n, vocab] (float64) of one sequence from its start.  `weights`: name -> tensor of any float
    type; `streams`, if a list, takes the stream after every layer; the rest: see `experts` and `layer`
    (`given` is {layer: {token index: experts}})."""
    w = {k: v.to(F64) for k, v in weights.items()}
    scale = (cfg.get("embedding") or {}).get("scale", 1.0)
    x = w["embed"][torch.tensor(list(tokens), dtype=torch.long)] * scale
    for i, spec in enumerate(cfg["layers"]):
        x = layer(x, tokens, w, i, spec, cfg, given, slack, margins, coarse)
        if streams is not None:
            streams.append(x.clone())
    x = dyt(x, w["final.norm.alpha"], w["final.norm"], w["final.norm.b"])
    return (coarse(x) if coarse else x) @ w["embed"].T
