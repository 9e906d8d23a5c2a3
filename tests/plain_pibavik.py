"""Pibavik, written out plainly: float64, one function per mechanism, whole sequences from their start,
explicit Python loops over tokens, heads and experts where a mechanism has them.  Shares no code with the
package; the tests compare the engine with it.

The design: x = embed[token] * scale; every layer is x <- x + mixer(norm1(x)), x <- x + experts(norm2(x)) with RMS
norms; logits are a matrix of their own times the final norm's rows.  Three mixers: windowed attention whose scores
lose a slope per head for every position of distance (a layer may read an earlier layer's keys and values),
attention through low-rank latents without positions, and a pair side by side: windowed attention with normed,
rotated queries and keys and a gate per head, and a state-space recurrence with one decay per head behind a short
convolution.  The experts square a relu; a token's weight for an expert multiplies what the expert reads.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + torch.clamp(z, min=0.0)


# ------------------------------------------------------------------ attention over heads

def slopes(H):
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / H) for h in range(H)], dtype=F64)


def attend(q, k, v, scale, window=0, slope=None):
    """q [n, H, dk], k [n, G, dk], v [n, G, dv] -> [n, H, dv].  A query at i sees the keys j <= i with i - j < window
    (0: all of them); slope [H]: slope_h * (i - j) is taken off the score."""
    n, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros((n, H, v.shape[-1]), dtype=F64)
    for i in range(n):
        lo = max(0, i - window + 1) if window else 0
        far = torch.arange(i - lo, -1, -1, dtype=F64)
        for h in range(H):
            g = h // (H // G)
            s = (k[lo:i + 1, g] @ q[i, h]) * scale
            if slope is not None:
                s = s - slope[h] * far
            out[i, h] = torch.softmax(s, 0) @ v[lo:i + 1, g]
    return out


def rotate(x, dims, base):
    """x [n, heads, d] at positions 0..n-1: entry i of the first `dims` turns with entry i + dims/2."""
    x = x.clone()
    half = dims // 2
    for p in range(x.shape[0]):
        for i in range(half):
            a = p * base ** (-2.0 * i / dims)
            u, v = x[p, :, i].clone(), x[p, :, i + half].clone()
            x[p, :, i] = u * math.cos(a) - v * math.sin(a)
            x[p, :, i + half] = v * math.cos(a) + u * math.sin(a)
    return x


def window_of(mx):
    return mx["mask"]["size"] if mx.get("mask") else 0


def sloped_attention(h, w, pre, mx, shared=None):
    """-> (rows, (k, v)); `shared`: another layer's (k, v)."""
    n = h.shape[0]
    H, G = mx["heads"], mx["kv_heads"]
    q = (h @ w[pre + "q"].T).view(n, H, mx["dim"])
    if shared is None:
        shared = ((h @ w[pre + "k"].T).view(n, G, mx["dim"]), (h @ w[pre + "v"].T).view(n, G, mx["vdim"]))
    o = attend(q, shared[0], shared[1], mx["scale"], window_of(mx), slopes(H))
    return o.reshape(n, -1) @ w[pre + "o"].T, shared


def latent_attention(h, w, pre, mx, eps):
    """Per-head keys and values are formed from the latents, head by head."""
    n, H = h.shape[0], mx["heads"]
    cq = rms(h @ w[pre + "dq"].T, eps) * w[pre + "dq.norm"]
    c = rms(h @ w[pre + "dkv"].T, eps) * w[pre + "dkv.norm"]
    q = (cq @ w[pre + "uq"].T).view(n, H, mx["dim"])
    k = (c @ w[pre + "uk"].T).view(n, H, mx["dim"])
    v = (c @ w[pre + "uv"].T).view(n, H, mx["vdim"])
    return attend(q, k, v, mx["scale"]).reshape(n, -1) @ w[pre + "o"].T


def gated_attention(h, w, pre, mx, eps):
    n, H, G, d = h.shape[0], mx["heads"], mx["kv_heads"], mx["dim"]
    q = rms((h @ w[pre + "q"].T).view(n, H, d), eps) * w[pre + "q.norm"]
    k = rms((h @ w[pre + "k"].T).view(n, G, d), eps) * w[pre + "k.norm"]
    v = (h @ w[pre + "v"].T).view(n, G, mx["vdim"])
    if mx.get("rot"):
        q, k = (rotate(t, mx["rot"]["dims"], mx["rot"]["base"]) for t in (q, k))
    o = attend(q, k, v, mx["scale"], window_of(mx)) * torch.sigmoid(h @ w[pre + "g"].T)[:, :, None]
    return o.reshape(n, -1) @ w[pre + "o"].T


# ------------------------------------------------------------------ state space with one decay per head

def causal_conv_silu(x, taps, bias):
    """x [n, c], taps [c, T]: the last column weighs the current token; zeros before the start."""
    n, T = x.shape[0], taps.shape[1]
    out = bias.repeat(n, 1)
    for t in range(n):
        for j in range(T):
            s = t - (T - 1) + j
            if s >= 0:
                out[t] += taps[:, j] * x[s]
    return silu(out)


def state_space(x, B, C, dt, A, D):
    """x [n, H, P], B, C [n, G, N], dt [n, H], A, D [H] -> y [n, H, P]: the literal recurrence
    S = exp(-A dt) S + dt B x^T, y = S^T C + D x."""
    n, H, P = x.shape
    G, N = B.shape[1:]
    y = torch.zeros_like(x)
    for h in range(H):
        g = h // (H // G)
        S = torch.zeros((N, P), dtype=F64)
        for t in range(n):
            S = torch.exp(-A[h] * dt[t, h]) * S + dt[t, h] * torch.outer(B[t, g], x[t, h])
            y[t, h] = S.T @ C[t, g] + D[h] * x[t, h]
    return y


def mamba2(h, w, pre, mx, eps):
    n, H, P, N, G = h.shape[0], mx["heads"], mx["vdim"], mx["state"], mx["groups"]
    I = H * P
    z, xbc, dt = (h @ w[pre + "in"].T).split([I, I + 2 * G * N, H], -1)
    x, B, C = causal_conv_silu(xbc, w[pre + "conv"], w[pre + "conv.b"]).split([I, G * N, G * N], -1)
    y = state_space(x.view(n, H, P), B.view(n, G, N), C.view(n, G, N), softplus(dt + w[pre + "dt_bias"]),
                    torch.exp(w[pre + "A_log"]), w[pre + "D"]).reshape(n, I)
    y = rms((y * silu(z)).view(n, mx["norm_groups"], -1), eps).reshape(n, I) * w[pre + "norm"]
    return y @ w[pre + "o"].T


def side_by_side(h, w, pre, mx, eps):
    return (mx["left_scale"] * gated_attention(h, w, pre + "left.", mx["left"], eps)
            + mx["right_scale"] * mamba2(h, w, pre + "right.", mx["right"], eps))


# ------------------------------------------------------------------ experts

def expert(h, w, pre):
    return torch.clamp(h @ w[pre + "up"].T, min=0.0) ** 2 @ w[pre + "down"].T


def choose(s, top):
    """(indices of one token's experts, how far the choice is from another one) from its scores s [E]."""
    order = sorted(range(s.shape[0]), key=lambda e: (-float(s[e]), e))
    return order[:top], float(s[order[top - 1]] - s[order[top]]) if top < len(order) else math.inf


def experts(h, w, pre, mlp, given=None, slack=0.0, margins=None, chosen=None):
    """`given` {token index: experts}: somebody else's choice is taken over for a token when moving every
    score by at most `slack` makes it this router's own.  `margins` (a list) takes the distances per token, `chosen`
    (a dictionary) the experts."""
    r = mlp["router"]
    s = torch.sigmoid(h @ w[pre + "router"].T)
    out = torch.zeros_like(h)
    far = []
    for t in range(h.shape[0]):
        idx, margin = choose(s[t], r["top"])
        far.append(margin)
        cand = [int(c) for c in (given or {}).get(t, [])]
        if cand and sorted(cand) != sorted(idx) and len(set(cand)) == r["top"]:
            moved = s[t].clone() - slack
            moved[cand] += 2 * slack
            if sorted(choose(moved, r["top"])[0]) == sorted(cand):
                idx = cand
        if chosen is not None:
            chosen[t] = list(idx)
        for e in idx:
            out[t] += expert(s[t, e] * h[t:t + 1], w, f"{pre}e{e}.")[0]
    if margins is not None:
        margins.append(far)
    if mlp.get("shared"):
        out = out + expert(h, w, pre + "shared.")
    return out


# ------------------------------------------------------------------ layer, model

def mixer(h, w, i, spec, eps, kv):
    """`kv` {layer: (keys, values)} of the sloped attention layers so far."""
    pre, mx = f"l{i}.mix.", spec["mixer"]
    if spec["type"] == "attention":
        src = mx.get("kv_from")
        y, kv[i] = sloped_attention(h, w, pre, mx, None if src is None else kv[src])
        return y
    if spec["type"] == "latent_attention":
        return latent_attention(h, w, pre, mx, eps)
    return side_by_side(h, w, pre, mx, eps)


def layer(x, w, i, spec, cfg, kv, given=None, slack=0.0, margins=None, coarse=None, chosen=None):
    """`coarse`, if given, is applied to what every sublayer reads and returns (operands of fewer bits)."""
    eps = cfg["norm"]["eps"]
    see = coarse or (lambda t: t)
    x = x + see(mixer(see(rms(x, eps) * w[f"l{i}.norm1"]), w, i, spec, eps, kv))
    if spec.get("mlp"):
        x = x + see(experts(see(rms(x, eps) * w[f"l{i}.norm2"]), w, f"l{i}.mlp.", spec["mlp"], (given or {}).get(i), slack,
                            margins, chosen.setdefault(i, {}) if chosen is not None else None))
    return x


def forward(cfg, weights, tokens, streams=None, margins=None, given=None, slack=0.0, coarse=None, chosen=None):
    """Logits [n, vocab] (float64) of one sequence from its start.  `weights`: name -> tensor of any float
    type; `streams`, if a list, takes the stream after every layer; the rest: see `experts` and `layer`
    (`given` and `chosen` are {layer: {token index: experts}})."""
    w = {k: v.to(F64) for k, v in weights.items()}
    x = w["embed"][torch.tensor(list(tokens), dtype=torch.long)] * cfg["embedding"]["scale"]
    kv = {}
    for i, spec in enumerate(cfg["layers"]):
        x = layer(x, w, i, spec, cfg, kv, given, slack, margins, coarse, chosen)
        if streams is not None:
            streams.append(x.clone())
    x = rms(x, cfg["norm"]["eps"]) * w["final.norm"]
    return (coarse(x) if coarse else x) @ w["head"].T
