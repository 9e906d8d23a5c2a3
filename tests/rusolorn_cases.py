"""Small Rusolorn configurations and random weights for the tests, made here (not by the package's
random-weights mode), and the glue that runs the plain implementation (tests/plain_rusolorn.py).  The
configurations differ from one another in every size, and inside a model from layer to layer; between them they cover
one and several key/value heads on either side, key heads of the delta rule smaller and larger than its value
heads, convolutions of 1 to 6 taps, windows from 1 key to none, experts with limits of their own, one group,
groups of one expert, all groups kept, one expert per token and all of them, no shared expert, layers without
a feed-forward, a model without token inputs, multipliers of 1, head sizes of 64 and 128 (the tensor-core attention
kernels) and sizes that are no multiple of 2, 4 or 8.
"""
from __future__ import annotations

import copy
import math

import torch

import plain_rusolorn


def moe(ff, experts, top, groups=None, shared=None, limit=1.2):
    m = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if groups:
        m["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared:
        m["shared"] = {"ff": shared[0], "limit": shared[1]}
    return m


def layer(left, right, mlp=None):
    """left: (heads, kv_heads, dim, window or 0, scale); right: (heads, kv_heads, dim, vdim, taps)."""
    H, G, dim, window, scale = left
    lt = {"heads": H, "kv_heads": G, "dim": dim, "vdim": dim, "scale": scale}
    if window:
        lt["mask"] = {"size": window}
    rt = dict(zip(("heads", "kv_heads", "dim", "vdim", "conv"), right))
    return {"type": "parallel", "mixer": {"left": lt, "right": rt}, "mlp": mlp}


def config(layers, width, vocab, side=8, eps=1e-5, mult=0.8, scale=3.0):
    cfg = {"architecture": "Rusolorn", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "layers": layers,
           "norm": {"eps": eps}, "residual_mult": mult}
    if side:
        cfg["token_side"] = {"dim": side}
    return cfg


CASES = {
    "one_layer": config([layer((4, 2, 12, 7, 0.5), (3, 3, 8, 20, 4), moe(20, 8, 3, (4, 2), (28, 0.9)))], width=36, vocab=61),
    "mixers_alone": config([layer((3, 3, 10, 0, 0.4), (4, 2, 16, 8, 3)), layer((2, 1, 8, 5, 0.9), (2, 1, 24, 16, 2))], width=28,
                           vocab=53, side=0, mult=1.0, scale=1.0),
    "window_1": config([layer((2, 2, 16, 1, 0.7), (2, 2, 32, 24, 1), moe(12, 4, 4))], width=24, vocab=47, side=3),
    "groups_of_one": config([layer((5, 1, 6, 11, 1.1), (1, 1, 40, 12, 6), moe(14, 6, 2, (6, 3), (10, 2.0), 0.7))], width=20,
                            vocab=43, side=12, eps=3e-6),
    "one_expert_each": config([layer((2, 1, 14, 4, 0.6), (6, 2, 12, 10, 5), moe(18, 9, 1, (3, 3)))], width=26, vocab=59, side=16),
    "wide_keys": config([layer((2, 2, 20, 9, 0.5), (2, 1, 136, 40, 4), moe(16, 4, 2, (2, 1), (16, 1.0)))], width=48, vocab=71),
    "wide_values": config([layer((2, 1, 24, 6, 0.5), (2, 2, 20, 168, 4))], width=40, vocab=67),
    # head sizes of 64 and 128 take the tensor-core attention kernels in bfloat16
    "heads64": config([layer((8, 2, 64, 21, 0.2), (4, 2, 64, 32, 4), moe(48, 8, 2, (2, 1), (40, 1.4))),
                       layer((2, 2, 64, 70, 0.15), (2, 2, 32, 64, 4), moe(32, 8, 4, (4, 2)))], width=64, vocab=113),
    "heads128": config([layer((3, 1, 128, 50, 0.1), (2, 2, 128, 128, 4)), layer((4, 4, 64, 3, 0.2), (3, 1, 48, 56, 3))], width=56,
                       vocab=103, side=20),
    # sizes that are no multiple of 2, 4 or 8 wherever the design allows it
    "odd_sizes": config([layer((3, 1, 7, 5, 0.7), (3, 3, 5, 3, 3), moe(9, 5, 2, None, (11, 0.6))),
                         layer((1, 1, 9, 2, 0.5), (5, 1, 33, 13, 2), moe(7, 6, 3, (2, 2)))], width=37, vocab=45, side=5, mult=0.55),
    # unlike layers in two orders
    "stack": config([layer((4, 2, 32, 13, 0.3), (4, 2, 16, 24, 4), moe(24, 8, 3, (4, 2), (40, 1.1), 1.6)),
                     layer((6, 3, 16, 30, 0.5), (2, 2, 48, 40, 3)),
                     layer((2, 1, 40, 6, 0.3), (6, 3, 8, 16, 4), moe(16, 12, 4, (3, 1), None, 0.8)),
                     layer((4, 4, 24, 0, 0.4), (2, 1, 64, 32, 2), moe(32, 6, 2, None, (24, 2.5)))], width=64, vocab=131, side=16,
                    mult=0.6, scale=4.0),
    "stack_other_order": config([layer((3, 1, 20, 44, 0.4), (3, 1, 24, 18, 2)),
                                 layer((2, 2, 16, 10, 0.6), (4, 4, 12, 30, 5), moe(20, 4, 2, (2, 2), (12, 0.8))),
                                 layer((8, 2, 8, 25, 0.8), (1, 1, 72, 24, 4), moe(12, 10, 3, (5, 2), (20, 1.3), 1.0))],
                                width=44, vocab=89, side=10, mult=0.9, scale=2.0),
}


def tensor_shapes(cfg):
    """name -> (shape, kind) from the configuration alone, written out from the model's description."""
    d, L = cfg["width"], len(cfg["layers"])
    side = (cfg.get("token_side") or {}).get("dim")
    out = {"embed": ((cfg["vocab"], d), "embed")}

    def dyt(name):
        out.update({name: ((d,), "norm"), name + ".b": ((d,), "shift"), name + ".alpha": ((), "alpha")})
    dyt("final.norm")
    if side:
        out["side.embed"] = ((cfg["vocab"], L * side), "embed")
    for i, ly in enumerate(cfg["layers"]):
        p = f"l{i}."
        dyt(p + "norm1")
        lt, rt, m = ly["mixer"]["left"], ly["mixer"]["right"], p + "mix."
        wq, wk = lt["heads"] * lt["dim"], lt["kv_heads"] * lt["dim"]
        out.update({m + "left.q": ((wq, d), "matrix"), m + "left.k": ((wk, d), "matrix"), m + "left.q.norm": ((wq,), "norm"),
                    m + "left.k.norm": ((wk,), "norm"), m + "left.o": ((d, wq), "matrix"), m + "left.out": ((d,), "norm"),
                    m + "right.out": ((d,), "norm")})
        H, qk, hv, T = rt["heads"], rt["kv_heads"] * rt["dim"], rt["heads"] * rt["vdim"], rt["conv"]
        r = m + "right."
        out.update({r + "q": ((qk, d), "matrix"), r + "k": ((qk, d), "matrix"), r + "v": ((hv, d), "matrix"),
                    r + "q.conv": ((qk, T), "taps"), r + "k.conv": ((qk, T), "taps"), r + "v.conv": ((hv, T), "taps"),
                    r + "b": ((H, d), "gate"), r + "a": ((H, d), "gate"), r + "A_log": ((H,), "unit"), r + "dt_bias": ((H,), "dt"),
                    r + "norm": ((rt["vdim"],), "norm"), r + "g": ((hv, d), "matrix"), r + "o": ((d, hv), "matrix")})
        mlp = ly.get("mlp")
        if mlp is not None:
            F, E = mlp["expert"]["ff"], mlp["router"]["experts"]
            out[p + "mlp.router"] = ((E, d), "router")
            units = [(f"e{e}", F) for e in range(E)] + ([("shared", mlp["shared"]["ff"])] if mlp.get("shared") else [])
            for n, f in units:
                out.update({f"{p}mlp.{n}.gate": ((f, d), "glu"), f"{p}mlp.{n}.up": ((f, d), "glu"),
                            f"{p}mlp.{n}.down": ((d, f), "matrix")})
        if side:
            out.update({p + "side.gate": ((side, d), "matrix"), p + "side.proj": ((d, side), "matrix"), p + "side.norm": ((d,), "norm")})
    return out


def make_weights(cfg, seed, dtype=torch.float32, gain=1.3):
    """Random tensors at which every mechanism moves the output: Dynamic Tanh bends (alpha x of order 1), clamps
    bite on both sides, decays lie between 0.3 and nearly 1, write strengths between 0.1 and 0.9, and the router's
    logits lie far enough apart that the choice seldom hangs on the last bits.  Stored in `dtype`."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    out = {}
    for name, (shape, kind) in tensor_shapes(cfg).items():
        fan = 1.0 / math.sqrt(shape[1]) if len(shape) == 2 else 1.0
        if kind in ("matrix", "glu"):
            t = rnd(*shape) * gain * fan * (1.5 if kind == "glu" else 1.0)
        elif kind == "router":
            t = rnd(*shape) * 5.0 * fan
        elif kind == "gate":
            t = rnd(*shape) * 2.0 * fan
        elif kind in ("embed", "taps"):
            t = rnd(*shape) * (1.0 if kind == "embed" else 1.3 * fan)
        elif kind == "norm":
            t = 1.0 + 0.2 * rnd(*shape)
        elif kind == "shift":
            t = 0.2 * rnd(*shape)
        elif kind == "alpha":
            t = torch.tensor(0.5, dtype=torch.float64) + 0.1 * rnd(1)[0]
        elif kind == "unit":
            t = 0.7 * rnd(*shape)
        elif kind == "dt":
            t = -2.5 + 1.5 * rnd(*shape)
        else:
            raise ValueError(kind)
        out[name] = t.to(dtype)
    return out


def oracle(cfg, weights, tokens, streams=None, given=None, slack=0.0):
    """float64 logits [T, vocab] of the plain implementation from the weights as stored.  The result carries
    `margin` [T], how far each token's choice of experts is from another choice (the smallest over the layers), and
    `again(given, slack)`: the logits once more with somebody else's choices taken over where they are as good
    as the plain router's own.  For weights stored in bfloat16 it also carries `noise` [T]: how far each row moves
    when every sublayer reads and returns rows rounded to bfloat16 (what rounding alone does to the row)."""
    margins = []
    logits = plain_rusolorn.forward(cfg, weights, tokens, streams, margins=margins, given=given, slack=slack)
    if weights["embed"].dtype == torch.bfloat16:
        coarse = plain_rusolorn.forward(cfg, weights, tokens, given=given, slack=slack,
                                        coarse=lambda t: t.to(torch.bfloat16).to(torch.float64))
        logits.noise = [row_error(coarse[p], logits[p]) for p in range(len(tokens))]
    m = torch.full((len(tokens),), math.inf, dtype=torch.float64)
    for per_token in margins:
        m = torch.minimum(m, torch.tensor(per_token, dtype=torch.float64))
    logits.margin = m
    logits.again = lambda given, slack: oracle(cfg, weights, tokens, given=given, slack=slack)
    return logits


def sharpened(cfg, factor, layers=None):
    """The same model with the attention scores multiplied by `factor`: rows then hang on few keys."""
    cfg = copy.deepcopy(cfg)
    for i, ly in enumerate(cfg["layers"]):
        if layers is None or i in layers:
            ly["mixer"]["left"]["scale"] *= factor
    return cfg


def with_windows(cfg, delta):
    """The same model with every window `delta` keys longer: what a mask that is off by one would compute."""
    cfg = copy.deepcopy(cfg)
    for ly in cfg["layers"]:
        if ly["mixer"]["left"].get("mask"):
            ly["mixer"]["left"]["mask"]["size"] += delta
    return cfg


def first_rows(cfg, w):
    """What layer 0's sublayers read, token id by token id [vocab, d] (before any token has met another)."""
    x = w["embed"].double() * cfg["embedding"]["scale"]
    return plain_rusolorn.dyt(x, w["l0.norm1.alpha"].double(), w["l0.norm1"].double(), w["l0.norm1.b"].double())


def marked_attention(cfg, w, asker, target, boost=6.0):
    """Layer 0: every query head asks with its group's key projection and the key norm's weights, and the token
    `asker` asks as if it were `target` (the map R with R h(asker) = h(target), the identity across h(asker)).
    With a sharp scale, a row of `asker` hangs on the key of a `target` token when one is inside the window and is
    spread over the other keys when none is.  The side's output weight is multiplied by `boost`, so that what
    attention finds is not drowned by the rest of the stream."""
    w = dict(w)
    lt = cfg["layers"][0]["mixer"]["left"]
    H, G, d = lt["heads"], lt["kv_heads"], lt["dim"]
    p = "l0.mix.left."
    h = first_rows(cfg, w)
    ha, ht = h[asker], h[target]
    R = torch.eye(cfg["width"], dtype=torch.float64) + torch.outer(ht - ha, ha) / (ha @ ha)
    k, kn = w[p + "k"].double().view(G, d, -1), w[p + "k.norm"].double().view(G, d)
    q = torch.stack([k[i // (H // G)] for i in range(H)]).reshape(H * d, -1) @ R
    w[p + "q"] = q.to(w[p + "q"].dtype)
    w[p + "q.norm"] = torch.stack([kn[i // (H // G)] for i in range(H)]).reshape(H * d).to(w[p + "q.norm"].dtype)
    w["l0.mix.left.out"] = (w["l0.mix.left.out"].double() * boost).to(w["l0.mix.left.out"].dtype)
    return w


def marked_delta(cfg, w, marker, gate=24.0, boost=30.0):
    """Layer 0: only the token `marker` writes (its write strength is nearly 1, the others' nearly 0) and nothing
    decays, so what the marker wrote is what the memory holds hundreds of tokens later: a state that is lost, reset
    or carried wrongly between steps and chunks changes every later row.  The stream's norm gets one column that is 1
    for every token, which serves as a bias."""
    w = dict(w)
    H = cfg["layers"][0]["mixer"]["right"]["heads"]
    dt = w["embed"].dtype
    for n, v in (("l0.norm1", 0.0), ("l0.norm1.b", 1.0)):
        w[n] = w[n].clone()
        w[n][0] = v
    hm = first_rows(cfg, w)[marker].clone()
    hm[0] = 0.0
    row = gate * hm / (hm @ hm)
    row[0] = -gate / 2
    w["l0.mix.right.b"] = row.repeat(H, 1).to(dt)
    w["l0.mix.right.a"] = torch.zeros_like(w["l0.mix.right.a"])
    w["l0.mix.right.dt_bias"] = torch.full((H,), -9.0).to(dt)
    w["l0.mix.right.A_log"] = torch.zeros_like(w["l0.mix.right.A_log"])
    w["l0.mix.right.out"] = (w["l0.mix.right.out"].double() * boost).to(dt)
    return w


def build_engine(cfg, weights, dtype, max_tokens, block_size=8, max_requests=4, use_graphs=None, device="cuda:0"):
    """`use_graphs` None: replay from graphs in float32 only (a replayed step does not show which experts
    it chose, and in bfloat16 the comparison wants to know: see `oracle`)."""
    if use_graphs is None:
        use_graphs = dtype == "float32"
    from rllm_b200.config import config_from_dict
    from rllm_b200.engine import Engine
    from rllm_b200.models.model import DecoderModel, parse_dtype
    from rllm_b200.parts import Runtime
    model = DecoderModel(config_from_dict(cfg).model_spec(), Runtime(torch.device(device), parse_dtype(dtype)))
    model.load_tensors(dict(weights))
    return Engine(model, block_size=block_size, max_tokens=max_tokens, max_requests=max_requests,
                  use_graphs=use_graphs)


def tokens_for(cfg, n, seed, avoid=()):
    g = torch.Generator().manual_seed(3000 + seed)
    free = [t for t in range(cfg["vocab"]) if t not in avoid]
    return [free[int(i)] for i in torch.randint(0, len(free), (n,), generator=g)]


def row_error(row, ref):
    """max |row - ref| / max |ref| with the rows' means taken off (logits are defined up to a shift)."""
    row, ref = row.double() - row.double().mean(), ref.double() - ref.double().mean()
    return float((row - ref).abs().max() / ref.abs().max().clamp_min(1e-30))
