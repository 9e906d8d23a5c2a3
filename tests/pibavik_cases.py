"""Small Pibavik configurations and random weights for the tests, made here (not by the package's random-weights mode), and
the glue that runs the plain implementation (tests/plain_pibavik.py).  The configurations differ from one another in every
size, and inside a model from layer to layer; between them they cover one and several key/value heads, value heads smaller and
larger than key heads, windows from 1 key to none, layers that read an earlier layer's keys through the same, a shorter, a
longer and no window, latents whose sizes are multiples of nothing, heads rotated wholly, in part and not at all, convolutions of 1
to 6 taps, one group per head and one for all, norms in one part and in many, state sizes from 3 to 200, one expert per
token and all of them, no shared expert, layers without a feed-forward, embedding scale 1, head sizes of 64 and 128 (the
tensor-core attention kernels) and sizes that are no multiple of 2, 4 or 8.
"""
from __future__ import annotations

import copy
import math

import torch

import plain_pibavik


def moe(ff, experts, top, shared=0):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def heads(H, G, dim, vdim, window, scale):
    m = {"heads": H, "kv_heads": G, "dim": dim, "vdim": vdim, "scale": scale}
    if window:
        m["mask"] = {"size": window}
    return m


def sloped(H, G, dim, vdim, window, scale, mlp=None, kv_from=None):
    m = heads(H, G, dim, vdim, window, scale)
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def latent(H, dim, vdim, q_rank, kv_rank, scale, mlp=None):
    return {"type": "latent_attention", "mixer": {"heads": H, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                                                  "scale": scale}, "mlp": mlp}


def parallel(left, rot, right, mlp=None, scales=(0.7, 0.8)):
    """left: as `heads`; rot: (dims, base) or None; right: (heads, vdim, state, groups, taps, norm_groups)."""
    lt = heads(*left)
    if rot:
        lt["rot"] = {"dims": rot[0], "base": rot[1]}
    rt = dict(zip(("heads", "vdim", "state", "groups", "conv", "norm_groups"), right))
    return {"type": "parallel", "mixer": {"left": lt, "right": rt, "left_scale": scales[0], "right_scale": scales[1]}, "mlp": mlp}


def config(layers, width, vocab, eps=1e-5, scale=2.0):
    return {"architecture": "Pibavik", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "layers": layers,
            "norm": {"eps": eps}}


CASES = {
    "sloped": config([sloped(4, 2, 12, 20, 7, 0.3, moe(20, 6, 2, 28))], width=36, vocab=61),
    "sloped_padded": config([sloped(5, 1, 72, 40, 21, 0.15), sloped(3, 3, 16, 56, 9, 0.3, moe(24, 4, 1))], width=40, vocab=59),
    "shared_keys": config([sloped(6, 2, 16, 12, 5, 0.4, moe(16, 4, 1, 8)), sloped(6, 2, 16, 12, 5, 0.6, None, 0),
                           sloped(6, 2, 16, 12, 19, 0.3, moe(12, 5, 3), 0), sloped(6, 2, 16, 12, 2, 0.5, None, 0)],
                          width=32, vocab=57, scale=1.0),
    "shared_keys_all": config([sloped(2, 1, 24, 24, 8, 0.4), sloped(2, 1, 24, 24, 0, 0.5, moe(18, 3, 2), 0)], width=28, vocab=43),
    "latent": config([latent(3, 16, 24, 20, 36, 0.4, moe(24, 8, 3, 16))], width=44, vocab=67),
    "latents": config([latent(2, 40, 12, 64, 64, 0.2), latent(5, 7, 9, 11, 13, 0.5, moe(10, 4, 4))], width=38, vocab=53, eps=3e-6),
    "pair": config([parallel((4, 2, 16, 24, 7, 0.5), (8, 10000.0), (6, 12, 20, 2, 4, 3), moe(20, 8, 2, 12))], width=36, vocab=61),
    "pair_unrotated": config([parallel((2, 1, 20, 12, 11, 0.4), None, (4, 24, 40, 4, 3, 1)),
                              parallel((3, 3, 14, 14, 0, 0.6), (14, 300.0), (2, 72, 10, 1, 1, 4), moe(14, 6, 6))], width=28, vocab=47),
    "pair_wide_state": config([parallel((2, 2, 16, 16, 5, 0.5), (2, 50.0), (3, 40, 130, 1, 4, 2)),
                               parallel((1, 1, 24, 8, 1, 0.5), (12, 1000.0), (2, 136, 200, 2, 6, 8))], width=40, vocab=71),
    # head sizes of 64 and 128 take the tensor-core attention kernels in bfloat16
    "heads64": config([sloped(8, 2, 64, 64, 21, 0.12, moe(48, 8, 2, 40)), sloped(8, 2, 64, 64, 70, 0.12, None, 0),
                       parallel((4, 2, 64, 64, 33, 0.15), (16, 50000.0), (4, 64, 64, 2, 4, 4), moe(32, 8, 1))], width=64, vocab=113),
    "heads128": config([sloped(3, 1, 128, 128, 34, 0.1), parallel((2, 2, 128, 128, 40, 0.1), (128, 10000.0), (3, 32, 128, 1, 4, 1)),
                        latent(4, 64, 48, 72, 128, 0.12, moe(40, 4, 2))], width=56, vocab=103),
    # sizes that are no multiple of 2, 4 or 8 wherever the design allows it
    "odd_sizes": config([sloped(3, 1, 7, 5, 6, 0.7, moe(9, 5, 2, 11)), parallel((3, 1, 9, 11, 4, 0.5), (6, 99.0), (5, 7, 3, 5, 3, 5), moe(7, 3, 1)),
                         latent(1, 9, 3, 5, 7, 0.5)], width=37, vocab=45, scale=1.3),
    # unlike layers in two orders
    "stack": config([sloped(4, 2, 32, 32, 13, 0.25, moe(24, 8, 3, 40)), parallel((4, 2, 32, 16, 30, 0.3), (12, 2000.0), (4, 32, 48, 2, 4, 2), moe(16, 12, 4)),
                     latent(4, 24, 32, 40, 48, 0.3, moe(32, 6, 2, 24)), sloped(4, 2, 32, 32, 45, 0.25, None, 0),
                     parallel((6, 3, 16, 24, 9, 0.5), (16, 700.0), (8, 16, 24, 4, 2, 4), moe(20, 4, 1, 12))], width=64, vocab=131, scale=3.0),
    "stack_other_order": config([parallel((3, 1, 20, 28, 25, 0.4), (10, 10000.0), (3, 24, 16, 3, 5, 9)), latent(2, 16, 40, 24, 32, 0.4, moe(12, 10, 3, 20)),
                                 sloped(8, 4, 8, 16, 3, 0.8, moe(18, 4, 2)), parallel((2, 2, 48, 32, 12, 0.2), (48, 5000.0), (6, 20, 72, 2, 4, 2), moe(16, 5, 1, 8)),
                                 sloped(8, 4, 8, 16, 11, 0.8, None, 2)], width=44, vocab=89, scale=2.0),
}


def tensor_shapes(cfg):
    """name -> (shape, kind) from the configuration alone, written out from the model's description."""
    d = cfg["width"]
    out = {"embed": ((cfg["vocab"], d), "embed"), "head": ((cfg["vocab"], d), "matrix"), "final.norm": ((d,), "norm")}
    for i, ly in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", ly["mixer"]
        out[p + "norm1"] = ((d,), "norm")
        m = p + "mix."
        if ly["type"] == "attention":
            out.update({m + "q": ((mx["heads"] * mx["dim"], d), "matrix"), m + "o": ((d, mx["heads"] * mx["vdim"]), "matrix")})
            if mx.get("kv_from") is None:
                out.update({m + "k": ((mx["kv_heads"] * mx["dim"], d), "matrix"), m + "v": ((mx["kv_heads"] * mx["vdim"], d), "matrix")})
        elif ly["type"] == "latent_attention":
            H, r, k = mx["heads"], mx["q_rank"], mx["kv_rank"]
            out.update({m + "dq": ((r, d), "matrix"), m + "dq.norm": ((r,), "norm"), m + "uq": ((H * mx["dim"], r), "matrix"),
                        m + "dkv": ((k, d), "matrix"), m + "dkv.norm": ((k,), "norm"), m + "uk": ((H * mx["dim"], k), "matrix"),
                        m + "uv": ((H * mx["vdim"], k), "matrix"), m + "o": ((d, H * mx["vdim"]), "matrix")})
        else:
            a, b, lt, rt = mx["left"], mx["right"], m + "left.", m + "right."
            out.update({lt + "q": ((a["heads"] * a["dim"], d), "matrix"), lt + "k": ((a["kv_heads"] * a["dim"], d), "matrix"),
                        lt + "v": ((a["kv_heads"] * a["vdim"], d), "matrix"), lt + "q.norm": ((a["dim"],), "norm"),
                        lt + "k.norm": ((a["dim"],), "norm"), lt + "g": ((a["heads"], d), "gate"),
                        lt + "o": ((d, a["heads"] * a["vdim"]), "matrix")})
            I, C = b["heads"] * b["vdim"], b["heads"] * b["vdim"] + 2 * b["groups"] * b["state"]
            out.update({rt + "in": ((I + C + b["heads"], d), "matrix"), rt + "conv": ((C, b["conv"]), "taps"), rt + "conv.b": ((C,), "shift"),
                        rt + "dt_bias": ((b["heads"],), "dt"), rt + "A_log": ((b["heads"],), "unit"), rt + "D": ((b["heads"],), "norm"),
                        rt + "norm": ((I,), "norm"), rt + "o": ((d, I), "matrix")})
        mlp = ly.get("mlp")
        if mlp is not None:
            out[p + "norm2"] = ((d,), "norm")
            F, E = mlp["expert"]["ff"], mlp["router"]["experts"]
            out[p + "mlp.router"] = ((E, d), "router")
            for n, f in [(f"e{e}", F) for e in range(E)] + ([("shared", mlp["shared"]["ff"])] if mlp.get("shared") else []):
                out.update({f"{p}mlp.{n}.up": ((f, d), "matrix"), f"{p}mlp.{n}.down": ((d, f), "matrix")})
    return out


def make_weights(cfg, seed, dtype=torch.float32, gain=1.1):
    """Random tensors at which every mechanism moves the output: decays lie between 0.1 and nearly 1, gates between 0.1 and 0.9,
    and the router's logits lie far enough apart that the choice seldom hangs on the last bits.  Stored in `dtype`."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    out = {}
    for name, (shape, kind) in tensor_shapes(cfg).items():
        fan = 1.0 / math.sqrt(shape[1]) if len(shape) == 2 else 1.0
        t = {"matrix": lambda: rnd(*shape) * gain * fan, "router": lambda: rnd(*shape) * 2.0 * fan, "gate": lambda: rnd(*shape) * 2.0 * fan,
             "embed": lambda: rnd(*shape), "taps": lambda: rnd(*shape) * 1.3 * fan, "norm": lambda: 1.0 + 0.2 * rnd(*shape),
             "shift": lambda: 0.2 * rnd(*shape), "unit": lambda: 0.7 * rnd(*shape), "dt": lambda: -1.5 + rnd(*shape)}[kind]()
        out[name] = t.to(dtype)
    return out


def oracle(cfg, weights, tokens, streams=None, given=None, slack=0.0):
    """float64 logits [T, vocab] of the plain implementation from the weights as stored.  The result carries
    `margin` [T], how far each token's choice of experts is from another choice (the smallest over the layers), and
    `again(given, slack)`: the logits once more with somebody else's choices taken over where they are as good
    as the plain router's own.  For weights stored in bfloat16 it also carries `noise` [T]: how far each row moves
    when every sublayer reads and returns rows rounded to bfloat16 (what rounding alone does to the row)."""
    margins, chosen = [], {}
    logits = plain_pibavik.forward(cfg, weights, tokens, streams, margins=margins, given=given, slack=slack, chosen=chosen)
    if weights["embed"].dtype == torch.bfloat16:
        coarse = plain_pibavik.forward(cfg, weights, tokens, given=chosen, slack=0.1,
                                       coarse=lambda t: t.to(torch.bfloat16).to(torch.float64))
        logits.noise = [row_error(coarse[p], logits[p]) for p in range(len(tokens))]
    m = torch.full((len(tokens),), math.inf, dtype=torch.float64)
    for per_token in margins:
        m = torch.minimum(m, torch.tensor(per_token, dtype=torch.float64))
    logits.margin = m
    logits.again = lambda given, slack: oracle(cfg, weights, tokens, given=given, slack=slack)
    return logits


def masks(cfg, layers=None):
    """The sections of a configuration that hold a head's scale and mask."""
    for i, ly in enumerate(cfg["layers"]):
        if layers is None or i in layers:
            yield ly["mixer"]["left"] if ly["type"] == "parallel" else ly["mixer"]


def sharpened(cfg, factor, layers=None):
    """The same model with the attention scores multiplied by `factor`: rows then hang on few keys."""
    cfg = copy.deepcopy(cfg)
    for sec in masks(cfg, layers):
        sec["scale"] *= factor
    return cfg


def with_windows(cfg, delta, layers=None):
    """The same model with windows `delta` keys longer: what a mask that is off by one would compute."""
    cfg = copy.deepcopy(cfg)
    for sec in masks(cfg, layers):
        if sec.get("mask"):
            sec["mask"]["size"] += delta
    return cfg


def first_rows(cfg, w):
    """What layer 0's mixer reads, token id by token id [vocab, d] (before any token has met another)."""
    return plain_pibavik.rms(w["embed"].double() * cfg["embedding"]["scale"], cfg["norm"]["eps"]) * w["l0.norm1"].double()


def _as_if(cfg, w, asker, target):
    """The map R with R h(asker) = h(target) of layer 0's rows, the identity across h(asker)."""
    h = first_rows(cfg, w)
    ha, ht = h[asker], h[target]
    return torch.eye(cfg["width"], dtype=torch.float64) + torch.outer(ht - ha, ha) / (ha @ ha)


def marked(cfg, w, asker, target, boost=4.0):
    """Layer 0 (any mixer with attention): every query head asks with its group's key projection (and norm), and the token `asker`
    asks as if it were `target`: with a sharp scale a row of `asker` hangs on the key of a `target` token when it is visible and is
    spread over the other keys when none is.  What attention gives is multiplied by `boost`, so that it is not drowned by
    the rest of the stream."""
    w = dict(w)
    ly = cfg["layers"][0]
    R = _as_if(cfg, w, asker, target)
    dt = w["embed"].dtype
    if ly["type"] == "latent_attention":
        p, mx = "l0.mix.", ly["mixer"]
        assert mx["q_rank"] == mx["kv_rank"]
        w[p + "dq"] = (w[p + "dkv"].double() @ R).to(dt)
        w[p + "dq.norm"], w[p + "uq"] = w[p + "dkv.norm"], w[p + "uk"]
    else:
        side = ly["type"] == "parallel"
        p, mx = ("l0.mix.left.", ly["mixer"]["left"]) if side else ("l0.mix.", ly["mixer"])
        H, G, d = mx["heads"], mx["kv_heads"], mx["dim"]
        k = w[p + "k"].double().view(G, d, -1)
        w[p + "q"] = (torch.stack([k[i // (H // G)] for i in range(H)]).reshape(H * d, -1) @ R).to(dt)
        if side:
            w[p + "q.norm"] = w[p + "k.norm"]
    w[p + "o"] = (w[p + "o"].double() * boost).to(dt)
    return w


def marked_memory(cfg, w, marker, gate=18.0, boost=4.0):
    """Layer 0 (a pair): only the token `marker` writes to the state (its step size is large, the others' nearly nothing), so
    nothing decays and what the marker wrote is all that the state holds hundreds of tokens later.  D is zero, so that the
    right side gives what the state gives."""
    w = dict(w)
    rt = cfg["layers"][0]["mixer"]["right"]
    dt, H, p = w["embed"].dtype, rt["heads"], "l0.mix.right."
    hm = first_rows(cfg, w)[marker]
    inp = w[p + "in"].double().clone()
    inp[-H:] = (gate * hm / (hm @ hm)).repeat(H, 1)
    w[p + "in"] = inp.to(dt)
    w[p + "dt_bias"] = torch.full((H,), -16.0).to(dt)
    w[p + "A_log"], w[p + "D"] = torch.full((H,), -2.0).to(dt), torch.zeros(H).to(dt)
    w[p + "o"] = (w[p + "o"].double() * boost).to(dt)
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
    g = torch.Generator().manual_seed(4000 + seed)
    free = [t for t in range(cfg["vocab"]) if t not in avoid]
    return [free[int(i)] for i in torch.randint(0, len(free), (n,), generator=g)]


def row_error(row, ref):
    """max |row - ref| / max |ref| with the rows' means taken off (logits are defined up to a shift)."""
    row, ref = row.double() - row.double().mean(), ref.double() - ref.double().mean()
    return float((row - ref).abs().max() / ref.abs().max().clamp_min(1e-30))
