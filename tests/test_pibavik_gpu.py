"""Pibavik through the engine against the plain implementation (tests/plain_pibavik.py, float64).

Each new kernel alone against its formula; each mechanism as a small model; whole prompts against token-by-token decoding;
portions down to two tokens; batches of unequal requests against each alone with pages and state slots used again; keys just
inside and just outside every window, in prompts and in decoding, with weights at which one key decides a row and a check that a
window that is one key off would show; a layer that reads another layer's keys behind that layer's own window; a key hundreds of
places back through the latents, and a token hundreds of places back that decides rows through the state; the first tokens of a
sequence; long portions; long decoding through CUDA-graph replay; head sizes the tensor-core kernels take; layer sizes of a real
model; greedy generation through ``LLM.generate`` and the scheduler; ``bin/trace_run``; the random-weights mode.  The
configurations and weights are made in tests/pibavik_cases.py.
"""
import json
import math

import pytest
import torch

import pibavik_cases as pc
import plain_pibavik as pp
from pibavik_cases import CASES, row_error

pytestmark = pytest.mark.gpu

# max |engine - plain| / max |plain| over a logits row (means taken off).  float32: the engine sums in another
# order than the float64 plain implementation.  bfloat16: weights, the operands of every product and the cache are
# rounded to 8 bits of mantissa; how much that alone moves a row differs from row to row, so a row's tolerance is this one
# plus three times what rounding the sublayers' inputs and outputs does to the row in the plain implementation
# (`oracle(...).noise`), and one row in fifty may pass it by less than a factor of two.  A lost key, state or
# token moves many rows, by more; the float32 runs of the same tests see it at 1e-4.
TOL = {"float32": 1e-4, "bfloat16": 2.5e-2}
STRAY = {"float32": 0, "bfloat16": 50}
# Where the plain router's choice hangs on less than this gap between scores, the comparison takes the engine's experts
# over if they are what it gives itself after moving every score by at most this much.
CLOSE = {"float32": 1e-5, "bfloat16": 0.04}
DEV = "cuda:0"


def stored(dtype):
    return torch.float32 if dtype == "float32" else torch.bfloat16


class Rows(dict):
    """{(request, position): logits row}, and `chosen` {request: {layer: {position: experts}}}."""
    def __init__(self):
        super().__init__()
        self.chosen = {}


def watch(engine):
    """Records which experts every layer of routed experts chooses (eager steps only)."""
    if getattr(engine, "_watched", None) is None:
        engine._watched = []
        for li, block in enumerate(engine.model.blocks):
            ffn = getattr(block, "ffn", None)
            if ffn is None or not hasattr(ffn, "route"):
                continue
            seen = []

            def spy(h, _inner=ffn.route, _seen=seen):
                r = _inner(h)
                if not torch.cuda.is_current_stream_capturing():
                    _seen.append(r[0].detach().cpu())
                return r
            ffn.route = spy
            engine._watched.append((li, seen))
    return engine._watched


def run(engine, steps):
    """`steps`: list of (entries, end); an entry is (request, tokens, want).  Returns Rows."""
    from rllm_b200.engine import StepItem
    pos, out = {}, Rows()
    watched = watch(engine)
    for entries, end in steps:
        for _, seen in watched:
            seen.clear()
        logits = engine.step([StepItem(r, toks, want) for r, toks, want in entries])
        n = sum(len(toks) for _, toks, _ in entries)
        for li, seen in watched:
            idx = torch.cat(seen) if seen else None
            if idx is None or idx.shape[0] != n:
                continue                                   # a replayed step
            at = 0
            for r, toks, _ in entries:
                mine = out.chosen.setdefault(r, {}).setdefault(li, {})
                for j in range(len(toks)):
                    mine[pos.get(r, 0) + j] = idx[at + j].tolist()
                at += len(toks)
        row = 0
        for r, toks, want in entries:
            start = pos.get(r, 0)
            for w in want:
                out[(r, start + w)] = logits[row].detach().float().cpu()
                row += 1
            pos[r] = start + len(toks)
        for r in end:
            engine.finish(r)
            pos.pop(r, None)
    engine.check_device_errors()
    return out


def compare(out, refs, dtype, what, tol=None):
    tol = tol or TOL[dtype]
    assert out, what
    refs = dict(refs)
    for r, ref in refs.items():
        margin = getattr(ref, "margin", None)
        if margin is not None and float(margin.min()) < CLOSE[dtype] and getattr(out, "chosen", {}).get(r):
            refs[r] = ref.again(out.chosen[r], CLOSE[dtype])
    bad, stray = [], 0
    for (r, p), row in sorted(out.items()):
        e = row_error(row, refs[r][p])
        noise = getattr(refs[r], "noise", None)
        tol_row = tol + (3 * noise[p] if noise is not None and dtype == "bfloat16" else 0.0)
        if not e <= tol_row:
            if e <= 2 * tol_row and STRAY[dtype] and stray < max(1, len(out) // STRAY[dtype]):
                stray += 1
                continue
            bad.append(f"request {r} position {p}: error {e:.3e} > {tol_row:.3e}")
    assert not bad, f"{what}: " + "; ".join(bad[:12]) + f" ({len(bad)} of {len(out)} rows)"


def cut(tokens, sizes):
    """Portions of the given sizes in turn (the last size repeats), every position wanted."""
    out, at, i = [], 0, 0
    while at < len(tokens):
        k = min(sizes[min(i, len(sizes) - 1)], len(tokens) - at)
        out.append((tokens[at:at + k], list(range(k))))
        at, i = at + k, i + 1
    return out


def one_by_one(r, toks, lo=0):
    return [([(r, [t], [0])], []) for t in toks[lo:]]


def closing(steps, r):
    steps[-1] = (steps[-1][0], [r])
    return steps


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


def step_context(lens, starts):
    """A StepContext of requests that bring `lens` tokens from positions `starts`."""
    from rllm_b200.engine.batch import StepContext
    n = sum(lens)
    cu = [0]
    for k in lens:
        cu.append(cu[-1] + k)
    pos = [s + j for k, s in zip(lens, starts) for j in range(k)]
    seq = [r for r, k in enumerate(lens) for _ in range(k)]
    ends = [s + k for k, s in zip(lens, starts)]
    return StepContext(n_tokens=n, n_requests=len(lens), tokens=i32([0] * n), positions=i32(pos), seq_ids=i32(seq),
                       cu_q=i32(cu), ctx_lens=i32(ends), logit_rows=None, q_lens=list(lens), start_pos=list(starts),
                       ctx_lens_host=ends, max_q_len=max(lens), max_ctx_len=max(ends))


# ---------------------------------------------------------------- each kernel alone

def gen(seed):
    return torch.Generator().manual_seed(seed)


def close(got, want, dtype, scale=1.0):
    got, want = got.double().cpu(), want.double()
    tol = (3e-5 if dtype == torch.float32 else 1.2e-2) * scale
    assert float((got - want).abs().max()) <= tol * float(want.abs().max().clamp_min(1e-3)), float((got - want).abs().max())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_activation_kernel_with_a_factor_and_a_scale_per_row(dtype):
    from rllm_b200.csrc import ops
    g = gen(1)
    x, s, m = torch.randn(9, 24, generator=g), torch.rand(9, generator=g), torch.randn(9, 3, generator=g)
    out = torch.empty(9, 24, dtype=dtype, device=DEV)
    ops.rows_act(x.to(DEV), out, act="relu2", row_scale=s.to(DEV), factor=0.7)
    close(out, 0.7 * torch.clamp(x.double() * s[:, None].double(), min=0) ** 2, dtype)
    xb = x.to(torch.bfloat16)
    wide = torch.zeros(9, 40, dtype=torch.bfloat16, device=DEV)          # the eight-column form, into columns of a wider matrix
    ops.rows_act(xb.to(DEV), wide[:, 8:32], mul=m.to(DEV), mul_act="sigmoid", mul_group=8, factor=0.6)
    close(wide[:, 8:32], 0.6 * xb.double() * torch.sigmoid(m.double()).repeat_interleave(8, 1), torch.bfloat16)
    assert not wide[:, :8].any() and not wide[:, 32:].any()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("q_rank,rank,W", [(20, 36, 64), (0, 13, 13), (300, 512, 512)])
def test_latent_norm_kernel(dtype, q_rank, rank, W):
    from rllm_b200.csrc import ops
    g = gen(2)
    n, bs = 7, 4
    low = torch.randn(n, q_rank + rank, generator=g) * 2
    qw, kw = 1 + 0.3 * torch.randn(max(q_rank, 1), generator=g), 1 + 0.3 * torch.randn(rank, generator=g)
    cache = torch.full((5, 1, bs, W), 9.0, dtype=dtype, device=DEV)
    cq = torch.empty(n, q_rank, dtype=dtype, device=DEV) if q_rank else None
    slots = [3, 17, 0, -1, 8, 9, 19]
    ops.latent_norm_store(low.to(DEV), qw.to(DEV) if q_rank else None, kw.to(DEV), i32(slots), cq, cache, q_rank, rank, bs, 1e-5)
    want = pp.rms(low[:, q_rank:].double(), 1e-5) * kw.double()
    flat = cache.view(20, W)
    for t, s in enumerate(slots):
        if s >= 0:
            close(flat[s, :rank], want[t], dtype)
            assert not flat[s, rank:].any()
    assert bool((flat[[1, 2, 4, 18]] == 9.0).all())
    if q_rank:
        close(cq, pp.rms(low[:, :q_rank].double(), 1e-5) * qw.double(), dtype)


@pytest.mark.parametrize("dtype,H,G,dk,dv", [(torch.float32, 6, 2, 20, 12), (torch.bfloat16, 6, 2, 20, 12), (torch.bfloat16, 8, 2, 64, 64),
                                             (torch.bfloat16, 5, 1, 64, 64), (torch.bfloat16, 4, 1, 128, 128), (torch.bfloat16, 6, 2, 128, 128),
                                             (torch.bfloat16, 3, 3, 128, 128)])
@pytest.mark.parametrize("window", [0, 1, 17, 150])
def test_sloped_attention_kernels(dtype, H, G, dk, dv, window):
    """Prompt portions, short portions and single tokens at several contexts, through every attention kernel: plain, mma.sync prompt
    and decode shapes, tcgen05.  Slopes from 2^-8 to 1/2 over contexts of 300 keys."""
    from rllm_b200.csrc import ops
    g = gen(3)
    bs, lens, starts = 16, [70, 1, 200, 5, 1, 33], [0, 299, 90, 40, 0, 7]
    ctx = step_context(lens, starts)
    slope = pp.slopes(H)
    table, pages = [], 0
    for L, s in zip(lens, starts):
        k = -(-(L + s) // bs)
        table.append(list(range(pages, pages + k)))
        pages += k
    width = max(len(t) for t in table)
    order = torch.randperm(pages, generator=g)
    bt = torch.zeros(len(lens), width, dtype=torch.int32)
    for r, t in enumerate(table):
        bt[r, :len(t)] = order[t].to(torch.int32)
    kc, vc = torch.randn(pages, G, bs, dk, generator=g).to(dtype), torch.randn(pages, G, bs, dv, generator=g).to(dtype)
    n = sum(lens)
    q = torch.randn(n, H * dk, generator=g).to(dtype)
    out = torch.empty(n, H * dv, dtype=dtype, device=DEV)
    scale = 2.0 / math.sqrt(dk)
    ops.paged_attention(q.to(DEV), kc.to(DEV), vc.to(DEV), out, ctx, bt.to(DEV), H, G, dk, bs, scale, window, v_head_dim=dv,
                        slopes=slope.to(DEV, torch.float32))
    ops.check_device_errors()
    at = 0
    for r, (L, s) in enumerate(zip(lens, starts)):
        pos = torch.arange(s + L)
        rows = lambda c: c[bt[r].long()[pos // bs], :, pos % bs].double()          # [keys, G, d]
        k, v = rows(kc), rows(vc)
        qq = q[at:at + L].double().view(L, H, dk)
        sc = torch.einsum("thd,jhd->thj", qq, k.repeat_interleave(H // G, 1)) * scale
        dist = (torch.arange(s, s + L)[:, None] - pos[None]).double()
        sc = sc - slope[None, :, None] * dist[:, None]
        hidden = (dist < 0) | ((dist >= window) if window else False)
        p = torch.softmax(sc.masked_fill(hidden[:, None], -math.inf), -1)
        want = torch.einsum("thj,jhd->thd", p, v.repeat_interleave(H // G, 1)).reshape(L, H * dv)
        close(out[at:at + L], want, dtype)
        at += L


def ssd_inputs(H, P, N, G, taps, n, seed, dt_shift=0.0):
    """(rows float32 [n, ...], parameters, plain(rows) -> the rows the output projection reads)."""
    g = gen(seed)
    I, C = H * P, H * P + 2 * G * N
    rnd = lambda *s: torch.randn(*s, generator=g)
    rows = rnd(n, I + C + H)
    rows[:, I + C:] += dt_shift
    par = {"conv": rnd(C, taps) / math.sqrt(taps), "b": 0.2 * rnd(C), "dt": rnd(H) - 1.0, "A": torch.exp(0.7 * rnd(H)), "D": 1 + 0.2 * rnd(H),
           "w": 1 + 0.2 * rnd(I)}

    def plain(rows, parts, eps):
        d = {k: v.double() for k, v in par.items()}
        z, xbc, dt = rows.double().split([I, C, H], -1)
        x, B, Cm = pp.causal_conv_silu(xbc, d["conv"], d["b"]).split([I, G * N, G * N], -1)
        m = rows.shape[0]
        y = pp.state_space(x.view(m, H, P), B.view(m, G, N), Cm.view(m, G, N), pp.softplus(dt + d["dt"]), d["A"], d["D"]).reshape(m, I)
        return pp.rms((y * pp.silu(z)).view(m, parts, -1), eps).reshape(m, I) * d["w"]
    return rows, par, plain


def run_ssd(rows, par, state, lens, starts, slots, H, P, N, G, dtype, parts=1, eps=1e-5):
    from rllm_b200.csrc import ops
    d = {k: v.to(DEV) for k, v in par.items()}
    out = torch.empty(rows.shape[0], H * P, dtype=dtype, device=DEV)
    ops.ssd(rows.to(DEV), d["conv"].t().contiguous(), d["b"], d["dt"], d["A"], d["D"], d["w"], eps, parts, state,
            step_context(lens, starts), i32(slots), out, H, G, P, N)
    return out


SSD_SIZES = [(4, 16, 32, 2, 4, 2), (6, 40, 56, 3, 4, 4), (2, 64, 128, 1, 4, 1), (3, 7, 5, 3, 3, 7), (4, 24, 16, 1, 1, 4), (2, 80, 64, 2, 2, 1),
             (1, 136, 20, 1, 6, 2), (3, 40, 130, 1, 4, 1), (2, 16, 256, 2, 4, 2), (5, 12, 9, 5, 5, 6), (8, 64, 64, 8, 4, 8), (2, 1, 3, 1, 4, 1)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,P,N,G,taps,parts", SSD_SIZES)
def test_state_space_kernels_under_every_cut(dtype, H, P, N, G, taps, parts):
    """Three requests of 150, 9 and 70 tokens: whole, in cuts of all kinds beside one another, token by token; the state in
    slots that hold something else before."""
    from rllm_b200.csrc import ops
    lens = {"a": 150, "b": 9, "c": 70}
    slot = {"a": 2, "b": 0, "c": 3}
    rows, par, plain = ssd_inputs(H, P, N, G, taps, sum(lens.values()), 5)
    rows = dict(zip(lens, rows.split(list(lens.values()))))
    want = {r: plain(x, parts, 1e-5) for r, x in rows.items()}
    plans = [[("a", 150), ("b", 9), ("c", 70)], "next", [("a", 65), ("c", 1)], [("c", 2), ("a", 64), ("b", 3)], [("b", 6), ("a", 21), ("c", 63)],
             [("c", 4)], "next", [("a", 2), ("b", 1), ("c", 20)]] + [[("a", 1), ("b", 1)]] * 8 + [[("c", 50), ("a", 8)], [("a", 7)], [("a", 125)]]
    state = torch.randn(5, ops.ssd_state_floats(H, P, N, G, taps), device=DEV)
    at = {}
    for step in plans:
        if step == "next":
            at = {}
            continue
        for r, _ in step:
            if r not in at:
                at[r] = 0
                state[slot[r]].zero_()
        x = torch.cat([rows[r][at[r]:at[r] + k] for r, k in step])
        out = run_ssd(x, par, state, [k for _, k in step], [at[r] for r, _ in step], [slot[r] for r, _ in step], H, P, N, G, dtype, parts)
        i = 0
        for r, k in step:
            got, ref = out[i:i + k], want[r][at[r]:at[r] + k]
            if dtype == torch.bfloat16 and H * P // parts < 8:
                # a part of few columns can be a difference of large terms as a whole: bfloat16 storage of x, B and C shows there
                bad = (got.double().cpu() - ref).abs().amax(1) > 0.05 * float(ref.abs().max())
                assert int(bad.sum()) <= max(1, k // 25)
            else:
                close(got, ref, dtype, 3.0 if dtype == torch.float32 else 4.0)
            at[r] += k
            i += k


@pytest.mark.parametrize("H,P,N,G,taps", [(4, 16, 32, 2, 4), (2, 64, 128, 1, 4), (3, 40, 100, 3, 3)])
def test_state_space_chunks_leave_the_state_that_single_tokens_leave(H, P, N, G, taps):
    """300 rows in one portion on the tensor cores and the same rows four at a time: the same state up to the rounding of the products
    (operands of 16 bits of mantissa), and the same outputs up to bfloat16."""
    from rllm_b200.csrc import ops
    rows, par, _ = ssd_inputs(H, P, N, G, taps, 300, 6)
    per = ops.ssd_state_floats(H, P, N, G, taps)
    a, b = torch.zeros(1, per, device=DEV), torch.zeros(1, per, device=DEV)
    one = run_ssd(rows, par, a, [300], [0], [0], H, P, N, G, torch.bfloat16)
    two = torch.cat([run_ssd(rows[i:i + 4], par, b, [4], [i], [0], H, P, N, G, torch.bfloat16) for i in range(0, 300, 4)])
    close(one, two.double().cpu(), torch.bfloat16)
    S = slice(0, H * P * N)
    close(a[:, S], b[:, S].double().cpu(), torch.float32, 3.0)
    R, C = taps - 1 + 8, H * P + 2 * G * N
    ring = lambda s: s[0, H * P * N:H * P * N + R * C].view(R, C)[[p % R for p in range(300 - taps + 1, 300)]]
    assert torch.equal(ring(a), ring(b))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_state_space_decays_of_every_size_in_one_chunk(dtype):
    """Step sizes from nothing to hundreds: a token that wipes the state beside tokens that keep it."""
    from rllm_b200.csrc import ops
    H, P, N, G, taps = 2, 16, 24, 1, 4
    rows, par, plain = ssd_inputs(H, P, N, G, taps, 140, 7, dt_shift=-6.0)
    I, C = H * P, H * P + 2 * G * N
    for t in (3, 4, 11, 63, 64, 90):
        rows[t, I + C:] = torch.tensor([300.0, 40.0])
    want = plain(rows, 2, 1e-5)
    for cuts in ([140], [70, 70], [4] * 35):
        state = torch.zeros(1, ops.ssd_state_floats(H, P, N, G, taps), device=DEV)
        at, got = 0, []
        for k in cuts:
            got.append(run_ssd(rows[at:at + k], par, state, [k], [at], [0], H, P, N, G, dtype, 2))
            at += k
        close(torch.cat(got), want, dtype, 3.0)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n", [1, 9, 64, 130])
@pytest.mark.parametrize("d,ff,shared,E,top", [(40, 24, 16, 6, 2), (37, 9, 0, 5, 1), (256, 128, 384, 8, 3), (64, 72, 8, 4, 4)])
def test_weighed_input_experts_on_every_path(dtype, n, d, ff, shared, E, top):
    """Few rows (expert by expert, or pair by pair where rows are odd) and many rows (sorted, through the package's products)."""
    from rllm_b200.config.base import PartSpec
    from rllm_b200.parts import Runtime, build_part
    g = gen(11)
    dt = stored(dtype)
    part = build_part("ffn", PartSpec("routed_experts", {
        "hidden_size": d, "intermediate_size": ff, "num_experts": E, "top_k": top, "score": "sigmoid", "normalize": False,
        "activation": "relu2", "weigh_input": True, "shared_size": shared}, "m."), Runtime(torch.device(DEV), dt))
    w = {k: (torch.randn(s, generator=g) * (1.5 if "router" not in k else 3.0) / math.sqrt(s[-1])).to(dt)
         for k, (s, _) in part.expected_tensors().items()}
    part.load(w)
    h = torch.randn(n, d, generator=g).to(dt)
    idx, _, _ = part.route(h.to(DEV))
    want = pp.experts(h.double(), {k: v.double() for k, v in w.items()}, "m.", pc.moe(ff, E, top, shared),
                      {t: r for t, r in enumerate(idx.tolist())}, CLOSE[dtype])
    close(part.forward(h.to(DEV)), want, dt, 1.0)


# ---------------------------------------------------------------- whole models

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CASES))
def test_whole_prompt(name, dtype):
    cfg = CASES[name]
    w = pc.make_weights(cfg, 1, stored(dtype))
    toks = pc.tokens_for(cfg, 61, 1)
    ref = pc.oracle(cfg, w, toks)
    eng = pc.build_engine(cfg, w, dtype, max_tokens=128)
    out = run(eng, [([("a", toks, list(range(61)))], ["a"])])
    compare(out, {"a": ref}, dtype, name)
    assert not eng.cache.requests


@pytest.mark.parametrize("name", ["stack", "odd_sizes", "shared_keys", "heads64"])
def test_stream_after_every_layer(name):
    """float32: the residual stream behind every layer is the plain implementation's."""
    cfg = CASES[name]
    w = pc.make_weights(cfg, 2)
    toks = pc.tokens_for(cfg, 40, 2)
    streams = []
    pc.oracle(cfg, w, toks, streams)
    eng = pc.build_engine(cfg, w, "float32", max_tokens=64)
    seen = []
    for b in eng.model.blocks:
        def wrapped(x, pending, ctx, cache, _f=b.forward, **kw):
            out = _f(x, pending, ctx, cache, **kw)
            s = x.detach().double().cpu().clone()
            seen.append(s + out.double().cpu() if isinstance(out, torch.Tensor) else s)     # what the block still owes the stream
            return out
        b.forward = wrapped
    run(eng, [([("a", toks, [39])], ["a"])])
    assert len(seen) == len(streams) == len(cfg["layers"])
    for i, (got, want) in enumerate(zip(seen, streams)):
        assert float((got - want).abs().max()) < 2e-5 * float(want.abs().max()), i


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CASES))
def test_token_by_token_and_portions(name, dtype):
    """The same prompt token by token from the start, in portions of 7, 2, 5, 3, 2, 2, 19, then 2s, and most of it
    followed by single tokens: every row against the plain implementation."""
    cfg = CASES[name]
    w = pc.make_weights(cfg, 3, stored(dtype))
    toks = pc.tokens_for(cfg, 58, 3)
    ref = {"a": pc.oracle(cfg, w, toks)}
    eng = pc.build_engine(cfg, w, dtype, max_tokens=128)
    compare(run(eng, closing(one_by_one("a", toks), "a")), ref, dtype, name + " token by token")
    steps = [([("a", t, want)], []) for t, want in cut(toks, [7, 2, 5, 3, 2, 2, 19, 2])]
    compare(run(eng, closing(steps, "a")), ref, dtype, name + " in portions")
    steps = [([("a", toks[:33], [0, 32])], [])] + one_by_one("a", toks, 33)
    compare(run(eng, closing(steps, "a")), ref, dtype, name + " prompt then single tokens")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["stack", "stack_other_order", "heads64", "heads128", "odd_sizes", "shared_keys", "pair_wide_state"])
def test_unequal_requests_in_one_batch_with_reuse(name, dtype):
    """Four requests of 70, 9, 31 and 2 tokens, longer runs of one beside a decoded token of another, a fifth
    that takes over the pages and the slot of one that ended: every row is what the request gives alone."""
    cfg = CASES[name]
    w = pc.make_weights(cfg, 4, stored(dtype))
    lens = {"a": 70, "b": 9, "c": 31, "d": 2, "e": 26}
    T = {r: pc.tokens_for(cfg, n, 10 + i) for i, (r, n) in enumerate(lens.items())}
    refs = {r: pc.oracle(cfg, w, t) for r, t in T.items()}
    eng = pc.build_engine(cfg, w, dtype, max_tokens=192, max_requests=4)
    all_ = lambda k: list(range(k))
    steps = [
        ([("a", T["a"][:40], all_(40)), ("b", T["b"][:3], all_(3))], []),
        ([("a", T["a"][40:41], [0]), ("b", T["b"][3:9], all_(6)), ("c", T["c"][:17], all_(17)), ("d", T["d"][:2], all_(2))], ["b", "d"]),
        ([("c", T["c"][17:18], [0]), ("e", T["e"][:11], all_(11)), ("a", T["a"][41:43], all_(2))], []),
        ([("e", T["e"][11:26], all_(15)), ("a", T["a"][43:44], [0]), ("c", T["c"][18:19], [0])], ["e"]),
        ([("a", T["a"][44:70], all_(26)), ("c", T["c"][19:31], all_(12))], ["a", "c"]),
    ]
    compare(run(eng, steps), refs, dtype, name)
    assert not eng.cache.requests
    eng.cache.check_invariants()


def test_pages_and_slots_used_again_give_the_same_bits():
    """A request run alone in a fresh engine, and again in an engine whose pages and slots other requests
    have used and given back: the same bits."""
    cfg = CASES["stack"]
    w = pc.make_weights(cfg, 5)
    toks, other = pc.tokens_for(cfg, 45, 20), pc.tokens_for(cfg, 60, 21)
    steps = lambda r, t: closing([([(r, t[:30], list(range(30)))], [])] + one_by_one(r, t, 30), r)
    fresh = run(pc.build_engine(cfg, w, "float32", max_tokens=64, max_requests=2), steps("a", toks))
    eng = pc.build_engine(cfg, w, "float32", max_tokens=64, max_requests=2)
    run(eng, steps("x", other))
    run(eng, steps("y", other[::-1]))
    again = run(eng, steps("a", toks))
    for key, row in fresh.items():
        assert torch.equal(row, again[key]), key


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["sloped", "pair", "heads64", "heads128", "sloped_padded"])
def test_keys_at_the_windows_edges_decide_rows(name, dtype):
    """Marked attention in layer 0 with a sharp scale: the token `asker` asks for the keys of `target`.  A prompt in which an asker
    follows a target at every distance around the window (the last key inside, the first key outside, one further, the key
    right before), whole, in portions that cut the window, and decoded token by token across page borders: every row against the
    plain implementation, which itself changes by far more than the tolerance when that window is one key longer."""
    cfg = pc.sharpened(CASES[name], 6.0, layers=[0])
    first = next(pc.masks(cfg, [0]))
    window = first["mask"]["size"]
    asker, target = 5, 9
    w = pc.marked(cfg, pc.make_weights(cfg, 6, stored(dtype)), asker, target)
    toks = pc.tokens_for(cfg, 13 * window + 40, 30, avoid=(asker, target))
    asks, at = [], 3
    for dist in (window - 1, window, window + 1, 1, window - 1, window):     # the asker comes `dist` tokens behind
        toks[at] = target
        at += dist
        toks[at] = asker
        asks.append(at)
        at += window + 2                                                 # the next pair starts with a clean window
    toks = toks[:at]
    ref = pc.oracle(cfg, w, toks)
    off = pc.oracle(pc.with_windows(cfg, 1, [0]), w, toks)
    moved = [row_error(off[a], ref[a]) for a in asks]
    assert min(moved[1], moved[5]) > 3 * TOL[dtype], moved           # the key just outside would be seen
    eng = pc.build_engine(cfg, w, dtype, max_tokens=2 * len(toks), block_size=8)
    refs = {"a": ref}
    compare(run(eng, [([("a", toks, list(range(len(toks))))], ["a"])]), refs, dtype, "whole")
    steps = [([("a", t, want)], []) for t, want in cut(toks, [window - 2, 3, 2, window + 1, 5])]
    compare(run(eng, closing(steps, "a")), refs, dtype, "portions")
    compare(run(eng, closing([([("a", toks[:2], [0, 1])], [])] + one_by_one("a", toks, 2), "a")), refs, dtype, "decoded")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_layer_reads_shared_keys_far_behind_their_own_layers_window(dtype):
    """A layer without keys of its own sees everything, the layer whose keys it reads 8 keys: 400 tokens, long after the owner's window has
    passed the first pages, other requests take and give back pages meanwhile, decoded and in portions."""
    cfg = CASES["shared_keys_all"]
    w = pc.make_weights(cfg, 7, stored(dtype))
    toks, other = pc.tokens_for(cfg, 400, 33), pc.tokens_for(cfg, 90, 34)
    refs = {"a": pc.oracle(cfg, w, toks), "b": pc.oracle(cfg, w, other)}
    eng = pc.build_engine(cfg, w, dtype, max_tokens=512, block_size=8, max_requests=2)
    steps = [([("a", toks[:300], [0, 7, 8, 9, 150, 299])], []), ([("b", other, [0, 89])], ["b"]),
             ([("a", toks[300:360], [0, 59])], []), ([("b", other[:50], [49])], ["b"])] + one_by_one("a", toks, 360)
    compare(run(eng, closing(steps, "a")), refs, dtype, "longer reader")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_key_hundreds_of_places_back_through_the_latents(dtype):
    """Marked latents with a sharp scale: an asker 300 and 430 tokens behind the only target, in a prompt, in portions and
    decoded; the plain rows change by much more than the tolerance when the target is another token."""
    cfg = pc.sharpened(CASES["latents"], 5.0, layers=[0])
    asker, target = 5, 9
    w = pc.marked(cfg, pc.make_weights(cfg, 8, stored(dtype)), asker, target)
    toks = pc.tokens_for(cfg, 440, 35, avoid=(asker, target))
    toks[304] = toks[434] = asker
    without = list(toks)
    toks[4] = target
    ref, other = pc.oracle(cfg, w, toks), pc.oracle(cfg, w, without)
    assert min(row_error(other[p], ref[p]) for p in (304, 434)) > 4 * TOL[dtype]
    want = list(range(0, 440, 37)) + [303, 304, 305, 433, 434, 435]
    eng = pc.build_engine(cfg, w, dtype, max_tokens=512, block_size=16)
    refs = {"a": ref}
    compare(run(eng, [([("a", toks, want)], ["a"])]), refs, dtype, "whole")
    steps = [([("a", t, [0, len(t) - 1])], []) for t, _ in cut(toks, [290, 15, 2, 120, 8, 2, 3])]
    compare(run(eng, closing(steps, "a")), refs, dtype, "portions")
    compare(run(eng, closing([([("a", toks[:300], [299])], [])] + one_by_one("a", toks, 300), "a")), refs, dtype, "decoded")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["pair", "pair_wide_state"])
def test_a_token_hundreds_of_places_back_decides_rows_through_the_state(name, dtype):
    """The marked pair: one token near the start is all that the state holds 500 tokens later.  The prompt whole, in portions, and its
    last 60 tokens decoded: every row against the plain implementation, whose rows far behind the marker change by much more than
    the tolerance when the marker is another token."""
    cfg, marker = CASES[name], 7
    w = pc.marked_memory(cfg, pc.make_weights(cfg, 13, stored(dtype)), marker)
    toks = pc.tokens_for(cfg, 550, 80, avoid=(marker,))
    without = list(toks)
    toks[5] = marker
    ref, other = pc.oracle(cfg, w, toks), pc.oracle(cfg, w, without)
    moved = sorted(row_error(other[p], ref[p]) for p in range(300, 550))
    assert moved[len(moved) // 2] > 4 * TOL[dtype], moved[len(moved) // 2]
    want = list(range(8, 550, 41)) + list(range(500, 550))
    eng = pc.build_engine(cfg, w, dtype, max_tokens=1024, block_size=16)
    refs = {"a": ref}
    compare(run(eng, [([("a", toks, want)], ["a"])]), refs, dtype, "whole")
    steps = [([("a", t, [len(t) - 1])], []) for t, _ in cut(toks, [290, 2, 130, 7, 100, 21])]
    compare(run(eng, closing(steps, "a")), refs, dtype, "portions")
    compare(run(eng, closing([([("a", toks[:490], [489])], [])] + one_by_one("a", toks, 490), "a")), refs, dtype, "decoded")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["stack", "stack_other_order", "pair_wide_state"])
def test_the_first_tokens(name, dtype):
    """Requests of 1, 2, 3 and 5 tokens alone and together: the convolutions reach before the start of the sequence, the
    state is empty, the windows hold one key."""
    cfg = CASES[name]
    w = pc.make_weights(cfg, 8, stored(dtype))
    toks = {r: pc.tokens_for(cfg, n, 40 + n) for r, n in (("a", 1), ("b", 2), ("c", 3), ("d", 5))}
    refs = {r: pc.oracle(cfg, w, t) for r, t in toks.items()}
    eng = pc.build_engine(cfg, w, dtype, max_tokens=64)
    steps = [([(r, t, list(range(len(t)))) for r, t in toks.items()], list(toks))]
    compare(run(eng, steps), refs, dtype, "together")
    for r, t in toks.items():
        compare(run(eng, closing(one_by_one(r, t), r)), refs, dtype, "alone " + r)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_portions(dtype):
    """A prompt of 600 tokens in one step (the windows have long passed the first pages), the same in two steps of 351 and
    249, and 20 more tokens one by one."""
    cfg = CASES["stack"]
    w = pc.make_weights(cfg, 9, stored(dtype))
    toks = pc.tokens_for(cfg, 620, 50)
    refs = {"a": pc.oracle(cfg, w, toks)}
    want = list(range(0, 600, 37)) + [255, 256, 257, 599]
    eng = pc.build_engine(cfg, w, dtype, max_tokens=1024, block_size=16)
    steps = [([("a", toks[:600], want)], [])] + one_by_one("a", toks, 600)
    compare(run(eng, closing(steps, "a")), refs, dtype, "one step")
    steps = [([("a", toks[:351], [0, 300, 350])], []), ([("a", toks[351:600], [0, 100, 248])], [])] + one_by_one("a", toks, 600)
    compare(run(eng, closing(steps, "a")), refs, dtype, "two steps")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_through_graph_replay(dtype):
    """Two requests decode 150 tokens each after prompts of 20 and 3: replayed from CUDA graphs and launched
    one by one, both against the plain implementation (float32) and against each other."""
    cfg = CASES["stack_other_order"]
    w = pc.make_weights(cfg, 10, stored(dtype))
    toks = {"a": pc.tokens_for(cfg, 170, 60), "b": pc.tokens_for(cfg, 153, 61)}
    steps = [([("a", toks["a"][:20], [19]), ("b", toks["b"][:3], [2])], [])]
    steps += [([("a", [toks["a"][20 + i]], [0]), ("b", [toks["b"][3 + i]], [0])], []) for i in range(150)]
    outs = []
    for graphs in (True, False):
        eng = pc.build_engine(cfg, w, dtype, max_tokens=512, use_graphs=graphs)
        outs.append(run(eng, steps))
        if graphs:
            assert eng.stats["graph_replays"] > 100
    if dtype == "float32":
        refs = {r: pc.oracle(cfg, w, t) for r, t in toks.items()}
        compare(outs[0], refs, dtype, "replayed")
        compare(outs[1], refs, dtype, "launched")
    for key, row in outs[0].items():
        assert row_error(row, outs[1][key]) < (1e-6 if dtype == "float32" else 2e-2), key


REAL = pc.config([pc.sloped(8, 2, 128, 128, 100, 0.088, pc.moe(384, 16, 4, 512)), pc.latent(8, 128, 128, 384, 512, 0.088, pc.moe(256, 8, 2)),
                  pc.parallel((8, 2, 128, 128, 60, 0.088), (64, 10000.0), (16, 64, 128, 4, 4, 4), pc.moe(256, 8, 1, 256)),
                  pc.sloped(8, 2, 128, 128, 130, 0.088, None, 0)], width=1024, vocab=1531, scale=3.0)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_layer_sizes_of_a_real_model(dtype):
    """Width 1,024 and layers of real sizes: the products take the library, the tcgen05 and the weight-streaming
    kernels, attention the tensor-core kernels.  A prompt of 250 tokens, a portion of 40 beside another request's
    20, then single tokens of both."""
    cfg = REAL
    w = pc.make_weights(cfg, 16, stored(dtype), gain=1.0)
    toks = {"a": pc.tokens_for(cfg, 302, 70), "b": pc.tokens_for(cfg, 32, 71)}
    refs = {r: pc.oracle(cfg, w, t) for r, t in toks.items()}
    eng = pc.build_engine(cfg, w, dtype, max_tokens=512, block_size=32, max_requests=2)
    steps = [([("a", toks["a"][:250], list(range(0, 250, 23)) + [99, 100, 159, 160, 249])], []),
             ([("a", toks["a"][250:290], list(range(40))), ("b", toks["b"][:20], [0, 19])], [])]
    steps += [([("a", [toks["a"][290 + i]], [0]), ("b", [toks["b"][20 + i]], [0])], []) for i in range(12)]
    compare(run(eng, steps), refs, dtype, "real layer sizes")


# ---------------------------------------------------------------- the entry points a user calls

def write_folder(path, cfg, w):
    from rllm_b200.weights.safetensors_io import write_safetensors
    path.mkdir(exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(path / "model.safetensors", w)
    return path


def test_greedy_generation_through_the_scheduler(tmp_path):
    """LLM.generate (scheduler, continuous batching, prompts cut into portions of 16, device sampler)
    on a folder written in the stored format: the greedy continuation of each prompt is the plain
    implementation's."""
    from rllm_b200.llm import LLM
    cfg = CASES["stack"]
    w = pc.make_weights(cfg, 11)
    write_folder(tmp_path, cfg, w)
    prompts = [pc.tokens_for(cfg, n, 40 + i) for i, n in enumerate((37, 3, 21, 50, 9))]
    llm16 = LLM(str(tmp_path), dtype="bfloat16", ctx=128, block_size=8, prefill_chunk=16, parallel=3)
    got16 = llm16.generate(prompts, max_tokens=12, temperature=0.7, top_k=20, seed=5)
    assert all(len(g) == 12 and all(0 <= t < cfg["vocab"] for t in g) for g in got16)
    assert not llm16.engine.cache.requests
    del llm16
    llm = LLM(str(tmp_path), dtype="float32", ctx=128, block_size=8, prefill_chunk=16, parallel=3)
    got = llm.generate(prompts, max_tokens=12)
    checked = 0
    for p, g in zip(prompts, got):
        seq = list(p)
        for tok in g:
            logits = pc.oracle(cfg, w, seq)[-1]
            top2 = torch.topk(logits, 2).values
            if float(top2[0] - top2[1]) < 1e-4:       # a tie at float32 precision decides nothing
                break
            assert int(logits.argmax()) == tok
            seq.append(tok)
            checked += 1
    assert all(len(g) == 12 for g in got) and checked > 40
    assert not llm.engine.cache.requests


def test_trace_replay_program_chooses_the_model_by_its_config(tmp_path):
    """bin/trace_run on a Pibavik folder: steps from standard input, rows out as little-endian float32; two
    requests share the steps, one pauses, pages and slots go back at the end."""
    import subprocess
    import sys
    from pathlib import Path
    import numpy as np
    cfg = CASES["stack_other_order"]
    w = pc.make_weights(cfg, 12, torch.bfloat16)
    model = write_folder(tmp_path / "model", cfg, w)
    toks, other = pc.tokens_for(cfg, 30, 6), pc.tokens_for(cfg, 9, 7)
    lines = [json.dumps({"step": 0, "entries": [{"id": "x", "tokens": toks[:20], "want": [0, 19]}], "end": []}),
             json.dumps({"step": 1, "entries": [{"id": "y", "tokens": other[:8], "want": []}], "end": []}),
             json.dumps({"step": 2, "entries": [{"id": "x", "tokens": toks[20:], "want": [9]},
                                                {"id": "y", "tokens": other[8:], "want": [0]}], "end": ["x", "y"]})]
    root = Path(__file__).resolve().parent.parent
    proc = subprocess.run([sys.executable, str(root / "bin" / "trace_run"), "--model", str(model), "--dtype", "float32",
                           "--out", str(tmp_path / "out"), "--max-tokens", "128"], input="\n".join(lines) + "\n",
                          capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    rows = torch.from_numpy(np.fromfile(tmp_path / "out" / "0.f32", dtype="<f4").reshape(2, cfg["vocab"]))
    ref, ref_other = pc.oracle(cfg, w, toks), pc.oracle(cfg, w, other)
    assert row_error(rows[0], ref[0]) < TOL["float32"] and row_error(rows[1], ref[19]) < TOL["float32"]
    assert not (tmp_path / "out" / "1.f32").exists()
    rows = torch.from_numpy(np.fromfile(tmp_path / "out" / "2.f32", dtype="<f4").reshape(2, cfg["vocab"]))
    assert row_error(rows[0], ref[29]) < TOL["float32"] and row_error(rows[1], ref_other[8]) < TOL["float32"]


def test_random_weights_mode_writes_a_folder_the_engine_loads(tmp_path):
    """The package's own random-weights mode knows the design's tensors."""
    from rllm_b200.config import config_from_dict
    from rllm_b200.models.model import load_model
    from rllm_b200.weights import write_random_model
    write_random_model(config_from_dict(CASES["stack"]), tmp_path, seed=3, dtype=torch.bfloat16)
    cfg, model = load_model(tmp_path, "bfloat16", DEV)
    assert cfg.to_dict() == CASES["stack"] and model.loaded
    from rllm_b200.engine import Engine, StepItem
    eng = Engine(model, block_size=16, max_tokens=64, max_requests=2)
    logits = eng.step([StepItem("a", [1, 2, 3, 4, 5], [4])])
    assert logits.shape == (1, CASES["stack"]["vocab"]) and bool(torch.isfinite(logits).all())
