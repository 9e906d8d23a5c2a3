"""Rusolorn through the engine against the plain implementation (tests/plain_rusolorn.py, float64).

Each new kernel alone against its formula; each mechanism as a small model; whole prompts against
token-by-token decoding; portions down to two tokens; batches of unequal requests against each alone with
pages and state slots used again; keys just inside and just outside every window, in prompts and in
decoding, with weights at which one key decides a row and a check that a window that is one key off would
show; a token hundreds of places back that decides rows through the delta rule's memory; the first tokens of
a sequence (inside the reach of the convolutions); long portions; long decoding through CUDA-graph replay; head
sizes the tensor-core kernels take; layer sizes of a real model; greedy generation through ``LLM.generate`` and
the scheduler; ``bin/trace_run``; the random-weights mode.  The configurations and weights are made in
tests/rusolorn_cases.py.
"""
import json
import math

import pytest
import torch

import plain_rusolorn as pr
import rusolorn_cases as rc
from rusolorn_cases import CASES, row_error

pytestmark = pytest.mark.gpu

# max |engine - plain| / max |plain| over a logits row (means taken off).  float32: the engine sums in another
# order than the float64 plain implementation.  bfloat16: weights, the operands of every product and the cache are
# rounded to 8 bits of mantissa; how much that alone moves a row differs from row to row (a head of the memory and
# both sides' outputs are divided by their root mean square), so a row's tolerance is this one plus three times
# what rounding the sublayers' inputs and outputs does to the row in the plain implementation
# (`oracle(...).noise`), and one row in fifty may pass it by less than a factor of two.  A lost key, state or
# token moves many rows, by more; the float32 runs of the same tests see it at 1e-4.
TOL = {"float32": 1e-4, "bfloat16": 3e-2}
STRAY = {"float32": 0, "bfloat16": 50}
# A token whose choice of experts hangs on less than this gap between scores may take another expert when the
# router's input carries the rounding of the mode.  Where the plain router's choice hangs on less than this, the
# comparison takes the engine's experts over if they are what it gives itself after moving every score by at most
# this much.
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
@pytest.mark.parametrize("n,d", [(7, 50), (3, 1028), (200, 264)])
def test_dynamic_tanh_kernel(dtype, n, d):
    """With and without a delta that joins first, with and without a gather of rows."""
    from rllm_b200.csrc import ops
    g = gen(1)
    x, delta = torch.randn(n, d, generator=g) * 3, torch.randn(n, d, generator=g)
    w, b = 1 + 0.3 * torch.randn(d, generator=g), torch.randn(d, generator=g)
    out = torch.empty(n, d, dtype=dtype, device=DEV)
    ops.dyt_rows(x.to(DEV), 0.4, w.to(DEV), b.to(DEV), out)
    close(out, pr.dyt(x.double(), 0.4, w.double(), b.double()), dtype)
    xd = x.to(DEV)
    ops.dyt_rows(xd, 0.4, w.to(DEV), b.to(DEV), out, delta=delta.to(DEV), delta_scale=0.7)
    close(xd, x.double() + 0.7 * delta.double(), torch.float32)
    close(out, pr.dyt(x.double() + 0.7 * delta.double(), 0.4, w.double(), b.double()), dtype)
    rows = [n - 1, 0, n // 2]
    few = torch.empty(3, d, dtype=dtype, device=DEV)
    ops.dyt_rows(x.to(DEV), -1.3, w.to(DEV), b.to(DEV), few, rows=i32(rows))
    close(few, pr.dyt(x.double()[rows], -1.3, w.double(), b.double()), dtype)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,d", [(5, 36), (3, 1024), (150, 2056), (4, 4095), (2, 8200)])
def test_two_normed_outputs_and_a_third_join_the_stream(dtype, n, d):
    from rllm_b200.csrc import ops
    g = gen(2)
    a, b, c, x = (torch.randn(n, d, generator=g) * s for s in (2.0, 0.1, 1.0, 3.0))
    wa, wb = 1 + 0.3 * torch.randn(d, generator=g), 1 + 0.3 * torch.randn(d, generator=g)
    to = lambda t: t.to(DEV)
    na, nb = pr.rms(a.double(), 1e-5) * wa.double(), pr.rms(b.double(), 1e-2) * wb.double()
    xd, low = to(x), torch.empty(n, d, dtype=dtype, device=DEV)
    ops.join_sum_rows(to(a), xd, 0.6, norm_a=(to(wa), 1e-5), scale_a=0.5, b=to(b), norm_b=(to(wb), 1e-2), scale_b=0.25, c=to(c), low=low)
    want = x.double() + 0.6 * (0.5 * na + 0.25 * nb + c.double())
    close(xd, want, torch.float32)
    close(low, want, dtype)
    xd = to(x)
    ops.join_sum_rows(to(a), xd, 1.5, norm_a=(to(wa), 1e-5))                      # one output alone
    close(xd, x.double() + 1.5 * na, torch.float32)
    xd = to(x)
    ops.join_sum_rows(to(a), xd, 2.0, add=False, scale_a=0.5, b=to(b), norm_b=(to(wb), 1e-2))      # written, not added
    close(xd, 2.0 * (0.5 * a.double() + nb), torch.float32)
    wide = torch.randn(n, d + 8, generator=g)
    xd = to(x)
    ops.join_sum_rows(to(a), xd, 1.0, c=to(wide)[:, 4:4 + d], low=low)            # columns of a wider matrix
    close(xd, x.double() + a.double() + wide.double()[:, 4:4 + d], torch.float32)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,d", [(5, 36), (3, 1024), (150, 2056), (4, 4095), (2, 8200)])
def test_normed_rows_join_and_the_next_dynamic_tanh(dtype, n, d):
    from rllm_b200.csrc import ops
    g = gen(3)
    y, x = torch.randn(n, d, generator=g) * 0.2, torch.randn(n, d, generator=g) * 2
    wy, w, b = (1 + 0.3 * torch.randn(d, generator=g) for _ in range(3))
    to = lambda t: t.to(DEV)
    xd, out = to(x), torch.empty(n, d, dtype=dtype, device=DEV)
    ops.join_dyt_rows(to(y), (to(wy), 1e-3), 0.7, xd, 0.45, to(w), to(b), out)
    want = x.double() + 0.7 * pr.rms(y.double(), 1e-3) * wy.double()
    close(xd, want, torch.float32)
    close(out, pr.dyt(want, 0.45, w.double(), b.double()), dtype)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,dim,padded", [(5, 3, 8), (70, 24, 24), (1, 257, 264)])
def test_token_gate_kernel(dtype, n, dim, padded):
    from rllm_b200.csrc import ops
    g = gen(4)
    z = torch.randn(n, padded + 4, generator=g) * 2
    table = torch.randn(31, dim, generator=g).to(dtype)
    toks = [int(t) for t in torch.randint(0, 31, (n,), generator=g)]
    out = torch.full((n, padded), float("nan"), dtype=dtype, device=DEV)
    ops.token_gate(z.to(DEV)[:, :padded], table.to(DEV), i32(toks), out, dim)
    close(out[:, :dim], pr.gelu_tanh(z[:, :dim].double()) * table.double()[toks], dtype)
    assert not out[:, dim:].any()


@pytest.mark.parametrize("H,G,dk,bs", [(3, 1, 10, 8), (4, 2, 16, 16), (2, 2, 64, 8)])
def test_row_norm_store_with_the_keys_as_values(H, G, dk, bs):
    """Queries and keys normed over the whole row, the values the key columns as projected."""
    from rllm_b200.csrc import ops
    g = gen(5)
    n = 11
    rows = torch.randn(n, (H + G) * dk + 6, generator=g)
    qw, kw = 1 + 0.3 * torch.randn(H * dk, generator=g), 1 + 0.3 * torch.randn(G * dk, generator=g)
    slots = [int(s) for s in torch.randperm(4 * bs, generator=g)[:n]]
    slots[3] = -1
    q = torch.empty(n, H * dk, device=DEV)
    kc, vc = torch.zeros(4, G, bs, dk, device=DEV), torch.zeros(4, G, bs, dk, device=DEV)
    ops.qkv_rownorm_store(rows.to(DEV)[:, :(H + G) * dk], None, qw.to(DEV), kw.to(DEV), i32(slots), q, kc, vc, H, G, dk, dk, bs, 1e-5,
                          v_tied=True)
    rd = rows.double()
    close(q, pr.rms(rd[:, :H * dk], 1e-5) * qw.double(), torch.float32)
    raw = rd[:, H * dk:(H + G) * dk]
    kn = pr.rms(raw, 1e-5) * kw.double()
    for t, s in enumerate(slots):
        if s >= 0:
            close(kc[s // bs, :, s % bs].reshape(-1), kn[t], torch.float32)
            close(vc[s // bs, :, s % bs].reshape(-1), raw[t], torch.float32)
    written = {s for s in slots if s >= 0}
    assert all(not kc[s // bs, :, s % bs].any() for s in range(4 * bs) if s not in written)


def delta_inputs(H, G, dk, dv, taps, n, seed):
    """Projection rows with room behind them, the parameters, and the plain rule on any run of rows."""
    g = gen(seed)
    widths = {"q": G * dk, "k": G * dk, "v": H * dv, "g": H * dv, "b": H, "a": H}
    offs, at = {}, 0
    for s, c in widths.items():
        offs[s] = at
        at += c
    rows = torch.randn(n, at + 3, generator=g)
    par = {s + ".conv": torch.randn(widths[s], taps, generator=g) * 0.6 for s in "qkv"}
    par.update(A_log=0.7 * torch.randn(H, generator=g), dt_bias=-2 + torch.randn(H, generator=g),
               norm=1 + 0.3 * torch.randn(dv, generator=g))
    eye = torch.eye(at + 3, dtype=torch.float64)
    w = {s: eye[offs[s]:offs[s] + c] for s, c in widths.items()}
    w.update({k: v.double() for k, v in par.items()}, o=torch.eye(H * dv, dtype=torch.float64))
    mx = {"heads": H, "kv_heads": G, "dim": dk, "vdim": dv}
    return rows, offs, par, lambda x: pr.gated_delta(x.double(), w, "", mx, 1e-5)


def run_delta(rows, offs, par, state, lens, slots, H, G, dk, dv, dtype, max_q=None):
    from rllm_b200.csrc import ops
    n = sum(lens)
    out = torch.empty(n, H * dv, dtype=dtype, device=DEV)
    cu = [0]
    for k in lens:
        cu.append(cu[-1] + k)
    conv = torch.cat([par[s + ".conv"] for s in "qkv"], 0).to(DEV)
    ops.gated_delta(rows.to(DEV), tuple(offs[s] for s in "qkvgba"), conv, torch.exp(par["A_log"]).to(DEV), par["dt_bias"].to(DEV),
                    par["norm"].to(DEV), dk ** -0.5, 1e-6, 1e-5, state, i32(cu), i32(slots), out, len(lens), max_q or max(lens), H, G,
                    dk, dv)
    return out


DELTA_SIZES = [(3, 3, 8, 20, 4), (4, 2, 16, 8, 3), (2, 1, 24, 16, 2), (2, 2, 32, 24, 1), (1, 1, 40, 12, 6), (5, 1, 33, 13, 2), (2, 1, 64, 32, 4),
               (2, 2, 128, 128, 4), (4, 2, 128, 64, 4), (2, 1, 136, 40, 4), (2, 2, 20, 168, 4), (1, 1, 5, 3, 9), (2, 1, 300, 24, 3), (1, 1, 8, 300, 4)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,dk,dv,taps", DELTA_SIZES)
def test_gated_delta_kernels(dtype, H, G, dk, dv, taps):
    """Three requests' rows through both ways (chunks, and token by token), in cuts of all kinds (inside a chunk, shorter
    than the convolution's reach, one token), the states in slots that are not in order and hold garbage elsewhere."""
    from rllm_b200.csrc import ops
    lens = {"a": 61, "b": 8, "c": 17}
    data = {r: delta_inputs(H, G, dk, dv, taps, n, 6) for r, n in lens.items()}
    rows, offs, par, plain = data["a"]
    rows = {r: torch.randn(n, rows.shape[1], generator=gen(60 + i)) for i, (r, n) in enumerate(lens.items())}
    want = {r: plain(x) for r, x in rows.items()}
    slot = {"a": 3, "b": 0, "c": 2}
    plans = [[("a", 61), ("b", 8), ("c", 17)], "next", [("a", 30), ("c", 1)], [("b", 3), ("a", 9), ("c", 9)], [("a", 2)], [("c", 7), ("a", 20), ("b", 5)],
             "next", [("a", 1), ("b", 2)], [("a", 8), ("b", 1)], [("a", 3), ("c", 4), ("b", 5)], [("a", 49), ("c", 13)]]
    per = ops.delta_state_floats(H, dk, dv, taps)
    state = torch.randn(5, per, device=DEV)
    at = {}
    for step in plans + ["next"]:
        if step == "next":
            at = {}
            continue
        for r, _ in step:
            if r not in at:
                at[r] = 0
                state[slot[r]].zero_()
        x = torch.cat([rows[r][at[r]:at[r] + k] for r, k in step])
        out = run_delta(x, offs, par, state, [k for _, k in step], [slot[r] for r, _ in step], H, G, dk, dv, dtype)
        i = 0
        for r, k in step:
            close(out[i:i + k], want[r][at[r]:at[r] + k], dtype, 3.0 if dtype == torch.float32 else 1.0)
            at[r] += k
            i += k


@pytest.mark.parametrize("H,G,dk,dv,taps", [(4, 2, 16, 24, 4), (2, 2, 128, 128, 4), (3, 1, 40, 20, 3)])
def test_gated_delta_chunks_against_tokens_on_the_same_state(H, G, dk, dv, taps):
    """300 rows in one portion and the same rows token by token leave the same state and outputs, up to rounding."""
    from rllm_b200.csrc import ops
    rows, offs, par, _ = delta_inputs(H, G, dk, dv, taps, 300, 8)
    per = ops.delta_state_floats(H, dk, dv, taps)
    a, b = torch.zeros(1, per, device=DEV), torch.zeros(1, per, device=DEV)
    one = run_delta(rows, offs, par, a, [300], [0], H, G, dk, dv, torch.float32)
    two = torch.cat([run_delta(rows[i:i + 4], offs, par, b, [4], [0], H, G, dk, dv, torch.float32) for i in range(0, 300, 4)])
    close(one, two.double().cpu(), torch.float32, 3.0)
    close(a, b.double().cpu(), torch.float32, 3.0)


def test_gated_delta_decays_of_every_size_in_one_chunk():
    """Step sizes from nothing to hundreds: a token that wipes the memory beside tokens that keep it (the chunk's decays
    are products, never quotients), in a chunk and token by token."""
    H, G, dk, dv, taps = 2, 1, 16, 12, 4
    rows, offs, par, plain = delta_inputs(H, G, dk, dv, taps, 40, 9)
    rows[:, offs["a"]:offs["a"] + H] = -8.0
    for t in (3, 4, 11, 23):
        rows[t, offs["a"]:offs["a"] + H] = torch.tensor([300.0, 40.0])
    want = plain(rows)
    from rllm_b200.csrc import ops
    for cuts in ([40], [4] * 10):
        state = torch.zeros(1, ops.delta_state_floats(H, dk, dv, taps), device=DEV)
        at, got = 0, []
        for k in cuts:
            got.append(run_delta(rows[at:at + k], offs, par, state, [k], [0], H, G, dk, dv, torch.float32))
            at += k
        close(torch.cat(got), want, torch.float32, 3.0)


@pytest.mark.parametrize("E,top,count,keep", [(8, 3, 4, 2), (12, 4, 3, 1), (6, 2, 6, 3), (9, 9, 3, 3), (10, 1, 1, 1), (64, 6, 8, 4)])
def test_router_kernel_with_the_largest_score_of_a_group(E, top, count, keep):
    from rllm_b200.csrc import ops
    g = gen(10)
    z = torch.randn(90, E, generator=g) * 3
    idx, wt = torch.empty(90, top, dtype=torch.int32, device=DEV), torch.empty(90, top, device=DEV)
    ops.moe_route(z.to(DEV), None, idx, wt, E, top, count, keep, 1, "softmax", True, 1e-20, 1.0)
    s = torch.softmax(z.double(), -1)
    for t in range(90):
        want, margin = pr.choose(s[t], top, count, keep)
        if margin < 1e-6:
            continue
        got = idx[t].tolist()
        assert got == want
        assert torch.allclose(wt[t].double().cpu(), s[t, got] / s[t, got].sum(), atol=1e-5)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n", [1, 9, 64, 130])
@pytest.mark.parametrize("d,ff,shared", [(40, 24, 16), (37, 9, 11), (256, 128, 384)])
def test_clamped_experts_on_every_path(dtype, n, d, ff, shared):
    """Few rows (expert by expert, or pair by pair where rows are odd) and many rows (sorted, through the package's
    products): limits of their own for the experts and the shared one, which bite."""
    from rllm_b200.config.base import PartSpec
    from rllm_b200.parts import Runtime, build_part
    g = gen(11)
    dt = stored(dtype)
    mlp = rc.moe(ff, 6, 2, (3, 2), (shared, 2.0), 0.7)
    form = lambda l: {"limit": l, "alpha": 1.702, "shift": 1.0}
    part = build_part("ffn", PartSpec("routed_experts", {
        "hidden_size": d, "intermediate_size": ff, "num_experts": 6, "top_k": 2, "n_groups": 3, "keep_groups": 2, "group_best": 1,
        "score": "softmax", "normalize": True, "weight_eps": 1e-20, "expert_form": form(0.7), "shared_size": shared,
        "shared_form": form(2.0)}, "m."), Runtime(torch.device(DEV), dt))
    w = {k: (torch.randn(s, generator=g) * (2.0 if "router" not in k else 6.0) / math.sqrt(s[-1])).to(dt)
         for k, (s, _) in part.expected_tensors().items()}
    part.load(w)
    h = torch.randn(n, d, generator=g).to(dt)
    idx, _, _ = part.route(h.to(DEV))
    want = pr.experts(h.double(), {k: v.double() for k, v in w.items()}, "m.", mlp,
                      {t: r for t, r in enumerate(idx.tolist())}, CLOSE[dtype])
    close(part.forward(h.to(DEV)), want, dt, 1.0)


# ---------------------------------------------------------------- whole models

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CASES))
def test_whole_prompt(name, dtype):
    cfg = CASES[name]
    w = rc.make_weights(cfg, 1, stored(dtype))
    toks = rc.tokens_for(cfg, 61, 1)
    ref = rc.oracle(cfg, w, toks)
    eng = rc.build_engine(cfg, w, dtype, max_tokens=128)
    out = run(eng, [([("a", toks, list(range(61)))], ["a"])])
    compare(out, {"a": ref}, dtype, name)
    assert not eng.cache.requests


@pytest.mark.parametrize("name", ["stack", "odd_sizes", "mixers_alone"])
def test_stream_after_every_layer(name):
    """float32: the residual stream behind every layer is the plain implementation's."""
    cfg = CASES[name]
    w = rc.make_weights(cfg, 2)
    toks = rc.tokens_for(cfg, 40, 2)
    streams = []
    rc.oracle(cfg, w, toks, streams)
    eng = rc.build_engine(cfg, w, "float32", max_tokens=64)
    seen = []
    for b in eng.model.blocks:
        def wrapped(x, pending, ctx, cache, _f=b.forward, **kw):
            out = _f(x, pending, ctx, cache, **kw)
            seen.append(x.detach().double().cpu().clone())
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
    w = rc.make_weights(cfg, 3, stored(dtype))
    toks = rc.tokens_for(cfg, 58, 3)
    ref = {"a": rc.oracle(cfg, w, toks)}
    eng = rc.build_engine(cfg, w, dtype, max_tokens=128)
    compare(run(eng, closing(one_by_one("a", toks), "a")), ref, dtype, name + " token by token")
    steps = [([("a", t, want)], []) for t, want in cut(toks, [7, 2, 5, 3, 2, 2, 19, 2])]
    compare(run(eng, closing(steps, "a")), ref, dtype, name + " in portions")
    steps = [([("a", toks[:33], [0, 32])], [])] + one_by_one("a", toks, 33)
    compare(run(eng, closing(steps, "a")), ref, dtype, name + " prompt then single tokens")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["stack", "stack_other_order", "heads64", "heads128", "odd_sizes", "one_layer"])
def test_unequal_requests_in_one_batch_with_reuse(name, dtype):
    """Four requests of 70, 9, 31 and 2 tokens, longer runs of one beside a decoded token of another, a fifth
    that takes over the pages and the slot of one that ended: every row is what the request gives alone."""
    cfg = CASES[name]
    w = rc.make_weights(cfg, 4, stored(dtype))
    lens = {"a": 70, "b": 9, "c": 31, "d": 2, "e": 26}
    T = {r: rc.tokens_for(cfg, n, 10 + i) for i, (r, n) in enumerate(lens.items())}
    refs = {r: rc.oracle(cfg, w, t) for r, t in T.items()}
    eng = rc.build_engine(cfg, w, dtype, max_tokens=192, max_requests=4)
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
    w = rc.make_weights(cfg, 5)
    toks, other = rc.tokens_for(cfg, 45, 20), rc.tokens_for(cfg, 60, 21)
    steps = lambda r, t: closing([([(r, t[:30], list(range(30)))], [])] + one_by_one(r, t, 30), r)
    fresh = run(rc.build_engine(cfg, w, "float32", max_tokens=64, max_requests=2), steps("a", toks))
    eng = rc.build_engine(cfg, w, "float32", max_tokens=64, max_requests=2)
    run(eng, steps("x", other))
    run(eng, steps("y", other[::-1]))
    again = run(eng, steps("a", toks))
    for key, row in fresh.items():
        assert torch.equal(row, again[key]), key


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["one_layer", "groups_of_one", "heads64", "heads128"])
def test_keys_at_the_windows_edges_decide_rows(name, dtype):
    """The marked attention side with a sharp scale: the token `asker` asks for the keys of `target`.  A prompt in
    which an asker follows a target at every distance around the window (the last key inside, the first key outside,
    one further, the key right before), whole, in portions that cut the window, and decoded token by token across page
    borders: every row against the plain implementation, which itself changes by far more than the tolerance when
    its windows are one key longer."""
    cfg = rc.sharpened(CASES[name], 6.0, layers=[0])
    cfg["embedding"]["scale"] = 4.0
    window = cfg["layers"][0]["mixer"]["left"]["mask"]["size"]
    asker, target = 5, 9
    w = rc.marked_attention(cfg, rc.make_weights(cfg, 6, stored(dtype)), asker, target)
    toks = rc.tokens_for(cfg, 13 * window + 40, 30, avoid=(asker, target))
    asks, at = [], 3
    for dist in (window - 1, window, window + 1, 1, window - 1, window):     # the asker comes `dist` tokens behind
        toks[at] = target
        at += dist
        toks[at] = asker
        asks.append(at)
        at += window + 2                                                 # the next pair starts with a clean window
    toks = toks[:at]
    ref = rc.oracle(cfg, w, toks)
    off = rc.oracle(rc.with_windows(cfg, 1), w, toks)
    moved = [row_error(off[a], ref[a]) for a in asks]
    assert min(moved[1], moved[5]) > 1.5 * TOL[dtype], moved           # the key just outside would be seen
    eng = rc.build_engine(cfg, w, dtype, max_tokens=2 * len(toks), block_size=8)
    refs = {"a": ref}
    compare(run(eng, [([("a", toks, list(range(len(toks))))], ["a"])]), refs, dtype, "whole")
    steps = [([("a", t, want)], []) for t, want in cut(toks, [window - 2, 3, 2, window + 1, 5])]
    compare(run(eng, closing(steps, "a")), refs, dtype, "portions")
    compare(run(eng, closing([([("a", toks[:2], [0, 1])], [])] + one_by_one("a", toks, 2), "a")), refs, dtype, "decoded")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["one_layer", "wide_keys", "heads64"])
def test_a_token_hundreds_of_places_back_decides_rows_through_the_memory(name, dtype):
    """The marked delta side: one token near the start is all that the memory holds 500 tokens later.  The prompt whole, in
    portions, and its last 60 tokens decoded: every row against the plain implementation, whose rows far behind the
    marker change by much more than the tolerance when the marker is another token."""
    cfg = copy_with_scale(CASES[name], 1.0)
    marker = 7
    w = rc.marked_delta(cfg, rc.make_weights(cfg, 13, stored(dtype)), marker)
    toks = rc.tokens_for(cfg, 550, 80, avoid=(marker,))
    without = list(toks)
    toks[5] = marker
    ref, other = rc.oracle(cfg, w, toks), rc.oracle(cfg, w, without)
    moved = sorted(row_error(other[p], ref[p]) for p in range(300, 550))
    assert moved[len(moved) // 2] > 4 * TOL[dtype], moved[len(moved) // 2]
    want = list(range(8, 550, 41)) + list(range(500, 550))
    eng = rc.build_engine(cfg, w, dtype, max_tokens=1024, block_size=16)
    refs = {"a": ref}
    compare(run(eng, [([("a", toks, want)], ["a"])]), refs, dtype, "whole")
    steps = [([("a", t, [len(t) - 1])], []) for t, _ in cut(toks, [290, 2, 130, 7, 100, 21])]
    compare(run(eng, closing(steps, "a")), refs, dtype, "portions")
    compare(run(eng, closing([([("a", toks[:490], [489])], [])] + one_by_one("a", toks, 490), "a")), refs, dtype, "decoded")


def copy_with_scale(cfg, scale):
    return dict(cfg, embedding={"scale": scale})


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["stack", "stack_other_order", "groups_of_one"])
def test_the_first_tokens(name, dtype):
    """Requests of 1, 2, 3 and 5 tokens alone and together: the convolutions reach before the start of the sequence, the
    memory is empty, the window holds one key."""
    cfg = CASES[name]
    w = rc.make_weights(cfg, 8, stored(dtype))
    toks = {r: rc.tokens_for(cfg, n, 40 + n) for r, n in (("a", 1), ("b", 2), ("c", 3), ("d", 5))}
    refs = {r: rc.oracle(cfg, w, t) for r, t in toks.items()}
    eng = rc.build_engine(cfg, w, dtype, max_tokens=64)
    steps = [([(r, t, list(range(len(t)))) for r, t in toks.items()], list(toks))]
    compare(run(eng, steps), refs, dtype, "together")
    for r, t in toks.items():
        compare(run(eng, closing(one_by_one(r, t), r)), refs, dtype, "alone " + r)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_portions(dtype):
    """A prompt of 700 tokens in one step (the windows have long passed the first pages), the same in two steps of 411 and
    289, and 20 more tokens one by one."""
    cfg = CASES["stack"]
    w = rc.make_weights(cfg, 9, stored(dtype))
    toks = rc.tokens_for(cfg, 720, 50)
    refs = {"a": rc.oracle(cfg, w, toks)}
    want = list(range(0, 700, 37)) + [255, 256, 257, 699]
    eng = rc.build_engine(cfg, w, dtype, max_tokens=1024, block_size=16)
    steps = [([("a", toks[:700], want)], [])] + one_by_one("a", toks, 700)
    compare(run(eng, closing(steps, "a")), refs, dtype, "one step")
    steps = [([("a", toks[:411], [0, 300, 410])], []), ([("a", toks[411:700], [0, 100, 288])], [])] + one_by_one("a", toks, 700)
    compare(run(eng, closing(steps, "a")), refs, dtype, "two steps")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_through_graph_replay(dtype):
    """Two requests decode 150 tokens each after prompts of 20 and 3: replayed from CUDA graphs and launched
    one by one, both against the plain implementation (float32) and against each other."""
    cfg = CASES["stack_other_order"]
    w = rc.make_weights(cfg, 10, stored(dtype))
    toks = {"a": rc.tokens_for(cfg, 170, 60), "b": rc.tokens_for(cfg, 153, 61)}
    steps = [([("a", toks["a"][:20], [19]), ("b", toks["b"][:3], [2])], [])]
    steps += [([("a", [toks["a"][20 + i]], [0]), ("b", [toks["b"][3 + i]], [0])], []) for i in range(150)]
    outs = []
    for graphs in (True, False):
        eng = rc.build_engine(cfg, w, dtype, max_tokens=512, use_graphs=graphs)
        outs.append(run(eng, steps))
        if graphs:
            assert eng.stats["graph_replays"] > 100
    if dtype == "float32":
        refs = {r: rc.oracle(cfg, w, t) for r, t in toks.items()}
        compare(outs[0], refs, dtype, "replayed")
        compare(outs[1], refs, dtype, "launched")
    for key, row in outs[0].items():
        assert row_error(row, outs[1][key]) < (1e-6 if dtype == "float32" else 2e-2), key


REAL = rc.config([rc.layer((8, 2, 128, 100, 0.1), (8, 4, 64, 128, 4), rc.moe(256, 32, 4, (8, 4), (512, 1.8))),
                  rc.layer((12, 4, 64, 33, 0.15), (6, 6, 128, 96, 4), rc.moe(384, 8, 2, None, None))], width=1024, vocab=1531, side=72,
                 scale=5.0)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_layer_sizes_of_a_real_model(dtype):
    """Width 1,024 and layers of real sizes: the products take the library, the tcgen05 and the weight-streaming
    kernels, attention the tensor-core kernels.  A prompt of 300 tokens, a portion of 40 beside another request's
    20, then single tokens of both."""
    cfg = REAL
    w = rc.make_weights(cfg, 16, stored(dtype), gain=1.0)
    toks = {"a": rc.tokens_for(cfg, 352, 70), "b": rc.tokens_for(cfg, 32, 71)}
    refs = {r: rc.oracle(cfg, w, t) for r, t in toks.items()}
    eng = rc.build_engine(cfg, w, dtype, max_tokens=512, block_size=32, max_requests=2)
    steps = [([("a", toks["a"][:300], list(range(0, 300, 23)) + [99, 100, 159, 160, 299])], []),
             ([("a", toks["a"][300:340], list(range(40))), ("b", toks["b"][:20], [0, 19])], [])]
    steps += [([("a", [toks["a"][340 + i]], [0]), ("b", [toks["b"][20 + i]], [0])], []) for i in range(12)]
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
    w = rc.make_weights(cfg, 11)
    write_folder(tmp_path, cfg, w)
    prompts = [rc.tokens_for(cfg, n, 40 + i) for i, n in enumerate((37, 3, 21, 50, 9))]
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
            logits = rc.oracle(cfg, w, seq)[-1]
            top2 = torch.topk(logits, 2).values
            if float(top2[0] - top2[1]) < 1e-4:       # a tie at float32 precision decides nothing
                break
            assert int(logits.argmax()) == tok
            seq.append(tok)
            checked += 1
    assert all(len(g) == 12 for g in got) and checked > 40
    assert not llm.engine.cache.requests


def test_trace_replay_program_chooses_the_model_by_its_config(tmp_path):
    """bin/trace_run on a Rusolorn folder: steps from standard input, rows out as little-endian float32; two
    requests share the steps, one pauses, pages and slots go back at the end."""
    import subprocess
    import sys
    from pathlib import Path
    import numpy as np
    cfg = CASES["stack_other_order"]
    w = rc.make_weights(cfg, 12, torch.bfloat16)
    model = write_folder(tmp_path / "model", cfg, w)
    toks, other = rc.tokens_for(cfg, 30, 6), rc.tokens_for(cfg, 9, 7)
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
    ref, ref_other = rc.oracle(cfg, w, toks), rc.oracle(cfg, w, other)
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
