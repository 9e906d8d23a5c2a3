"""The gated delta rule behind short causal convolutions: linear attention whose memory is decayed by one
number per head and token and corrected towards the token's value along its key.

For input rows h [n, d] of one request in order, H value heads of dv entries, G query/key heads of dk (value
head i uses query/key head floor(i / (H / G))):

    q, k = h Wq^T, h Wk^T ([G, dk]),  v = h Wv^T ([H, dv]);  every channel of the three passes a causal convolution
        of `conv` taps over the request's tokens (no bias, the last tap weighs the current token, zeros
        before the start) and silu
    q <- q / sqrt(sum q^2 + unit_eps) * q_scale,  k <- k / sqrt(sum k^2 + unit_eps)          per head
    beta = sigmoid(h Wb^T),  g = exp(-exp(A_log) softplus(h Wa^T + dt_bias))                 one each per value head
    per head, a memory M_t [dk, dv], M before the first token zero:
        w_t = beta_t (v_t - g_t M_(t-1)^T k_t),   M_t = g_t M_(t-1) + k_t w_t^T,   o_t = M_t^T q_t
    out = ((o / rms(o) per head, eps inside the root, times norm [dv]) * gate(h Wg^T)) Wo^T

State per request (float32): M of every head in the kernels' own order and the convolutions' last conv - 1
inputs (csrc/delta.cu).  Parameters: hidden_size, num_heads, num_kv_heads, head_dim, v_head_dim, conv, q_scale, unit_eps,
eps, gate ("silu", "sigmoid" or None).  Tensors under <prefix>: q, k [G*dk, d]; v, g [H*dv, d]; b, a [H, d]; q.conv, k.conv,
v.conv [channels, conv]; A_log, dt_bias [H]; norm [dv]; o [d, H*dv].  q, k, v, the gate, b and a are one stacked product (rows
of zeros up to a multiple of 8) whose result stays float32; everything up to the gated output is float32 in
every mode.
"""
from __future__ import annotations

import torch

from ..csrc import ops
from .base import Mixer, PartError, StateNeed, register_part


@register_part("mixer", "gated_delta")
class GatedDelta(Mixer):
    CAPTURE_SAFE = True
    INPUT_MATRIX = "w_in"         # the stacked product on h; a mixer made of mixers may run it with its neighbour's

    def __init__(self, params, prefix, runtime):
        super().__init__(params, prefix, runtime)
        p = params
        self.hidden_size = int(p["hidden_size"])
        self.H, self.G = int(p["num_heads"]), int(p["num_kv_heads"])
        self.dk, self.dv, self.taps = int(p["head_dim"]), int(p["v_head_dim"]), int(p["conv"])
        self.q_scale, self.unit_eps = float(p["q_scale"]), float(p.get("unit_eps", 1e-6))
        self.eps = float(p.get("eps", 1e-6))
        self.gate = p.get("gate", "silu")
        if self.gate not in ops.GATES:
            raise PartError(f"gated_delta: gate {self.gate!r} is not known")
        if self.H % self.G:
            raise PartError(f"gated_delta: {self.H} heads are not a multiple of {self.G} query/key heads")
        if self.dk > 512 or not 1 <= self.taps <= 64:
            raise PartError("gated_delta: key heads up to 512 entries, 1 to 64 taps")
        self.has_gate = bool(ops.GATES[self.gate])
        names, offs, at = ["q", "k", "v"] + (["g"] if self.has_gate else []) + ["b", "a"], {"g": 0}, 0
        for s in names:
            offs[s] = at
            at += {"q": self.G * self.dk, "k": self.G * self.dk, "b": self.H, "a": self.H}.get(s, self.H * self.dv)
        self.names, self.offs = names, tuple(offs[s] for s in "qkvgba")
        self.w_in = self.w_o = self.conv_w = self.A = self.dt_bias = self.norm_w = None

    def cache_need(self):
        return StateNeed((ops.delta_state_floats(self.H, self.dk, self.dv, self.taps),), torch.float32)

    def expected_tensors(self):
        d, p, qk, hv = self.hidden_size, self.prefix, self.G * self.dk, self.H * self.dv
        t = {p + "q": ((qk, d), "matrix"), p + "k": ((qk, d), "matrix"), p + "v": ((hv, d), "matrix"),
             p + "b": ((self.H, d), "matrix"), p + "a": ((self.H, d), "matrix"), p + "A_log": ((self.H,), "bias"),
             p + "dt_bias": ((self.H,), "bias"), p + "norm": ((self.dv,), "norm"), p + "o": ((d, hv), "matrix")}
        t.update({f"{p}{s}.conv": ((c, self.taps), "conv") for s, c in (("q", qk), ("k", qk), ("v", hv))})
        if self.has_gate:
            t[p + "g"] = ((hv, d), "matrix")
        return t

    def load(self, tensors):
        p, dt, f32 = self.prefix, self.runtime.dtype, torch.float32
        stack = [tensors[p + s].to(dt) for s in self.names]
        rows = sum(t.shape[0] for t in stack)
        if rows % 8:                 # the projection's float32 rows stay aligned for every product kernel
            stack.append(torch.zeros((8 - rows % 8, self.hidden_size), dtype=dt, device=stack[0].device))
        self.w_in = self._to_device(torch.cat(stack, 0))
        self.w_o = self._to_device(tensors[p + "o"])
        self.conv_w = self._to_device(torch.cat([tensors[f"{p}{s}.conv"].to(f32) for s in "qkv"], 0), f32)
        self.A = self._to_device(torch.exp(tensors[p + "A_log"].to(f32)), f32)
        self.dt_bias = self._to_device(tensors[p + "dt_bias"], f32)
        self.norm_w = self._to_device(tensors[p + "norm"], f32)

    def forward(self, h, ctx, cache, position=None, residual=None, rows=None):
        """`rows`: h . w_in^T (float32), where somebody else has run that product."""
        if rows is None:
            rows = ops.linear(h, self.w_in, out_dtype=torch.float32)
        out = torch.empty((h.shape[0], self.H * self.dv), dtype=self.runtime.dtype, device=h.device)
        ops.gated_delta(rows, self.offs, self.conv_w, self.A, self.dt_bias, self.norm_w, self.q_scale, self.unit_eps,
                        self.eps, cache.state, ctx.cu_q, cache.slots, out, ctx.n_requests, ctx.max_q_len, self.H, self.G,
                        self.dk, self.dv, gate=self.gate)
        return ops.linear(out, self.w_o, out_dtype=torch.float32)
