"""Mamba (selective state-space) mixer.

For normed input rows h [n, d] of one request in order, `inner` channels, N state entries per
channel, a convolution of `conv` taps:

    [x | z] = h Win^T                                   (inner each)
    x  <- silu(conv_b + sum_j conv[:, j] * x(t - (conv-1) + j))    causal per channel, zeros before the start,
                                                                   the last tap weighs the current token
    [dt | B | C] = x Wx^T                               (dt_rank, N, N)
    dt <- softplus(dt Wdt^T + dt_b)                     one step size per channel
    A  = -exp(A_log)                                    [inner, N]
    S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n;   y_c = sum_n S[c, n] C_n + D_c x_c
    out = (y * silu(z)) Wo^T

State per request (float32): S and the last conv-1 inputs of the convolution.  Parameters:
hidden_size, inner, state, dt_rank, conv.  Tensors under <prefix>: in [2*inner, d], conv [inner,
conv], conv.b, x [dt_rank + 2N, inner], dt [inner, dt_rank], dt.b, A_log [inner, N], D, o [d,
inner].  Step sizes, decays, their exponentials and the state are float32 in every mode.
"""
from __future__ import annotations

import torch

from ..csrc import ops
from .base import Mixer, PartError, StateNeed, register_part


@register_part("mixer", "mamba1")
class Mamba1(Mixer):
    CAPTURE_SAFE = True

    def __init__(self, params, prefix, runtime):
        super().__init__(params, prefix, runtime)
        self.hidden_size = int(params["hidden_size"])
        self.inner, self.N = int(params["inner"]), int(params["state"])
        self.R, self.taps = int(params["dt_rank"]), int(params["conv"])
        if self.N > 256:
            raise PartError("mamba1: at most 256 state entries per channel")
        if self.taps < 1:
            raise PartError("mamba1: the convolution needs at least one tap")
        self.conv_off = self.inner * self.N

    def cache_need(self):
        return StateNeed((self.conv_off + self.inner * (self.taps - 1),), torch.float32)

    def expected_tensors(self):
        d, I, N, R, p = self.hidden_size, self.inner, self.N, self.R, self.prefix
        return {p + "in": ((2 * I, d), "matrix"), p + "conv": ((I, self.taps), "conv"), p + "conv.b": ((I,), "bias"),
                p + "x": ((R + 2 * N, I), "matrix"), p + "dt": ((I, R), "matrix"), p + "dt.b": ((I,), "bias"),
                p + "A_log": ((I, N), "bias"), p + "D": ((I,), "norm"), p + "o": ((d, I), "matrix")}

    def load(self, tensors):
        p, f32 = self.prefix, torch.float32
        self.w_in, self.w_x, self.w_dt, self.w_o = (self._to_device(tensors[p + s]) for s in ("in", "x", "dt", "o"))
        self.conv_w = self._to_device(tensors[p + "conv"], f32)
        self.conv_b = self._to_device(tensors[p + "conv.b"], f32)
        self.dt_b = self._to_device(tensors[p + "dt.b"], f32)
        self.A = self._to_device(-torch.exp(tensors[p + "A_log"].to(f32)), f32)
        self.Dp = self._to_device(tensors[p + "D"], f32)

    def forward(self, h, ctx, cache, position=None, residual=None):
        n, dt, dev, I, N, R = h.shape[0], self.runtime.dtype, h.device, self.inner, self.N, self.R
        xz = ops.linear(h, self.w_in, out_dtype=torch.float32)
        x = torch.empty((n, I), dtype=dt, device=dev)
        ops.conv_silu(xz, self.conv_w, self.conv_b, cache.state, self.conv_off, ctx.seq_ids, ctx.cu_q, cache.slots,
                      x, I)
        low = ops.linear(x, self.w_x, out_dtype=torch.float32)
        step_in = torch.empty((n, R), dtype=dt, device=dev)
        ops.rows_act(low[:, :R], step_in)
        dtr = ops.linear(step_in, self.w_dt, out_dtype=torch.float32)
        y = torch.empty((n, I), dtype=dt, device=dev)
        ops.selective_scan(x, xz, low, R, R + N, dtr, self.dt_b, self.A, self.Dp, cache.state, self.conv_off,
                           ctx.cu_q, cache.slots, y, ctx.n_requests, I, N, self.taps,
                           segments=ops.time_segments(ctx, dev))
        return ops.linear(y, self.w_o, out_dtype=torch.float32)


@register_part("mixer", "mamba2")
class Mamba2(Mixer):
    """State spaces with one decay per head (Mamba-2).  For normed input rows h [n, d] of one request in order, H heads of P
    entries (inner = H P), G groups of N state entries, a convolution of `conv` taps:

        [z | x | B | C | dt] = h Win^T                        (inner, inner, G N, G N, H)
        x, B, C <- silu(conv_b + causal convolution per channel)   (zeros before the start, the last tap weighs the current token)
        dt <- softplus(dt + dt_bias);  per head, with B and C of group floor(head / (H / G)):
        S <- exp(-exp(A_log) dt) S + dt B x^T;   y = S^T C + D x
        v = y * silu(z);  v divided by its root mean square in `norm_groups` equal runs of columns, times a weight;  out = v Wo^T

    State per request (float32): S and the last inputs of the convolution.  Parameters: hidden_size, num_heads, v_head_dim (P),
    state (N), groups, conv, norm_groups, eps.  Tensors under <prefix>: in [2 inner + 2 G N + H, d], conv [channels, taps],
    conv.b, dt_bias, A_log, D, norm [inner], o [d, inner].  Load-time transforms: the in-projection gets rows of zeros up to a
    multiple of 8 rows, the taps are kept [taps, channels].  Step sizes, decays, the state, the gate and the norm are float32 in
    every mode.  ``forward(..., rows=)``: h . in^T from a stacked product (INPUT_MATRIX); ``into=, factor=``: the rows that the output
    projection would read, times `factor`, go to the matrix `into` and the projection is left to the caller (OUTPUT_MATRIX)."""
    CAPTURE_SAFE = True
    INPUT_MATRIX = "w_in"
    OUTPUT_MATRIX = "w_o"

    def __init__(self, params, prefix, runtime):
        super().__init__(params, prefix, runtime)
        p = params
        self.hidden_size, self.H, self.P = int(p["hidden_size"]), int(p["num_heads"]), int(p["v_head_dim"])
        self.N, self.G, self.taps = int(p["state"]), int(p["groups"]), int(p["conv"])
        self.norm_groups, self.eps = int(p["norm_groups"]), float(p["eps"])
        self.inner = self.H * self.P
        if self.H % self.G or self.inner % self.norm_groups:
            raise PartError(f"mamba2: {self.H} heads do not form {self.G} groups, or {self.inner} columns {self.norm_groups} parts")
        if self.N > 256:
            raise PartError("mamba2: at most 256 state entries")
        self.w_in = self.w_o = None
        self._scaled = {}

    @property
    def output_columns(self):
        return self.inner

    def cache_need(self):
        return StateNeed((ops.ssd_state_floats(self.H, self.P, self.N, self.G, self.taps),), torch.float32)

    def expected_tensors(self):
        d, I, p, H = self.hidden_size, self.inner, self.prefix, self.H
        C = I + 2 * self.G * self.N
        return {p + "in": ((I + C + H, d), "matrix"), p + "conv": ((C, self.taps), "conv"), p + "conv.b": ((C,), "bias"),
                p + "dt_bias": ((H,), "unit"), p + "A_log": ((H,), "unit"), p + "D": ((H,), "norm"), p + "norm": ((I,), "norm"),
                p + "o": ((d, I), "matrix")}

    def load(self, tensors):
        p, f32, dt = self.prefix, torch.float32, self.runtime.dtype
        w = tensors[p + "in"].to(dt)
        if w.shape[0] % 8:
            w = torch.cat([w, w.new_zeros((8 - w.shape[0] % 8, self.hidden_size))], 0)
        self.w_in, self.w_o = self._to_device(w), self._to_device(tensors[p + "o"])
        self.conv_w = self._to_device(tensors[p + "conv"].to(f32).t(), f32)
        self.conv_b, self.dt_b, self.Dp, self.norm_w = (self._to_device(tensors[p + s], f32)
                                                        for s in ("conv.b", "dt_bias", "D", "norm"))
        self.A = self._to_device(torch.exp(tensors[p + "A_log"].to(f32)), f32)
        self._scaled = {}

    def scaled_norm(self, factor):
        """The norm's weight times a constant (made once)."""
        if factor == 1.0:
            return self.norm_w
        if factor not in self._scaled:
            self._scaled[factor] = self.norm_w * factor
        return self._scaled[factor]

    def forward(self, h, ctx, cache, position=None, residual=None, rows=None, into=None, factor=1.0):
        if rows is None:
            rows = ops.linear(h, self.w_in, out_dtype=torch.float32)
        y = into if into is not None else torch.empty((h.shape[0], self.inner), dtype=self.runtime.dtype, device=h.device)
        ops.ssd(rows, self.conv_w, self.conv_b, self.dt_b, self.A, self.Dp, self.scaled_norm(factor), self.eps, self.norm_groups,
                cache.state, ctx, cache.slots, y, self.H, self.G, self.P, self.N)
        if into is not None:
            return None
        return ops.linear(y, self.w_o, out_dtype=torch.float32)
