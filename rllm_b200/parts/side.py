"""What a layer joins to the stream behind its sublayers: a per-token input from a second table.

    e = table[token, part * dim : (part + 1) * dim]
    x <- x + mult * norm(P (gelu_tanh(G x) * e))

with gelu_tanh the tanh form of gelu and an RMS norm with a plain weight.  The table holds `parts` runs of `dim`
entries per token, one per layer; a layer keeps its own run as a table [vocab, dim].

Parameters: hidden_size, vocab_size, dim, part, parts, tensor (the table's name), eps.  Tensors: <tensor> [vocab, parts * dim],
<prefix>gate [dim, d], <prefix>proj [d, dim], <prefix>norm [d].  Load-time transforms: the gate's rows and the projection's
columns are padded with zeros to a multiple of 8.  The gate's pre-activation, the activation, the norm and the
sum are float32 in every mode.
"""
from __future__ import annotations

import torch

from ..config.base import PartSpec
from ..csrc import ops
from .base import PartError, Side, build_part, register_part


@register_part("side", "token_table")
class TokenTable(Side):
    CAPTURE_SAFE = True

    def __init__(self, params, prefix, runtime):
        super().__init__(params, prefix, runtime)
        p = params
        self.hidden_size, self.vocab, self.dim = int(p["hidden_size"]), int(p["vocab_size"]), int(p["dim"])
        self.part, self.n_parts, self.table_name = int(p["part"]), int(p["parts"]), p["tensor"]
        if not 0 <= self.part < self.n_parts:
            raise PartError(f"token_table: part {self.part} is not one of {self.n_parts}")
        self.padded = -(-self.dim // 8) * 8
        self.norm = build_part("norm", PartSpec("rms_norm", {"size": self.hidden_size, "eps": p["eps"],
                                                             "tensor": prefix + "norm"}), runtime)
        self.table = self.w_gate = self.w_proj = None

    def expected_tensors(self):
        d, p = self.hidden_size, self.prefix
        return {self.table_name: ((self.vocab, self.n_parts * self.dim), "matrix"), p + "gate": ((self.dim, d), "matrix"),
                p + "proj": ((d, self.dim), "matrix"), **self.norm.expected_tensors()}

    def load(self, tensors):
        p, dim = self.prefix, self.dim
        self.table = self._to_device(tensors[self.table_name][:, self.part * dim:(self.part + 1) * dim])
        gate, proj = tensors[p + "gate"], tensors[p + "proj"]
        if self.padded > dim:
            gate = torch.cat([gate, gate.new_zeros((self.padded - dim, self.hidden_size))], 0)
            proj = torch.cat([proj, proj.new_zeros((self.hidden_size, self.padded - dim))], 1)
        self.w_gate, self.w_proj = self._to_device(gate), self._to_device(proj)
        self.norm.load(tensors)

    def forward(self, x, rows, ctx, mult, next_norm=None):
        z = ops.linear(rows, self.w_gate, out_dtype=torch.float32)
        g = torch.empty((x.shape[0], self.padded), dtype=self.runtime.dtype, device=x.device)
        ops.token_gate(z, self.table, ctx.tokens, g, self.dim)
        y = ops.linear(g, self.w_proj, out_dtype=torch.float32)
        if next_norm is not None and hasattr(next_norm, "tanh_form"):
            return self.norm.join_then(x, y, next_norm, mult)
        self.norm.join(x, y, mult=mult)
        return None
