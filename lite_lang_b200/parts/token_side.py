"""A per-token table that enters every layer, gated by the layer's residual.

    out = W_proj (gelu_tanh(W_gate x) * E_i[token]),      x the residual itself (rounded to the engine's dtype)

E holds ``dim`` numbers a layer and token side by side, [vocab, layers * dim]; a layer's part is its columns
[index * dim, (index + 1) * dim), kept as a table of its own on the device.  The output's norm and the sum with the residual
are the block's.  Tensors: ``gate`` [dim, hidden], ``proj`` [hidden, dim], ``table``, by full names (``tensor_names``): the
table is one tensor of the checkpoint that all layers read.
"""

from __future__ import annotations

from typing import Dict, Optional

import torch

from .. import ops
from .base import FeedForward, TensorDecl, register_part


class TokenSide(FeedForward):
    def __init__(self, spec):
        super().__init__(spec)
        p = spec.params
        self.hidden_size = int(p["hidden_size"])
        self.vocab_size = int(p["vocab_size"])
        self.dim = int(p["dim"])
        self.index = int(p["index"])
        self.layers = int(p["layers"])
        self.names = dict(p.get("tensor_names") or {"gate": "gate", "proj": "proj", "table": "table"})
        if self.dim <= 0 or not (0 <= self.index < self.layers):
            raise ValueError("token_side: dim must be positive and index one of the layers")
        self.w_gate = self.w_proj = None
        self.table: Optional[torch.Tensor] = None
        self.dtype: Optional[torch.dtype] = None

    def tensors(self) -> Dict[str, TensorDecl]:
        return {self.names["gate"]: TensorDecl((self.dim, self.hidden_size)),
                self.names["proj"]: TensorDecl((self.hidden_size, self.dim)),
                self.names["table"]: TensorDecl((self.vocab_size, self.layers * self.dim))}

    def load(self, fetch, dtype, device) -> None:
        # rows of the gate's product, and of the table, are padded to whole 16-byte pieces; the padding's activations are
        # zeros and meet zero columns of the projection
        wide = (self.dim + 7) // 8 * 8
        gate, proj = fetch(self.names["gate"]).to(dtype), fetch(self.names["proj"]).to(dtype)
        part = fetch(self.names["table"])[:, self.index * self.dim:(self.index + 1) * self.dim].to(dtype)
        if wide != self.dim:
            gate = torch.nn.functional.pad(gate, (0, 0, 0, wide - self.dim))
            proj = torch.nn.functional.pad(proj, (0, wide - self.dim))
            part = torch.nn.functional.pad(part, (0, wide - self.dim))
        self.w_gate, self.w_proj = gate.to(device).contiguous(), proj.to(device).contiguous()
        self.table = part.to(device).contiguous()
        self.dtype = dtype

    def kernel_libraries(self):
        bf16 = self.w_gate is not None and self.w_gate.dtype == torch.bfloat16
        return ["core", "sandwich"] + (["gemm_smallm", "gemm_stream", "gemm_tc"] if bf16 else [])

    def weight_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in (self.w_gate, self.w_proj))

    def forward(self, x, step):
        g = ops.linear(x, self.w_gate)
        ops.token_side_act(g, self.table, step.token_ids, step.status)
        return ops.linear(g, self.w_proj, partial_ok=True)


register_part("feed_forward", "token_side", TokenSide)
