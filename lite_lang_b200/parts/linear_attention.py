"""Linear attention with a decay per head ("lightning attention"): a recurrent mixer with a matrix state.

q = silu(W_q x), k = silu(W_k x) (``heads`` x ``key_dim``) and v = silu(W_v x) (``heads`` x ``value_dim``);
per head, token by token,

    S_t = decay_h * S_(t-1) + k_t v_t^T,      o_t = S_t^T q_t        (nothing else multiplies the scores)

The heads' o side by side are RMS-normed as one vector with the weight ``norm``, multiplied by
sigmoid(W_g x) and projected by W_o.  A request's state is all zeros before its first token; it is float32 and
lives in the request's record of the cache manager's state pool, so a request goes on in a later step, alone or
beside others, from where it stopped.  Everything between the projections and the output projection is float32.
Tensors: ``q``, ``k``, ``v``, ``g``, ``o``, ``norm``; ``decay`` is a parameter (one number a head).
"""

from __future__ import annotations

from typing import Dict

import torch

from .. import ops
from ..config.spec import PartSpec
from .base import Mixer, StateNeed, TensorDecl, build_part, register_part


def _pad8(n: int) -> int:
    return (n + 7) // 8 * 8


def stacked_rows(named, width: int, dtype, device):
    """One matrix for all products that read the same input, every segment starting at a multiple of 8 rows, and the
    segments' first rows by name."""
    off, rows, at = {}, [], 0
    for name, w in named:
        w = w.to(dtype)
        off[name] = at
        rows.append(w)
        pad = _pad8(w.shape[0]) - w.shape[0]
        if pad:
            rows.append(torch.zeros((pad, width), dtype=dtype, device=w.device))
        at += _pad8(w.shape[0])
    return torch.cat(rows, dim=0).to(device).contiguous(), off


class DecayLinearAttention(Mixer):
    def __init__(self, spec: PartSpec):
        super().__init__(spec)
        p = spec.params
        self.hidden_size = int(p["hidden_size"])
        self.H = int(p["heads"])
        self.dk = int(p["key_dim"])
        self.dv = int(p["value_dim"])
        self.decay_values = [float(d) for d in p["decay"]]
        self.eps = float(p["eps"])
        if len(self.decay_values) != self.H:
            raise ValueError(f"decay_linear_attention: {len(self.decay_values)} decays for {self.H} heads")
        if not (0 < self.dk <= 256):
            raise ValueError("decay_linear_attention: key heads of 1 to 256 channels are built")
        self.Cq, self.Cv = self.H * self.dk, self.H * self.dv
        self.w_in = None

    def tensors(self) -> Dict[str, TensorDecl]:
        h = self.hidden_size
        return {"q": TensorDecl((self.Cq, h)), "k": TensorDecl((self.Cq, h)), "v": TensorDecl((self.Cv, h)),
                "g": TensorDecl((self.Cv, h)), "o": TensorDecl((h, self.Cv)), "norm": TensorDecl((self.Cv,), "norm")}

    def load(self, fetch, dtype, device) -> None:
        self.w_in, self.off = stacked_rows([(n, fetch(n)) for n in ("q", "k", "v", "g")], self.hidden_size, dtype, device)
        self.w_o = fetch("o").to(dtype).to(device).contiguous()
        self.norm_w = fetch("norm").to(torch.float32).to(device).contiguous()
        self.decay = torch.tensor(self.decay_values, dtype=torch.float32, device=device)

    def weight_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in (self.w_in, self.w_o, self.norm_w))

    def cache_need(self):
        return StateNeed((self.H * self.dv * self.dk,), "float32")

    def kernel_libraries(self):
        libs = ["core", "linear_attn"]
        if self.w_in is not None and self.w_in.dtype == torch.bfloat16:
            libs.extend(["gemm_smallm", "gemm_stream", "gemm_tc"])
        return libs

    def forward(self, x, step, cache):
        n, dev = x.shape[0], x.device
        proj = ops.linear(x, self.w_in)
        ops.silu_rows(proj[:, :self.off["g"]])        # q | k | v (and the zero columns that pad them)
        o = torch.empty((n, self.Cv), dtype=torch.float32, device=dev)
        ops.decay_scan(proj, self.off["q"], self.off["k"], self.off["v"], self.decay, cache.state, step, o,
                       self.H, self.dk, self.dv, cache.writable)
        y = torch.empty((n, self.Cv), dtype=x.dtype, device=dev)
        ops.linear_attn_out(y, o, self.norm_w, proj[:, self.off["g"]:self.off["g"] + self.Cv], self.eps)
        return ops.linear(y, self.w_o, partial_ok=self.partial_ok)


class Retention(Mixer):
    """Retention: linear attention with a fixed decay per head whose queries and keys are rotated by the token's position.

    q = rot(W_q x), k = rot(W_k x) * ``key_scale`` (``heads`` x ``key_dim``), v = W_v x (``heads`` x ``value_dim``), no
    activation; S_t = decay_h S_(t-1) + k_t v_t^T, o_t = S_t^T q_t per head; every head's o divided by its own root mean
    square (``eps``), the heads side by side times silu(W_g x), projected by W_o.  ``position``: a ``rope_computed`` part or
    None.  The record and its place are those of ``decay_linear_attention``, and so is the scan; the rotated q and k (and
    the v beside them) are float32 rows of their own, so nothing that enters the recurrence is rounded after the projection.
    Tensors: ``q``, ``k``, ``v``, ``g``, ``o``; ``decay`` is a parameter (one number a head)."""

    def __init__(self, spec: PartSpec):
        super().__init__(spec)
        p = spec.params
        self.hidden_size = int(p["hidden_size"])
        self.H = int(p["heads"])
        self.dk = int(p["key_dim"])
        self.dv = int(p["value_dim"])
        self.decay_values = [float(d) for d in p["decay"]]
        self.key_scale = float(p.get("key_scale", 1.0))
        self.eps = float(p["eps"])
        if len(self.decay_values) != self.H:
            raise ValueError(f"retention: {len(self.decay_values)} decays for {self.H} heads")
        if not (0 < self.dk <= 256):
            raise ValueError("retention: key heads of 1 to 256 channels are built")
        pos = p.get("position")
        self.position = build_part("position", pos) if pos is not None else None
        if self.position is not None and (not getattr(self.position, "computed", False) or self.position.amplitude != 1.0):
            raise ValueError("retention: the position part must make its angles in the kernel (rope_computed), without an "
                             "amplitude")
        self.Cq, self.Cv = self.H * self.dk, self.H * self.dv
        self.w_in = None

    def tensors(self) -> Dict[str, TensorDecl]:
        h = self.hidden_size
        return {"q": TensorDecl((self.Cq, h)), "k": TensorDecl((self.Cq, h)), "v": TensorDecl((self.Cv, h)),
                "g": TensorDecl((self.Cv, h)), "o": TensorDecl((h, self.Cv))}

    def load(self, fetch, dtype, device) -> None:
        self.w_in, self.off = stacked_rows([(n, fetch(n)) for n in ("q", "k", "v", "g")], self.hidden_size, dtype, device)
        self.w_o = fetch("o").to(dtype).to(device).contiguous()
        self.decay = torch.tensor(self.decay_values, dtype=torch.float32, device=device)
        # the float32 rows q | k | v
        self.row = (0, _pad8(self.Cq), 2 * _pad8(self.Cq))
        self.row_width = self.row[2] + _pad8(self.Cv)

    def weight_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in (self.w_in, self.w_o))

    def cache_need(self):
        return StateNeed((self.H * self.dv * self.dk,), "float32")

    def kernel_libraries(self):
        libs = ["core", "linear_attn"]
        if self.w_in is not None and self.w_in.dtype == torch.bfloat16:
            libs.extend(["gemm_smallm", "gemm_stream", "gemm_tc"])
        return libs

    def prepare(self, device, dtype) -> None:
        if self.position is not None:
            self.position.prepare(device)

    def forward(self, x, step, cache):
        n, dev = x.shape[0], x.device
        proj = ops.linear(x, self.w_in)
        rows = torch.empty((n, self.row_width), dtype=torch.float32, device=dev)
        pos = self.position
        ops.rotate_rows_f32(rows, self.row, proj, (self.off["q"], self.off["k"], self.off["v"]), step.positions,
                            None if pos is None else pos.freq, bool(pos is None or pos.interleaved), self.H, self.dk, self.Cv,
                            1.0, self.key_scale)
        o = torch.empty((n, self.Cv), dtype=torch.float32, device=dev)
        ops.decay_scan(rows, *self.row, self.decay, cache.state, step, o, self.H, self.dk, self.dv, cache.writable)
        y = torch.empty((n, self.Cv), dtype=x.dtype, device=dev)
        ops.head_norm_gate_out(y, o, proj[:, self.off["g"]:self.off["g"] + self.Cv], self.eps, self.H, self.dv, "silu")
        return ops.linear(y, self.w_o, partial_ok=self.partial_ok)


register_part("mixer", "decay_linear_attention", DecayLinearAttention)
register_part("mixer", "retention", Retention)
