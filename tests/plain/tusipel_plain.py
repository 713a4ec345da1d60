"""Plain, slow Tusipel forward pass: the oracle of the Tusipel tests.

Whole sequences, no cache, no batching, one function for each mechanism, float64
throughout.  It shares no code with ``lite_lang_b200``: it reads ``config.json``
and ``model.safetensors`` itself and works on torch tensors on the CPU.

The design in this file's notation (x: residual row of a token, p: its position
from 0, E: embedding table).

*Residual.*  x = a E[token] =: x0.  The layers run in order; those of a range
[start, stop) run several times in a row, and every pass but the first begins with
x += x0.  A layer is x += mixer(C1(N1(x))); x += ff(C2(N2(x))) (the second only if it
has a feed-forward).  N(x) = R(x) (1 + w), R(x) = x / sqrt(mean x^2 + eps).
C(h)_t = h_t + K(h)_t, where K is a causal convolution a channel:
K(u)_t = sum_{j=0}^{n-1} w_j u_{t-n+1+j}, u before the first token zero.  Logits = H N_f(x).

*Mixer "latent_attention".*  c_q = R(W_dq u) w_dq, q = W_uq c_q, per head [d plain | r
rotated]; W_dkv u = [c' | k_r], c = R(c') w_dkv, k_r one rotated part for all heads; head
a's plain key (W_uk c)_a, value (W_uv c)_a; s_ij = scale (q_plain . k_plain + rot(q_r) .
rot(k_r)); j visible if 0 <= i - j < W; softmax; the heads side by side times
sigmoid(W_g u), then W_o.  Rotation: channels (i, i + n/2) of the first n turned by p f_i,
cos and sin times c_m.  With b_i = base^(-2i/n), d(t) = n ln(orig / (2 pi t)) / (2 ln base),
lo = max(floor d(fast), 0), hi = min(ceil d(slow), n - 1), g_i = clamp((i - lo) / max(hi -
lo, 0.001), 0, 1): f_i = (b_i / F) g_i + b_i (1 - g_i), c_m = 0.1 ln F + 1.

*Mixer "attention".*  q = K(Wq u), k = K(Wk u), v = K(Wv u), each with its own taps; query
head a reads key/value head a // (H/G); s_ij = scale q_i . k_j - 2^(-8 (a + 1) / H) (i - j);
j visible if j <= i and i // C = j // C; softmax; Wo.

*Feed-forward.*  dense: g = min(W_g u, L), c = clamp(W_u u, -L, L), W_d (g sigmoid(1.702 g)
(c + 1)).  moe: s = softmax(W_r u) over all n outputs, choice score s + b; the n outputs
form equal groups of neighbours, only those of the groups with the largest maxima of the
choice score may be chosen; of them the largest choice scores are.  Output: sum over chosen e of
c s_e f_e(u), with f_e(u) = W_d,e (silu(W_g,e u) (W_u,e u)), or u itself for the last ones.
"""

from __future__ import annotations

import json
import math
import os
from typing import Dict, List, Mapping, Optional

import torch
from safetensors import safe_open

F = torch.float64


def read_model_folder(model_dir: str):
    with open(os.path.join(model_dir, "config.json"), "r", encoding="utf-8") as fh:
        cfg = json.load(fh)
    tensors: Dict[str, torch.Tensor] = {}
    with safe_open(os.path.join(model_dir, "model.safetensors"), framework="pt") as fh:
        for name in fh.keys():
            t = fh.get_tensor(name)
            tensors[name] = t.to(F) if t.is_floating_point() else t
    return cfg, tensors


# --------------------------------------------------------------------------
# small pieces
# --------------------------------------------------------------------------

def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def unit_rms(u: torch.Tensor, eps: float) -> torch.Tensor:
    return u / torch.sqrt((u * u).mean(-1, keepdim=True) + eps)


def centred_norm(u: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return unit_rms(u, eps) * (1.0 + w)


def causal_convolution(u: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """u [T, C], w [C, taps], the last tap for the token itself; zeros before the first token."""
    T, taps = u.shape[0], w.shape[1]
    padded = torch.cat([torch.zeros((taps - 1, u.shape[1]), dtype=u.dtype), u])
    out = torch.zeros_like(u)
    for j in range(taps):
        out = out + padded[j:j + T] * w[:, j]
    return out


def with_convolution(h: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    return h + causal_convolution(h, w)


def visible_window(T: int, W: Optional[int]) -> torch.Tensor:
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) if W is None else (j <= i) & (i - j < W)


def visible_chunk(T: int, C: Optional[int]) -> torch.Tensor:
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) if C is None else (j <= i) & (i // C == j // C)


def slopes(H: int) -> torch.Tensor:
    return torch.tensor([2.0 ** (-8.0 * (a + 1) / H) for a in range(H)], dtype=F)


def distance_penalty(T: int, H: int) -> torch.Tensor:
    """[H, T, T]: what is taken off the score of query i and key j."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return slopes(H)[:, None, None] * (i - j).to(F)


def softmax_attention(q, k, v, scale, vis, penalty=None):
    """q [T, H, d], k [T, G, d], v [T, G, dv], vis [T, T], penalty [H, T, T] -> [T, H, dv]."""
    H, G = q.shape[1], k.shape[1]
    out = []
    for a in range(H):
        b = a // (H // G)
        s = (q[:, a] @ k[:, b].T) * scale
        if penalty is not None:
            s = s - penalty[a]
        out.append(torch.softmax(s.masked_fill(~vis, -math.inf), dim=-1) @ v[:, b])
    return torch.stack(out, dim=1)


def scaled_frequencies(rot: Mapping):
    n, base = int(rot["dims"]), float(rot["base"])
    i = torch.arange(n // 2, dtype=F)
    b = base ** (-2.0 * i / n)
    sc = rot.get("scaling")
    if not sc:
        return b, 1.0
    factor, orig = float(sc["factor"]), float(sc["original"])

    def d(t):
        return n * math.log(orig / (2.0 * math.pi * t)) / (2.0 * math.log(base))

    lo = max(math.floor(d(float(sc["fast"]))), 0)
    hi = min(math.ceil(d(float(sc["slow"]))), n - 1)
    g = torch.clamp((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return b / factor * g + b * (1.0 - g), 0.1 * math.log(factor) + 1.0


def rotate(u: torch.Tensor, pos: torch.Tensor, rot: Mapping) -> torch.Tensor:
    """u [T, heads, width]; pairs (i, i + n/2) of the first n = rot.dims channels turned, the rest kept."""
    n = int(rot["dims"])
    if n == 0:
        return u
    f, c = scaled_frequencies(rot)
    ang = pos.to(F)[:, None] * f[None, :]
    cs, sn = (torch.cos(ang) * c)[:, None, :], (torch.sin(ang) * c)[:, None, :]
    a, b = u[..., :n // 2], u[..., n // 2:n]
    return torch.cat([a * cs - b * sn, b * cs + a * sn, u[..., n:]], dim=-1)


# --------------------------------------------------------------------------
# mixers
# --------------------------------------------------------------------------

def _mask_size(m: Mapping) -> Optional[int]:
    mask = m.get("mask") or {}
    return None if mask.get("size") is None else int(mask["size"])


def mixer_latent_attention(u, pos, m, w, p, eps):
    T = u.shape[0]
    H, d, r, dv, R = int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"])
    cq = unit_rms(u @ w[p + "dq"].T, eps) * w[p + "dq.norm"]
    q = (cq @ w[p + "uq"].T).view(T, H, d + r)
    ckv = u @ w[p + "dkv"].T
    c = unit_rms(ckv[:, :R], eps) * w[p + "dkv.norm"]
    k_rot = rotate(ckv[:, None, R:], pos, m["rot"])                       # [T, 1, r]
    q_rot = rotate(q[:, :, d:], pos, m["rot"])
    k_plain = (c @ w[p + "uk"].T).view(T, H, d)
    v = (c @ w[p + "uv"].T).view(T, H, dv)
    qq = torch.cat([q[:, :, :d], q_rot], dim=-1)
    kk = torch.cat([k_plain, k_rot.expand(T, H, r)], dim=-1)
    o = softmax_attention(qq, kk, v, float(m["scale"]), visible_window(T, _mask_size(m)))
    return (o.reshape(T, H * dv) * sigmoid(u @ w[p + "g"].T)) @ w[p + "o"].T


def mixer_attention(u, pos, m, w, p, eps):
    T = u.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q, k, v = (causal_convolution(u @ w[p + n].T, w[p + n + ".conv"]) for n in ("q", "k", "v"))
    o = softmax_attention(q.view(T, H, d), k.view(T, G, d), v.view(T, G, dv), float(m["scale"]),
                          visible_chunk(T, _mask_size(m)), distance_penalty(T, H))
    return o.reshape(T, H * dv) @ w[p + "o"].T


MIXERS = {"attention": mixer_attention, "latent_attention": mixer_latent_attention}


# --------------------------------------------------------------------------
# feed-forward
# --------------------------------------------------------------------------

def dense_ff(u, mlp, w, p):
    L = float(mlp["limit"])
    g = torch.clamp(u @ w[p + "gate"].T, max=L)
    c = torch.clamp(u @ w[p + "up"].T, min=-L, max=L)
    return (g * sigmoid(1.702 * g) * (c + 1.0)) @ w[p + "down"].T


def choose(choice: torch.Tensor, count: int, keep: int, top: int):
    """One token's choice scores [n] -> the chosen outputs (ties: the lower index) and the margin: how far the choice
    is from another one (of the groups and of the outputs)."""
    n = choice.numel()
    size = n // count
    best = [float(choice[g * size:(g + 1) * size].max()) for g in range(count)]
    order = sorted(range(count), key=lambda g: (-best[g], g))
    margin = best[order[keep - 1]] - best[order[keep]] if keep < count else math.inf
    allowed = [e for g in sorted(order[:keep]) for e in range(g * size, (g + 1) * size)]
    ranked = sorted(allowed, key=lambda e: (-float(choice[e]), e))
    if top < len(ranked):
        margin = min(margin, float(choice[ranked[top - 1]] - choice[ranked[top]]))
    return ranked[:top], margin


def routed_ff(u, mlp, w, p, margins=None):
    r = mlp["router"]
    E, ident, top = int(r["experts"]), int(r.get("identity") or 0), int(r["top"])
    groups = r.get("groups") or {"count": 1, "keep": 1}
    s = torch.softmax(u @ w[p + "router"].T, dim=-1)                      # [T, E + ident]
    assert s.shape[1] == E + ident
    out = torch.zeros_like(u)
    low = []
    for t in range(u.shape[0]):
        chosen, margin = choose(s[t] + w[p + "correction"], int(groups["count"]), int(groups["keep"]), top)
        low.append(margin)
        for e in chosen:
            y = u[t] if e >= E else (silu(u[t] @ w[f"{p}e{e}.gate"].T) * (u[t] @ w[f"{p}e{e}.up"].T)) @ w[f"{p}e{e}.down"].T
            out[t] += float(r["scale"]) * s[t, e] * y
    if margins is not None:
        margins.append(torch.tensor(low, dtype=F))
    return out


def feed_forward(u, mlp, w, p, margins=None):
    return dense_ff(u, mlp, w, p) if mlp["kind"] == "dense" else routed_ff(u, mlp, w, p, margins)


# --------------------------------------------------------------------------
# the model
# --------------------------------------------------------------------------

def run_order(cfg: Mapping) -> List[tuple]:
    """(layer, whether x0 is added before it) in the order in which the layers run."""
    n = len(cfg["layers"])
    loop = cfg.get("loop") or {"start": 0, "stop": 0, "times": 1}
    a, b, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    order = [(i, False) for i in range(a)]
    for k in range(times):
        order += [(i, k > 0 and i == a) for i in range(a, b)]
    return order + [(i, False) for i in range(b, n)]


def forward(cfg: Mapping, w: Mapping[str, torch.Tensor], tokens: List[int], layers_out: Optional[list] = None,
            margins: Optional[list] = None):
    """Logits [T, vocab] of one whole sequence.  ``layers_out``: receives the residual after every layer run;
    ``margins``: every routed layer run's margins (see ``choose``)."""
    eps = float(cfg["norm"]["eps"])
    ids = torch.tensor(tokens, dtype=torch.long)
    pos = torch.arange(len(tokens))
    x0 = w["embed"][ids] * float(cfg["embedding"]["scale"])
    x = x0
    for i, add in run_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if add:
            x = x + x0
        h = with_convolution(centred_norm(x, w[p + "norm1"], eps), w[p + "canon1"])
        x = x + MIXERS[layer["type"]](h, pos, layer["mixer"], w, p + "mix.", eps)
        if layer.get("mlp") is not None:
            h = with_convolution(centred_norm(x, w[p + "norm2"], eps), w[p + "canon2"])
            x = x + feed_forward(h, layer["mlp"], w, p + "mlp.", margins)
        if layers_out is not None:
            layers_out.append(x.clone())
    return centred_norm(x, w["final.norm"], eps) @ w["head"].T
