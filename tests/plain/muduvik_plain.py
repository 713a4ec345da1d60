"""Plain, slow Muduvik forward pass: the oracle of the Muduvik tests.

Whole sequences, no cache, no batching, one function for each mechanism, float64
throughout.  It shares no code with ``lite_lang_b200``: it reads ``config.json``
and ``model.safetensors`` itself and works on torch tensors on the CPU.

The design in this file's notation (x: residual row of a token, p: its position
from 0; R(u) = u / sqrt(mean u^2 + eps); N_a(u) = R(u) a for a weight a).

*Residual.*  x = N_embed(E[token]).  The layers run in order; those of a range
[start, stop) run several times in a row, and pass t of the range begins with
x += s_t, s the rows of ``loop.step``.  Layer i:
    x += l1 N_1b(mixer(N_1(x)));   x += l2 N_2b(ff(N_2(x)))       (if it has a feed-forward)
    e = slice i of the token's row of ``side.embed``;  x += N_side(P (gelu(G x) e))
Logits = H N_final(x).

*Mixer "attention"* (two softmax maps over the same values).  Head a of H reads key and
value head b = a // (H / K).  With q = W_q u + b_q cut into [head][map 1 | map 2] and k
alike, every (head, map) part z becomes rot(R(z) w) (weights ``q.norm``, ``k.norm`` for
all); A_m = softmax over the visible j (i - W < j <= i) of scale q_m,i . k_m,j, times v;
    z = A_1 - lambda A_2,  lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + d;
    head a's output: (1 - d) R(z) sigmoid(g_a . u);   then W_o on the heads side by side.
rot: neighbours (2i, 2i + 1) of the first n channels turned by p f_i, where
f_i = base^(-2i/n) is kept for wavelengths l = 2 pi / f below orig / high, divided by F
above orig / low, and in between (1 - s) f / F + s f with s = (orig / l - low) / (high - low).

*Mixer "latent_attention"*.  q = W_uq N_dq(W_dq u), c = N_dkv(W_dkv u), k = W_uk c,
v = W_uv c by heads; causal softmax of scale q . k; W_o.

*Mixer "retention"*.  q = rot(W_q u), k = rot(W_k u) / sqrt(dim), v = W_v u; rot turns
(i, i + n/2) of the first n channels by p base^(-2i/n).  By heads S_t = d S_(t-1) + k_t v_t^T,
o_t = S_t^T q_t; W_o (R(o) by heads, side by side, times silu(W_g u)).

*Feed-forward.*  W_down (gelu(W_gate u) (W_up u)), gelu in its tanh form.
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


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def unit_rms(u: torch.Tensor, eps: float) -> torch.Tensor:
    return u / torch.sqrt((u * u).mean(-1, keepdim=True) + eps)


def norm(u: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return unit_rms(u, eps) * w


def output_norm(y: torch.Tensor, w: torch.Tensor, layer_scale: torch.Tensor, eps: float) -> torch.Tensor:
    return norm(y, w, eps) * layer_scale


def visible(T: int, W: Optional[int]) -> torch.Tensor:
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) if W is None else (j <= i) & (i - j < W)


def frequencies(rot: Mapping) -> torch.Tensor:
    n, base = int(rot["dims"]), float(rot["base"])
    f = base ** (-2.0 * torch.arange(n // 2, dtype=F) / n)
    sc = rot.get("scaling")
    if not sc:
        return f
    factor, low, high, orig = (float(sc[k]) for k in ("factor", "low", "high", "original"))
    out = []
    for x in f.tolist():
        wave = 2.0 * math.pi / x
        if wave < orig / high:
            out.append(x)
        elif wave > orig / low:
            out.append(x / factor)
        else:
            s = (orig / wave - low) / (high - low)
            out.append((1.0 - s) * x / factor + s * x)
    return torch.tensor(out, dtype=F)


def rotate_neighbours(u: torch.Tensor, pos: torch.Tensor, rot: Mapping) -> torch.Tensor:
    """u [T, heads, width]: channels (2i, 2i + 1) of the first n = rot.dims turned, the rest kept."""
    n = int(rot["dims"])
    ang = (pos.to(F)[:, None] * frequencies(rot)[None, :])[:, None, :]
    out = u.clone()
    a, b = u[..., 0:n:2], u[..., 1:n:2]
    out[..., 0:n:2] = a * torch.cos(ang) - b * torch.sin(ang)
    out[..., 1:n:2] = b * torch.cos(ang) + a * torch.sin(ang)
    return out


def rotate_halves(u: torch.Tensor, pos: torch.Tensor, rot: Mapping) -> torch.Tensor:
    """u [T, heads, width]: channels (i, i + n/2) of the first n = rot.dims turned, the rest kept."""
    n = int(rot["dims"])
    ang = (pos.to(F)[:, None] * frequencies(rot)[None, :])[:, None, :]
    a, b = u[..., :n // 2], u[..., n // 2:n]
    return torch.cat([a * torch.cos(ang) - b * torch.sin(ang), b * torch.cos(ang) + a * torch.sin(ang), u[..., n:]], dim=-1)


def softmax_attention(q, k, v, scale, vis):
    """q [T, H, d], k [T, K, d], v [T, K, dv], vis [T, T] -> [T, H, dv]."""
    H, K = q.shape[1], k.shape[1]
    out = []
    for a in range(H):
        b = a // (H // K)
        s = ((q[:, a] @ k[:, b].T) * scale).masked_fill(~vis, -math.inf)
        out.append(torch.softmax(s, dim=-1) @ v[:, b])
    return torch.stack(out, dim=1)


# --------------------------------------------------------------------------
# mixers
# --------------------------------------------------------------------------

def map_weight(m: Mapping, w: Mapping, p: str) -> float:
    """lambda: what the second map's output is multiplied by before it is taken off the first's."""
    return float(torch.exp((w[p + "lq1"] * w[p + "lk1"]).sum()) - torch.exp((w[p + "lq2"] * w[p + "lk2"]).sum())) + float(m["diff"])


def combine_maps(a1: torch.Tensor, a2: torch.Tensor, lam: float, diff: float, eps: float) -> torch.Tensor:
    return unit_rms(a1 - lam * a2, eps) * (1.0 - diff)


def normed_parts(z: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return norm(z, w, eps)


def mixer_attention(u, pos, m, w, p, eps):
    T = u.shape[0]
    H, K, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = (u @ w[p + "q"].T + w[p + "q.b"]).view(T, 2 * H, d)
    k = (u @ w[p + "k"].T + w[p + "k.b"]).view(T, 2 * K, d)
    v = (u @ w[p + "v"].T + w[p + "v.b"]).view(T, K, dv)
    q = rotate_neighbours(normed_parts(q, w[p + "q.norm"], eps), pos, m["rot"]).view(T, H, 2, d)
    k = rotate_neighbours(normed_parts(k, w[p + "k.norm"], eps), pos, m["rot"]).view(T, K, 2, d)
    mask = m.get("mask") or {}
    vis = visible(T, None if mask.get("size") is None else int(mask["size"]))
    a1, a2 = (softmax_attention(q[:, :, i], k[:, :, i], v, float(m["scale"]), vis) for i in (0, 1))
    z = combine_maps(a1, a2, map_weight(m, w, p), float(m["diff"]), eps)
    z = z * sigmoid(u @ w[p + "g"].T)[:, :, None]
    return z.reshape(T, H * dv) @ w[p + "o"].T


def mixer_latent_attention(u, pos, m, w, p, eps):
    T = u.shape[0]
    H, d, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = (norm(u @ w[p + "dq"].T, w[p + "dq.norm"], eps) @ w[p + "uq"].T).view(T, H, d)
    c = norm(u @ w[p + "dkv"].T, w[p + "dkv.norm"], eps)
    k, v = (c @ w[p + "uk"].T).view(T, H, d), (c @ w[p + "uv"].T).view(T, H, dv)
    o = softmax_attention(q, k, v, float(m["scale"]), visible(T, None))
    return o.reshape(T, H * dv) @ w[p + "o"].T


def decayed_sums(q, k, v, decay):
    """q, k [T, H, d], v [T, H, dv], decay [H] -> o [T, H, dv] of S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t."""
    T, H, d = q.shape
    S = torch.zeros((H, d, v.shape[2]), dtype=F)
    out = []
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out)


def mixer_retention(u, pos, m, w, p, eps):
    T = u.shape[0]
    H, d, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = rotate_halves((u @ w[p + "q"].T).view(T, H, d), pos, m["rot"])
    k = rotate_halves((u @ w[p + "k"].T).view(T, H, d), pos, m["rot"]) * d ** -0.5
    v = (u @ w[p + "v"].T).view(T, H, dv)
    o = unit_rms(decayed_sums(q, k, v, torch.tensor([float(x) for x in m["decay"]], dtype=F)), eps)
    return (o.reshape(T, H * dv) * silu(u @ w[p + "g"].T)) @ w[p + "o"].T


MIXERS = {"attention": mixer_attention, "latent_attention": mixer_latent_attention, "retention": mixer_retention}


# --------------------------------------------------------------------------
# feed-forward, token input, the model
# --------------------------------------------------------------------------

def feed_forward(u, w, p):
    return (gelu_tanh(u @ w[p + "gate"].T) * (u @ w[p + "up"].T)) @ w[p + "down"].T


def side_slice(ids, i, dim, w):
    return w["side.embed"][ids][:, i * dim:(i + 1) * dim]


def token_side(x, ids, i, dim, w, eps):
    p = f"l{i}.side."
    g = gelu_tanh(x @ w[p + "gate"].T) * side_slice(ids, i, dim, w)
    return norm(g @ w[p + "proj"].T, w[p + "norm"], eps)


def run_order(cfg: Mapping) -> List[tuple]:
    """(layer, row of loop.step that is added before it or None) in the order in which the layers run."""
    n = len(cfg["layers"])
    loop = cfg.get("loop") or {"start": 0, "stop": 0, "times": 0}
    a, b, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    order = [(i, None) for i in range(a)]
    for t in range(times):
        order += [(i, t if i == a else None) for i in range(a, b)]
    return order + [(i, None) for i in range(b, n)]


def forward(cfg: Mapping, w: Mapping[str, torch.Tensor], tokens: List[int], layers_out: Optional[list] = None):
    """Logits [T, vocab] of one whole sequence.  ``layers_out``: receives the residual after every layer run."""
    eps = float(cfg["norm"]["eps"])
    dim = int(cfg["token_side"]["dim"])
    ids = torch.tensor(tokens, dtype=torch.long)
    pos = torch.arange(len(tokens))
    x = norm(w["embed"][ids], w["embed.norm"], eps)
    for i, row in run_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if row is not None:
            x = x + w["loop.step"][row]
        y = MIXERS[layer["type"]](norm(x, w[p + "norm1"], eps), pos, layer["mixer"], w, p + "mix.", eps)
        x = x + output_norm(y, w[p + "norm1b"], w[p + "ls1"], eps)
        if layer.get("mlp") is not None:
            y = feed_forward(norm(x, w[p + "norm2"], eps), w, p + "mlp.")
            x = x + output_norm(y, w[p + "norm2b"], w[p + "ls2"], eps)
        x = x + token_side(x, ids, i, dim, w, eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return norm(x, w["final.norm"], eps) @ w["head"].T
