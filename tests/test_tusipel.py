"""Tusipel through the engine against the plain implementation (tests/plain/tusipel_plain.py).

CPU: configuration, registry, run order, cache groups, what blocks hand on as pending, the plain implementation's own
properties.  GPU: each mechanism's kernels alone (with inputs made so that a fault at an edge shows), whole prompts,
token-by-token decoding through captured steps, portions down to two tokens, mixed batches with pages and slots used
again, the command-line replay tool and greedy generation through the scheduler.
"""
import json
import math
import os
import subprocess
import sys
import types

import numpy as np
import pytest
import torch

from helpers import TraceRun, rel_err
from plain import tusipel_plain as P
from tusipel_cases import CASES, write_folder

TOL = {torch.float32: 2e-4, torch.bfloat16: 6e-2}
gpu = pytest.mark.gpu


def dev():
    return torch.device("cuda:0")


def row_errors(got, ref):
    got, ref = np.asarray(got, dtype=np.float64), np.asarray(ref, dtype=np.float64)
    assert got.shape == ref.shape, (got.shape, ref.shape)
    return np.abs(got - ref).max(axis=-1) / np.abs(ref).max(axis=-1)


# a router's margin (of its groups and of its outputs) below which bfloat16 rounding may choose otherwise
UNDECIDED = 0.004


def decided_rows(margins) -> int:
    """How many leading tokens of a sequence have every router's choice safely decided."""
    if not margins:
        return 1 << 30
    low = (torch.stack(margins).min(0).values < UNDECIDED).nonzero()
    return int(low[0]) if low.numel() else 1 << 30


def close(got, ref, dtype, strict=None) -> bool:
    """float32: every row within the tolerance.  bfloat16: random weights give a router a near-tie every few dozen tokens
    (``decided_rows`` finds them in the plain implementation's routers), which bfloat16 rounding may decide the other
    way; that moves the token's row, and through the convolutions and the peaked attention some of the rows after it, by
    far more than rounding does.  So in bfloat16 the rows must be finite, three in four of them within the tolerance and
    the median row well inside it; a wrong key, mask or state would move nearly all rows.  ``strict`` (a mask) names the
    rows before a sequence's first near-tie: of those, nine in ten must be within the tolerance.  The float32 runs, on
    the same kernels and cache, excuse no row."""
    e = row_errors(got, ref)
    if dtype in (torch.float32, "float32"):
        return bool(e.max() <= TOL[torch.float32])
    if not np.isfinite(np.asarray(got)).all():
        return False
    strict = np.ones(len(e), dtype=bool) if strict is None else np.asarray(strict, dtype=bool)
    tol = TOL[torch.bfloat16]
    return bool(int((e[strict] > tol).sum()) <= 0.1 * max(1, int(strict.sum())) and int((e > tol).sum()) <= 0.25 * len(e)
                and float(np.median(e)) <= 0.5 * tol)


def kernel_tol(dtype):
    return 2e-5 if dtype == torch.float32 else 1.6e-2


_FOLDERS = {}

# ---------------------------------------------------------------------------------------------------------
# CPU
# ---------------------------------------------------------------------------------------------------------

def test_config_registry_and_round_trip():
    from lite_lang_b200.config import ConfigError, config_from_dict, known_architectures
    assert "Tusipel" in known_architectures()
    cfg = config_from_dict(CASES["P"]["config"])
    assert config_from_dict(cfg.to_dict()) == cfg
    spec = cfg.model_spec()
    assert [l.block for l in spec.layers] == ["pre_norm_conv", "pre_norm_conv", "pre_norm_conv_mixer_only", "pre_norm_conv"]
    assert [l.parts["mixer"].kind for l in spec.layers] == ["modulated_attention", "latent_attention"] + ["modulated_attention"] * 2
    a = spec.layers[0].parts["mixer"].params
    assert a["mask"] == "chunk" and a["mask_size"] == 23 and a["conv"] == 4 and a["value_head_dim"] == 40 and a["scale"] == 0.5
    assert a["distance_slopes"] == tuple(2.0 ** (-8.0 * (h + 1) / 6) for h in range(6))
    lat = spec.layers[1].parts["mixer"].params
    assert lat["q_rank"] == 19 and lat["kv_rank"] == 37 and lat["window"] == 17 and lat["rot_dims"] == 4
    assert lat["rot_layout"] == "half_split" and lat["channel_gate"] and lat["rot_scaling"]["factor"] == 4.0
    moe = spec.layers[1].parts["feed_forward"].params
    assert (moe["experts"], moe["identity"], moe["top"], moe["expert_ff"], moe["groups"]) == (5, 3, 3, 20, (4, 2))
    assert moe["weight_scale"] == 1.5 and moe["correction"] and moe["score"] == "softmax" and moe["gate_form"] == "silu"
    dense = spec.layers[0].parts["feed_forward"].params
    assert dense["activation"] == "clamped_swish" and dense["limit"] == 0.7 and dense["swish_alpha"] == 1.702
    assert spec.embedding.params["scale"] == 2.5 and "tied_to" not in spec.head.params
    assert spec.layers[2].parts["mixer_conv"].params["taps"] == 3 and spec.final_norm.params["offset"] == 1.0
    # the range 1..2 runs three times; every pass but the first starts with the embedding's output
    assert [(r.layer, r.add_embedding) for r in spec.order] == [(0, False), (1, False), (2, False), (1, True), (2, False),
                                                               (1, True), (2, False), (3, False)]
    # no loop section, no mask section
    r = config_from_dict(CASES["R"]["config"])
    assert [s.layer for s in r.run_order()] == [0, 1, 2, 3] and not any(s.add_embedding for s in r.run_order())
    assert r.model_spec().layers[0].parts["mixer"].params["mask"] == "causal"
    assert r.model_spec().layers[2].parts["mixer"].params["window"] is None
    for path, value in ((("layers", 0, "type"), "attention_9"), (("layers", 0, "mixer", "kv_heads"), 4),
                        (("layers", 1, "mixer", "rot", "dims"), 3), (("layers", 0, "mlp", "kind"), "gated"),
                        (("layers", 0, "mixer", "mask", "size"), 0), (("layers", 0, "mlp", "limit"), 0.0),
                        (("layers", 1, "mlp", "router", "groups", "count"), 3), (("layers", 1, "mlp", "router", "top"), 5),
                        (("layers", 1, "mlp", "router", "groups", "keep"), 5), (("loop", "stop"), 5), (("loop", "times"), 0),
                        (("canon", "taps"), 0)):
        bad = cfg.to_dict()
        d = bad
        for key in path[:-1]:
            d = d[key]
        d[path[-1]] = value
        with pytest.raises(ConfigError):
            config_from_dict(bad)
    for key, sub in (("norm", None), ("canon", None), ("embedding", None), ("conv", 0), ("q_rank", 1), ("scale", 2)):
        bad = cfg.to_dict()
        del (bad if sub is None else bad["layers"][sub]["mixer"])[key]
        with pytest.raises(ConfigError):
            config_from_dict(bad)


def test_cache_groups_and_declared_tensors():
    from lite_lang_b200.config import config_from_dict
    from lite_lang_b200.engine.model import CausalLM
    from lite_lang_b200.ops import conv_record_floats
    model = CausalLM(config_from_dict(CASES["P"]["config"]).model_spec())
    # a run of a layer has planes of its own: layers 1 and 2 run three times
    paged = sorted((g.num_kv_heads, g.head_dim, g.value_dim, g.window, g.chunk, g.planes)
                   for g in model.cache_groups if g.kind == "paged")
    assert paged == [(1, 36, 20, None, 9, 3), (1, 43, 0, 17, None, 3), (2, 24, 40, None, 23, 1), (4, 20, 28, None, 64, 1)]
    state = {g.shape: (g.planes, g.dtype) for g in model.cache_groups if g.kind == "state"}
    canon = (conv_record_floats(3, 88),)
    # two convolutions a layer run, one where there is no feed-forward: 2 + 3 (2 + 1) + 2
    assert state[canon] == (13, "float32")
    assert state[(conv_record_floats(4, 6 * 24 + 2 * 64),)] == (1, "float32")
    assert state[(conv_record_floats(2, 36 + 56),)] == (3, "float32")
    assert conv_record_floats(4, 272) == 2 * 3 * 272 + 4 and conv_record_floats(1, 90) == 4 and conv_record_floats(2, 5) == 12
    names = model.declared_tensors()
    for n, shape in (("embed", (211, 88)), ("head", (211, 88)), ("final.norm", (88,)), ("l0.norm1", (88,)), ("l0.canon1", (88, 3)),
                     ("l0.canon2", (88, 3)), ("l0.mix.q", (144, 88)), ("l0.mix.k.conv", (48, 4)), ("l0.mix.v.conv", (80, 4)),
                     ("l0.mix.q.conv", (144, 4)), ("l0.mix.o", (88, 240)), ("l0.mlp.gate", (50, 88)), ("l0.mlp.down", (88, 50)),
                     ("l1.mix.dq", (19, 88)), ("l1.mix.dq.norm", (19,)), ("l1.mix.uq", (78, 19)), ("l1.mix.dkv", (43, 88)),
                     ("l1.mix.g", (36, 88)), ("l1.mix.uk", (60, 37)), ("l1.mix.o", (88, 36)), ("l1.mlp.router", (8, 88)),
                     ("l1.mlp.correction", (8,)), ("l1.mlp.e4.gate", (20, 88)), ("l1.mlp.e4.down", (88, 20)),
                     ("l2.canon1", (88, 3)), ("l3.mlp.e5.up", (28, 88))):
        assert tuple(names[n].shape) == shape, n
    assert not names["head"].optional
    for n in ("l2.norm2", "l2.canon2", "l2.mlp.up", "l1.mlp.e5.up", "l1.mix.q", "l0.mix.g", "l1.mix.dq.conv", "l1.mix.sink"):
        assert n not in names, n


def test_what_blocks_hand_on_as_pending():
    from lite_lang_b200.parts.base import Pending, ResidualCopy, settled, whole_output, with_extra
    g = torch.Generator().manual_seed(1)
    y, rows, extra = (torch.randn(5, 8, generator=g) for _ in range(3))
    w = torch.rand(5, generator=g)
    parts = torch.randn(3, 5, 8, generator=g)
    assert torch.equal(settled(y, torch.float32), y) and settled(None, torch.float32) is None
    assert settled(Pending(), torch.float32) is None
    got = settled(Pending(parts, rows, w, extra), torch.float32)
    assert torch.allclose(got, parts.sum(0) + rows * w[:, None] + extra)
    assert torch.equal(settled(with_extra(None, extra), torch.float32), extra)
    assert torch.equal(settled(with_extra(ResidualCopy(y), extra), torch.float32), extra)
    assert torch.allclose(settled(with_extra(with_extra(y, extra), extra), torch.float32), y + 2 * extra)
    assert torch.allclose(whole_output(Pending(y, rows, w), torch.float32), y + rows * w[:, None])
    with pytest.raises(TypeError):
        with_extra((y, y), extra)


def test_parts_refuse_what_is_not_built():
    from lite_lang_b200.config.spec import PartSpec
    from lite_lang_b200.parts import build_part
    base = {"hidden_size": 16, "experts": 4, "top": 2, "expert_ff": 8, "gated": True, "gate_form": "silu"}
    for bad in ({"groups": (3, 1)}, {"groups": (2, 3)}, {"groups": (4, 1)}, {"gate_form": "relu"}, {"gate_form": "clamped_swish"},
                {"identity": 300}):
        with pytest.raises(ValueError):
            build_part("feed_forward", PartSpec("routed_experts", {**base, **bad}))
    att = {"hidden_size": 16, "num_heads": 2, "num_kv_heads": 1, "head_dim": 8}
    for bad in ({"distance_slopes": (0.5,)}, {"conv": 3, "qkv_bias": True}, {"conv": 100},
                {"distance_slopes": (0.5, 0.2), "head_mix": True}):
        with pytest.raises(ValueError):
            build_part("mixer", PartSpec("modulated_attention", {**att, **bad}))
    with pytest.raises(ValueError):
        build_part("feed_forward", PartSpec("gated_mlp", {"hidden_size": 8, "intermediate_size": 8, "activation": "clamped_swish"}))
    conv = build_part("mixer", PartSpec("modulated_attention", {**att, "conv": 3}))
    assert conv.cache_need() is None and [n for n, _ in conv.sub_mixers()] == ["kv", "conv"]
    assert conv.sub_mixers()[1][1].cache_need().shape[0] == 2 * 2 * 32 + 4


def test_plain_pieces_against_closed_forms():
    g = torch.Generator().manual_seed(0)
    # the convolution: the last tap weighs the token itself; zeros before the start
    x = torch.randn(6, 3, generator=g, dtype=P.F)
    cw = torch.randn(3, 4, generator=g, dtype=P.F)
    y = P.causal_convolution(x, cw)
    assert torch.allclose(y[0], cw[:, 3] * x[0])
    assert torch.allclose(y[4], cw[:, 0] * x[1] + cw[:, 1] * x[2] + cw[:, 2] * x[3] + cw[:, 3] * x[4])
    assert torch.allclose(P.with_convolution(x, cw[:, 3:]), x * (1 + cw[:, 3]))
    # chunks counted from the first token, windows that move
    v = P.visible_chunk(10, 4)
    assert v[3].tolist() == [True] * 4 + [False] * 6 and v[4].tolist() == [False] * 4 + [True] + [False] * 5
    assert v[9].tolist() == [False] * 8 + [True, True] and P.visible_chunk(5, None)[4].all()
    w = P.visible_window(10, 4)
    assert w[9].tolist() == [False] * 6 + [True] * 4 and w[2].tolist() == [True] * 3 + [False] * 7
    # slopes: the last head's is 2^-8 whatever the number of heads
    assert P.slopes(8).tolist() == [2.0 ** -(h + 1) for h in range(8)] and float(P.slopes(5)[-1]) == 2.0 ** -8
    assert float(P.distance_penalty(7, 8)[2, 6, 1]) == 5 / 8
    # a penalty of a slope a head is a factor on the weights
    q, k, vv = torch.zeros(6, 2, 3, dtype=P.F), torch.zeros(6, 2, 3, dtype=P.F), torch.eye(6, dtype=P.F)[:, None].repeat(1, 2, 1)
    o = P.softmax_attention(q, k, vv, 1.0, P.visible_window(6, None), P.distance_penalty(6, 2))
    want = torch.exp(-P.slopes(2)[0] * (4 - torch.arange(5, dtype=P.F)))
    assert torch.allclose(o[4, 0, :5], want / want.sum()) and float(o[4, 0, 5]) == 0.0
    # groups: a group counts by its best; what is outside the kept groups cannot be chosen even if all else is negative
    c = torch.tensor([0.9, -5.0, -0.1, -0.2, -0.3, -0.4], dtype=P.F)
    assert P.choose(c, 3, 1, 2)[0] == [0, 1] and P.choose(c, 3, 2, 3)[0] == [0, 2, 3] and P.choose(c, 1, 1, 3)[0] == [0, 2, 3]
    assert abs(P.choose(c, 3, 1, 2)[1] - 1.0) < 1e-12 and abs(P.choose(c, 1, 1, 2)[1] - 0.1) < 1e-12
    # identities: with the identity alone chosen the output is the input times its weight
    wts = {"router": torch.zeros(2, 4, dtype=P.F), "correction": torch.tensor([0.0, 1.0], dtype=P.F),
           "e0.gate": torch.zeros(3, 4, dtype=P.F), "e0.up": torch.zeros(3, 4, dtype=P.F), "e0.down": torch.zeros(4, 3, dtype=P.F)}
    u = torch.randn(3, 4, generator=g, dtype=P.F)
    mlp = {"kind": "moe", "router": {"experts": 1, "identity": 1, "top": 1, "scale": 3.0}, "expert": {"ff": 3}}
    assert torch.allclose(P.routed_ff(u, mlp, wts, ""), 1.5 * u)
    # the clamped gate: beyond the limit only the limit counts
    one = {"gate": torch.full((1, 1), 1.0, dtype=P.F), "up": torch.full((1, 1), -1.0, dtype=P.F), "down": torch.ones(1, 1, dtype=P.F)}
    d = P.dense_ff(torch.tensor([[0.5], [9.0]], dtype=P.F), {"limit": 2.0}, one, "")
    assert torch.allclose(d[0], torch.tensor([0.5 / (1 + math.exp(-0.851)) * 0.5], dtype=P.F))
    assert torch.allclose(d[1], torch.tensor([2.0 / (1 + math.exp(-3.404)) * -1.0], dtype=P.F))
    # half-split pairs: channel 0 turns with channel 2
    t = P.rotate(torch.tensor([[[1.0, 0.0, 0.0, 0.0, 7.0]]], dtype=P.F), torch.tensor([3]), {"dims": 4, "base": 100.0})
    assert torch.allclose(t[0, 0], torch.tensor([math.cos(3.0), 0.0, math.sin(3.0), 0.0, 7.0], dtype=P.F))
    assert P.run_order({"layers": [0] * 4, "loop": {"start": 1, "stop": 3, "times": 2}}) == \
        [(0, False), (1, False), (2, False), (1, True), (2, False), (3, False)]


MISTAKES = {
    "window": ("visible_window", lambda f: lambda T, W: f(T, None if W is None else W + 1)),
    "chunk": ("visible_chunk", lambda f: lambda T, C: f(T, None if C is None else C + 1)),
    "slopes": ("distance_penalty", lambda f: lambda T, H: f(T, H) * 0.9),
    "oldest tap": ("causal_convolution", lambda f: lambda u, w: f(u, torch.cat([torch.zeros_like(w[:, :1]), w[:, 1:]], 1) if w.shape[1] > 1 else w)),
    "no convolution behind the norms": ("with_convolution", lambda f: lambda h, w: h),
    "norm weight not around zero": ("centred_norm", lambda f: lambda u, w, eps: f(u, w - 1.0, eps)),
    "embedding not added again": ("run_order", lambda f: lambda cfg: [(i, False) for i, _ in f(cfg)]),
    "groups": ("choose", lambda f: lambda c, count, keep, top: f(c, 1, 1, top)),
    "amplitude": ("scaled_frequencies", lambda f: lambda rot: (f(rot)[0], 1.0)),
    "unscaled frequencies": ("scaled_frequencies", lambda f: lambda rot: (f({**rot, "scaling": None})[0], f(rot)[1])),
    "rotation": ("rotate", lambda f: lambda u, pos, rot: u),
}


@pytest.mark.parametrize("mistake", sorted(MISTAKES))
def test_a_mistake_in_any_mechanism_would_show_in_the_logits(mistake, monkeypatch):
    """The cases' weights are such that a wrong mechanism, planted in the plain implementation, moves at least one row in
    twenty of the cases that have it by ten times what the float32 runs may differ by."""
    cases = {"groups": ("P", "W"), "amplitude": ("P",), "unscaled frequencies": ("P",), "window": ("P", "W"), "rotation": ("P", "Q"),
             "embedding not added again": ("P", "Q", "W")}.get(mistake, ("P", "Q", "W"))
    refs = {}
    for name in cases:
        folder, seqs, ref = _case(name)
        refs[name] = (P.read_model_folder(folder), seqs[0], ref[0])
    what, make = MISTAKES[mistake]
    monkeypatch.setattr(P, what, make(getattr(P, what)))
    for name, ((cfg, w), toks, ref) in refs.items():
        e = row_errors(P.forward(cfg, w, toks).numpy(), ref)
        assert float((e > 10 * TOL[torch.float32]).mean()) >= 0.05, (name, float(e.max()), float(np.median(e)))


# ---------------------------------------------------------------------------------------------------------
# GPU: kernels alone
# ---------------------------------------------------------------------------------------------------------

def _step(entries, ctx, slots):
    """The device arrays of a step whose entries bring ``entries[i]`` tokens after ``ctx[i]`` cached ones."""
    s = types.SimpleNamespace()

    def put(a):
        return torch.tensor(np.asarray(a), dtype=torch.int32, device=dev())

    s.req_slot = put(slots)
    s.token_req = put(np.repeat(np.arange(len(entries)), entries))
    s.positions = put(np.concatenate([np.arange(c, c + n) for n, c in zip(entries, ctx)]))
    s.cu_q = put(np.concatenate([[0], np.cumsum(entries)]))
    s.ctx_len = put(ctx)
    s.num_entries = len(entries)
    s.num_single = sum(1 for n in entries if n == 1) if all(n == 1 for n in entries) else 0
    s.status = torch.zeros(1, dtype=torch.int32, device=dev())
    return s


def _feeding(lens, cuts):
    """Steps that feed requests in portions: for each, [(request, first token, tokens)]."""
    at = [0] * len(lens)
    for k in range(max(len(c) for c in cuts)):
        who = []
        for r, c in enumerate(cuts):
            if k < len(c):
                who.append((r, at[r], c[k]))
                at[r] += c[k]
        yield who
    assert at == list(lens)


CUTS = ([37, 9, 64, 700], [[5, 1, 2, 20, 9], [1, 1, 1, 1, 5], [64], [2, 1, 690, 1, 6]])


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("W,taps", [(88, 3), (90, 4), (90, 1), (64, 6), (320, 2), (1536, 4), (1000, 3), (4608, 4), (2052, 1)])
def test_norm_and_convolution_in_portions_with_records_used_again(dtype, W, taps):
    """The residual sum, the norm and the convolution behind it for four requests fed in portions of unequal sizes (one
    token, fewer than the taps, hundreds), with what is pending in all its forms, through records that other requests
    held before, against the plain formulas on the whole sequences."""
    from lite_lang_b200 import ops
    g = torch.Generator().manual_seed(W + taps)
    lens, cuts = CUTS
    eps = 1e-5
    w = 1 + 0.3 * torch.randn(W, generator=g)
    cw = torch.randn(W, taps, generator=g)
    res = [torch.randn(n, W, generator=g) * 3 for n in lens]
    y = [torch.randn(n, W, generator=g).to(dtype) for n in lens]
    parts = [torch.randn(2, n, W, generator=g) for n in lens]
    rows = [torch.randn(n, W, generator=g).to(dtype) for n in lens]
    rw = [torch.rand(n, generator=g) for n in lens]
    extra = [torch.randn(n, W, generator=g) for n in lens]
    for form in ("y", "partial", "rows", "all", "none"):
        state = torch.full((6, ops.conv_record_floats(taps, W)), 7.0, device=dev())       # what another request left
        slots = [2, 0, 5, 3]
        for s in slots:
            state[s].zero_()                                                              # a slot is zeroed when opened
        got, got_res = [[] for _ in lens], [[] for _ in lens]
        for who in _feeding(lens, cuts):
            step = _step([c for _, _, c in who] + ([1, 1] if all(c == 1 for _, _, c in who) else []),
                         [a for _, a, _ in who] + ([0, 0] if all(c == 1 for _, _, c in who) else []),
                         [slots[r] for r, _, _ in who] + ([-1, -1] if all(c == 1 for _, _, c in who) else []))

            def cat(ts, dim=0):
                t = torch.cat([ts[r].narrow(dim, a, c) for r, a, c in who], dim=dim)
                pad = step.token_req.numel() - t.shape[dim]                               # (padding entries of a captured step)
                if pad:
                    t = torch.cat([t, torch.zeros_like(t.narrow(dim, 0, 1)).repeat_interleave(pad, dim)], dim=dim)
                return t.to(dev()).contiguous()

            r0 = cat(res)
            new = torch.full_like(r0, float("nan"))
            out = torch.full(r0.shape, float("nan"), dtype=dtype, device=dev())
            kw = {}
            if form in ("y", "all"):
                kw["delta"] = cat(y)
            if form == "partial":
                kw["delta"] = cat(parts, 1)
            if form in ("rows", "all"):
                kw.update(rows_in=cat(rows), rows_w=cat(rw))
            if form in ("rows", "all"):
                kw["extra"] = cat(extra)
            for _again in range(2):                     # a step that is run again at the same context changes nothing
                ops.norm_conv(out, r0, w.to(dev()), eps, res_out=new, conv_w=cw.t().contiguous().to(dev()), state=state,
                              step=step, **kw)
            o, n_ = out.float().cpu(), new.cpu()
            assert torch.equal(r0.cpu(), cat(res).cpu())                                  # the rows it reads stay as they are
            for r, _, c in who:
                got[r].append(o[:c])
                got_res[r].append(n_[:c])
                o, n_ = o[c:], n_[c:]
        for r in range(4):
            x = res[r].double()
            if form in ("y", "all"):
                x = x + y[r].double()
            if form == "partial":
                x = x + parts[r].double().sum(0)
            if form in ("rows", "all"):
                x = x + rows[r].double() * rw[r].double()[:, None] + extra[r].double()
            assert float((torch.cat(got_res[r]).double() - x).abs().max()) <= 4e-6 * float(x.abs().max())
            want = P.with_convolution(P.centred_norm(x, w.double() - 1, eps), cw.double())
            assert rel_err(torch.cat(got[r]).numpy(), want.numpy()) <= kernel_tol(dtype), (form, r)
        assert float(state[1].min()) == 7.0 and float(state[4].max()) == 7.0              # nobody's records are untouched
    # without a convolution: all rows in place, or chosen ones without a write
    r0 = res[3].to(dev()).clone()
    out = torch.empty(700, W, dtype=dtype, device=dev())
    ops.norm_conv(out, r0, w.to(dev()), eps, res_out=r0, delta=y[3].to(dev()))
    x = res[3].double() + y[3].double()
    want = P.centred_norm(x, w.double() - 1, eps)
    assert rel_err(out.float().cpu().numpy(), want.numpy()) <= kernel_tol(dtype)
    assert float((r0.cpu().double() - x).abs().max()) <= 4e-6 * float(x.abs().max())
    pick = torch.tensor([699, 0, 5, 5], dtype=torch.int32, device=dev())
    out = torch.empty(4, W, dtype=dtype, device=dev())
    r0 = res[3].to(dev())
    ops.norm_conv(out, r0, w.to(dev()), eps, delta=y[3].to(dev()), rows=pick)
    assert rel_err(out.float().cpu().numpy(), want[[699, 0, 5, 5]].numpy()) <= kernel_tol(dtype)


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("nh,nkv,hd,vd,ps,taps", [(6, 2, 24, 40, 4, 4), (1, 1, 36, 20, 8, 2), (8, 2, 64, 64, 16, 3), (3, 1, 5, 7, 4, 3),
                                                  (2, 1, 128, 128, 16, 1), (4, 2, 16, 16, 4, 6), (4, 2, 128, 64, 16, 4)])
def test_convolved_projections_go_into_the_cache(dtype, nh, nkv, hd, vd, ps, taps):
    """q beside the cache, k and v into their pages, in portions; and the same convolution added to its input."""
    from lite_lang_b200 import ops
    g = torch.Generator().manual_seed(hd * 10 + taps)
    rng = np.random.default_rng(hd)
    lens, cuts = CUTS
    qw, kw, vw = nh * hd, nkv * hd, nkv * vd
    C = qw + kw + vw
    width = (C + 7) // 8 * 8 + 8
    cw = torch.randn(C, taps, generator=g)
    u = [torch.randn(n, width, generator=g).to(dtype) for n in lens]
    n_pages = sum((n + ps - 1) // ps for n in lens) + 2
    order = rng.permutation(n_pages)
    table, at = [], 0
    for n in lens:
        k = (n + ps - 1) // ps
        table.append(order[at:at + k])
        at += k
    kc = torch.full((n_pages, nkv, ps, hd), float("nan"), dtype=dtype, device=dev())
    vc = torch.full((n_pages, nkv, ps, vd), float("nan"), dtype=dtype, device=dev())
    state = torch.full((6, ops.conv_record_floats(taps, C)), -3.0, device=dev())
    slots = [4, 1, 0, 2]
    for s in slots:
        state[s].zero_()
    state2 = state.clone()
    got = [[] for _ in lens]
    added = [[] for _ in lens]
    cwd = cw.t().contiguous().to(dev())
    for who in _feeding(lens, cuts):
        step = _step([c for _, _, c in who], [a for _, a, _ in who], [slots[r] for r, _, _ in who])
        x = torch.cat([u[r][a:a + c] for r, a, c in who]).to(dev())
        sm = np.concatenate([table[r][np.arange(a, a + c) // ps] * ps + np.arange(a, a + c) % ps for r, a, c in who])
        q = torch.full((x.shape[0], (qw + 7) // 8 * 8), float("nan"), dtype=dtype, device=dev())
        ops.short_conv(q[:, :qw], x, cwd, state, step,
                       store=(torch.tensor(sm, dtype=torch.int32, device=dev()), kc, vc, ps, qw, step.status))
        both = torch.full((x.shape[0], C), float("nan"), dtype=dtype, device=dev())
        ops.short_conv(both, x, cwd, state2, step, add_input=True)
        assert int(step.status.item()) == 0
        q, both = q[:, :qw].float().cpu(), both.float().cpu()
        for r, _, c in who:
            got[r].append(q[:c])
            added[r].append(both[:c])
            q, both = q[c:], both[c:]
    for r, n in enumerate(lens):
        y = P.causal_convolution(u[r][:, :C].double(), cw.double())
        assert rel_err(torch.cat(got[r]).numpy(), y[:, :qw].numpy()) <= kernel_tol(dtype)
        assert rel_err(torch.cat(added[r]).numpy(), (y + u[r][:, :C].double()).numpy()) <= kernel_tol(dtype)
        pages, place = table[r][np.arange(n) // ps], np.arange(n) % ps
        k = kc.cpu()[pages, :, place].reshape(n, kw)
        v = vc.cpu()[pages, :, place].reshape(n, vw)
        assert rel_err(k.float().numpy(), y[:, qw:qw + kw].numpy()) <= kernel_tol(dtype)
        assert rel_err(v.float().numpy(), y[:, qw + kw:].numpy()) <= kernel_tol(dtype)
    assert float(state[3].max()) == -3.0 and float(state[5].min()) == -3.0


def _paged(dtype, seqs_k, seqs_v, ps, nkv, hd, vd, rng, live):
    """Keys/values of several requests scattered over a pool whose other slots hold NaN.  ``live(r, page)`` says whether a
    logical page of request r is there; the others are -1 in the table, as when a chunk has given them back."""
    n_pages = sum((len(k) + ps - 1) // ps for k in seqs_k) + 3
    order = rng.permutation(n_pages)
    kc = torch.full((n_pages, nkv, ps, hd), float("nan"), dtype=dtype)
    vc = torch.full((n_pages, nkv, ps, vd), float("nan"), dtype=dtype)
    bt = torch.full((len(seqs_k), max((len(k) + ps - 1) // ps for k in seqs_k)), -1, dtype=torch.int32)
    at = 0
    for r, (k, v) in enumerate(zip(seqs_k, seqs_v)):
        for j in range(len(k)):
            if not live(r, j // ps):
                continue
            if bt[r, j // ps] < 0:
                bt[r, j // ps] = int(order[at])
                at += 1
            kc[bt[r, j // ps], :, j % ps] = k[j].to(dtype)
            vc[bt[r, j // ps], :, j % ps] = v[j].to(dtype)
    return kc.to(dev()), vc.to(dev()), bt.to(dev())


def _chunk_case(dtype, nh, nkv, hd, vd, ps, mask, size, lens, new, kernel, seed=0):
    """Prompt portions and single tokens of several requests in one launch, with slopes; pages no query sees are not
    there.  The last queries of every request are aimed (a large dot product with one key) at the keys on both sides of
    the mask's edge, and without a mask at a key far back."""
    from lite_lang_b200 import ops
    if kernel == "shaped":
        order = sorted(range(len(lens)), key=lambda r: new[r] != 1)
        lens, new = [lens[r] for r in order], [new[r] for r in order]
    rng = np.random.default_rng(hd + seed)
    g = torch.Generator().manual_seed(hd + seed)
    R, group = len(lens), nh // nkv
    ks = [torch.randn(n, nkv, hd, generator=g) for n in lens]
    ks = [k / k.norm(dim=-1, keepdim=True) * math.sqrt(hd) for k in ks]
    vs = [torch.randn(n, nkv, vd, generator=g) for n in lens]
    qs = [torch.randn(c, nh, hd, generator=g) for c in new]

    def first(p):
        return 0 if mask == "causal" else max(0, p - size + 1) if mask == "window" else p // size * size

    aimed = []
    for r in range(R):
        targets = [("far", lambda p: 1)] if mask == "causal" else [("in", first), ("out", lambda p: first(p) - 1)]
        for back, (which, where) in enumerate(targets):
            row, p = new[r] - 1 - back, lens[r] - 1 - back
            if row < 0 or not 0 <= where(p) <= p:
                continue
            for h in range(nh):
                qs[r][row, h] = 6.0 * ks[r][where(p), h // group]
            aimed.append((r, row, where(p), which))
    ks, vs, qs = ([t.to(dtype).float() for t in ts] for ts in (ks, vs, qs))
    kc, vc, bt = _paged(dtype, ks, vs, ps, nkv, hd, vd, rng, lambda r, page: page >= first(lens[r] - new[r]) // ps)
    step = _step(new, [n - c for n, c in zip(lens, new)], list(range(R)))
    n_tok = sum(new)
    proj = torch.cat([x.reshape(x.shape[0], -1) for x in qs]).to(dtype).to(dev())
    slopes = torch.tensor([2.0 ** (-8.0 * (h + 1) / nh) for h in range(nh)])
    out = torch.full((n_tok, nh * vd), float("nan"), dtype=dtype, device=dev())
    scale = 0.9 / math.sqrt(hd)
    if kernel == "blocks":
        ops.attention_modulated(out, proj, proj.stride(0), None, kc, vc, bt, step.token_req, step.req_slot, step.positions,
                                n_tok, nh, nkv, hd, vd, ps, mask, size, False, scale, None, None, step.status,
                                distance_slope=slopes.to(dev()))
    else:
        n_single = sum(1 for c in new if c == 1)
        tail = (nh, nkv, hd, vd, ps, mask, size, False, scale, step.status)
        head = (out, proj, proj.stride(0), False, None, None, kc, vc, bt)
        if n_single:
            stages = (max(lens) + 63) // 64 + 1 if mask == "causal" else (size + 62) // 64 + 1
            for want_parts in (32, 2):
                span = (stages + want_parts - 1) // want_parts
                ops.attn_shaped(*head, step.cu_q, step.ctx_len, step.req_slot, n_single, n_single * ((group + 127) // 128),
                                *tail, nsplit=(stages + span - 1) // span, span=span, distance_slope=slopes.to(dev()))
        if R > n_single:
            ops.attn_shaped(*head, step.cu_q[n_single:], step.ctx_len[n_single:], step.req_slot[n_single:], R - n_single,
                            ops.attn_shaped_blocks(new[n_single:], group), *tail, distance_slope=slopes.to(dev()))
    assert int(step.status.item()) == 0
    got, at = out.float().cpu(), 0
    for r in range(R):
        T, c = lens[r], new[r]
        q = torch.cat([torch.zeros(T - c, nh, hd, dtype=P.F), qs[r].double()])
        vis = P.visible_chunk(T, size) if mask == "chunk" else P.visible_window(T, size)
        o = P.softmax_attention(q, ks[r].double(), vs[r].double(), scale, vis, P.distance_penalty(T, nh))[-c:].reshape(c, nh * vd)
        assert rel_err(got[at:at + c].numpy(), o.numpy()) <= kernel_tol(dtype), (mask, size, r)
        for rr, row, j, which in aimed:
            if rr == r:             # the flattest head reads the key it is aimed at exactly if the mask shows it
                a = got[at + row].view(nh, vd)[-1]
                hit = float((a - vs[r][j, -1]).abs().max()) < 0.15 * float(vs[r][j, -1].abs().max())
                assert hit == (which != "out"), (mask, size, r, row, j, which)
        at += c
    return {w for *_, w in aimed}


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("nh,nkv,hd,vd,ps", [(6, 2, 24, 40, 4), (9, 1, 20, 28, 8), (1, 1, 36, 20, 4), (8, 2, 64, 64, 16),
                                             (2, 1, 128, 128, 64), (5, 5, 12, 20, 8)])
def test_chunks_and_slopes_a_block_a_token(dtype, nh, nkv, hd, vd, ps):
    seen = set()
    for mask, size in (("chunk", 23), ("chunk", 64), ("chunk", 9), ("chunk", 100), ("chunk", 1), ("chunk", 1000),
                       ("window", 40), ("causal", None)):
        seen |= _chunk_case(dtype, nh, nkv, hd, vd, ps, mask, size, [150, 61, 97, 300, 34], [40, 1, 97, 1, 5], "blocks")
    assert seen == {"in", "out", "far"}


@gpu
@pytest.mark.parametrize("nh,nkv,hd,vd,ps", [(8, 2, 64, 64, 16), (4, 4, 128, 128, 16), (2, 1, 128, 128, 64), (16, 8, 64, 128, 32),
                                             (7, 1, 128, 64, 16)])
def test_chunks_and_slopes_on_tensor_cores(nh, nkv, hd, vd, ps):
    seen = set()
    for mask, size in (("chunk", 44), ("chunk", 64), ("chunk", 77), ("chunk", 128), ("chunk", 130), ("chunk", 5), ("chunk", 1000),
                       ("window", 40), ("causal", None)):
        seen |= _chunk_case(torch.bfloat16, nh, nkv, hd, vd, ps, mask, size, [150, 61, 97, 300, 34, 700], [40, 1, 97, 1, 5, 1],
                            "shaped")
    assert seen == {"in", "out", "far"}


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_half_split_rotation_of_the_latents_parts_and_the_gate(dtype):
    from lite_lang_b200 import ops
    from lite_lang_b200.config.spec import PartSpec
    from lite_lang_b200.parts import build_part
    g = torch.Generator().manual_seed(2)
    for H, d, r, R, dims, sc in ((3, 20, 6, 37, 4, (4.0, 64, 32.0, 1.0)), (2, 48, 16, 64, 16, None), (1, 8, 4, 16, 4, (2.0, 16, 2.0, 1.0)),
                                 (4, 12, 8, 24, 0, None)):
        rot = {"dims": dims, "base": 5000.0}
        if sc:
            rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), sc))
        part = build_part("position", PartSpec("rope_computed", {"rotary_dim": dims, "theta": 5000.0, "layout": "half_split",
                                                                "scaling": rot.get("scaling") if dims else None}))
        n, ps = 13, 4
        pos = torch.tensor([0, 1, 2, 3, 50, 51, 511, 512, 4000, 4001, 7, 8, 100], dtype=torch.int32)
        proj = torch.randn(n, H * (d + r) + R + r, generator=g).to(dtype)
        kv = H * (d + r)
        cache = torch.full((5, 1, ps, R + r), float("nan"), dtype=dtype, device=dev())
        q_full = torch.full((n, H, R + r), float("nan"), dtype=dtype, device=dev())
        nw = 1 + 0.1 * torch.randn(R, generator=g)
        status = torch.zeros(1, dtype=torch.int32, device=dev())
        slot = torch.arange(n - 1, -1, -1, dtype=torch.int32, device=dev())
        freq = part.frequencies().float().to(dev()) if dims else torch.zeros(1, device=dev())
        ops.latent_prepare(proj.to(dev()), 0, kv, nw.to(dev()), 1e-5, freq, dims, pos.to(dev()), slot, cache, q_full, H, d, r, R,
                           status, amplitude=part.amplitude, half_split=True)
        want_q = P.rotate(proj[:, :kv].double().view(n, H, d + r)[:, :, d:], pos, rot)
        want_k = P.rotate(proj[:, None, kv + R:].double(), pos, rot)[:, 0]
        rows = cache.float().cpu().view(-1, R + r)[slot.cpu().long()]
        tol = 2e-4 if dtype == torch.float32 else 2e-2        # (float32 angles of positions in the thousands)
        assert float((q_full.float().cpu()[:, :, R:].double() - want_q).abs().max()) <= tol * float(want_q.abs().max())
        assert float((rows[:, R:].double() - want_k).abs().max()) <= tol * float(want_k.abs().max())
        c = P.unit_rms(proj[:, kv:kv + R].double(), 1e-5) * nw.double()
        assert rel_err(rows[:, :R].numpy(), c.numpy()) <= kernel_tol(dtype)
    for n, width in ((7, 36), (300, 128), (1, 5)):
        x, gate = torch.randn(n, width, generator=g).to(dtype), (torch.randn(n, width + 11, generator=g) * 3).to(dtype)
        xd = x.clone().to(dev())
        ops.gate_rows(xd, gate.to(dev())[:, 3:3 + width])
        want = x.double() * P.sigmoid(gate[:, 3:3 + width].double())
        assert rel_err(xd.float().cpu().numpy(), want.numpy()) <= kernel_tol(dtype)


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("M,K,I", [(5, 128, 200), (3, 96, 40), (24, 256, 130), (40, 320, 256), (200, 88, 50), (300, 256, 512), (16, 90, 33)])
@pytest.mark.parametrize("limit,alpha", [(0.7, 1.702), (7.0, 1.0)])
def test_clamped_gate_in_every_product(dtype, M, K, I, limit, alpha):
    """Inputs well beyond the limit on both sides, in every kernel that makes the gated product."""
    from lite_lang_b200 import ops
    ops.configure_matmul_precision()
    g = torch.Generator().manual_seed(M + I)
    x = torch.randn(M, K, generator=g).to(dtype)
    w = (torch.randn(2 * I, K, generator=g) * (2.0 * limit / math.sqrt(K))).to(dtype)
    got = ops.gated_linear(x.to(dev()), w.to(dev()), ops.GateAct("clamped_swish", limit, alpha)).float().cpu()
    a = (x.double() @ w[:I].double().T).clamp(max=limit)
    c = (x.double() @ w[I:].double().T).clamp(-limit, limit)
    want = a * P.sigmoid(alpha * a) * (c + 1)
    assert rel_err(got.numpy(), want.numpy()) <= (2e-5 if dtype == torch.float32 else 2.5e-2)


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hidden,E,ident,count,keep,top,scale,score", [
    (88, 5, 3, 4, 2, 3, 1.5, "softmax"), (96, 12, 4, 4, 3, 4, 2.0, "softmax"), (90, 3, 0, 1, 1, 3, 1.0, "softmax"),
    (64, 6, 0, 3, 2, 2, 0.8, "sigmoid"), (128, 60, 40, 10, 4, 7, 1.1, "softmax"), (40, 1, 1, 2, 1, 1, 3.0, "softmax"),
    (72, 200, 56, 16, 5, 8, 2.5, "softmax"), (64, 8, 4, 4, 4, 4, 1.0, "softmax")])
def test_router_groups_corrections_and_identities(dtype, hidden, E, ident, count, keep, top, scale, score):
    """Choice scores mostly negative (a group that is out must not come back as zeros), a few tokens and long portions."""
    from lite_lang_b200 import ops
    g = torch.Generator().manual_seed(E + hidden)
    n_out = E + ident
    w = torch.randn(n_out, hidden, generator=g) * 0.3
    corr = torch.randn(n_out, generator=g) * 0.2 - 0.4
    for n in (5, 1, 600):
        x = torch.randn(n, hidden, generator=g).to(dtype)
        gates = torch.full((n, E), float("nan"), device=dev())
        idx = torch.full((n, top), 99, dtype=torch.int32, device=dev())
        tw = torch.full((n, top), float("nan"), device=dev())
        iw = torch.full((n,), float("nan"), device=dev())
        ops.moe_router(x.to(dev()), w.to(dev()), gates, idx, tw, top, score, choice_bias=corr.to(dev()), groups=(count, keep),
                       weight_scale=scale, identity_w=iw)
        z = x.double() @ w.double().T
        s = torch.softmax(z, -1) if score == "softmax" else P.sigmoid(z)
        gates, idx, tw, iw = gates.cpu(), idx.cpu(), tw.cpu(), iw.cpu()
        compared = 0
        for t in range(n):
            chosen, margin = P.choose(s[t] + corr.double(), count, keep, top)
            if margin < 1e-5:
                continue
            compared += 1
            assert sorted(idx[t].tolist()) == sorted(chosen), t
            want = torch.zeros(n_out, dtype=P.F)
            want[chosen] = s[t, chosen] * scale
            assert torch.allclose(gates[t].double(), want[:E], atol=2e-6, rtol=1e-5)
            assert abs(float(iw[t]) - float(want[E:].sum())) <= 1e-5
            assert torch.allclose(tw[t].double(), want[idx[t].long()], atol=2e-6, rtol=1e-5)
        assert compared >= 0.9 * n


def _routed(hidden, E, ident, top, groups, scale, ff, dtype, g):
    from lite_lang_b200.config.spec import PartSpec
    from lite_lang_b200.parts import build_part
    part = build_part("feed_forward", PartSpec("routed_experts", {
        "hidden_size": hidden, "experts": E, "top": top, "expert_ff": ff, "gated": True, "gate_form": "silu", "score": "softmax",
        "correction": True, "groups": groups, "weight_scale": scale, "identity": ident}))
    w = {}
    for name, decl in part.tensors().items():
        std = 0.3 if name == "router" else 0.2 if name == "correction" else 0.1
        w[name] = (torch.randn(decl.shape, generator=g) * std).to(torch.bfloat16)
    part.load(lambda n: w[n], dtype, dev())
    return part, {k: v.double() for k, v in w.items()}


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hidden,E,ident,top,groups,ff", [(88, 5, 3, 3, (4, 2), 20), (96, 8, 8, 4, (4, 4), 24), (64, 2, 6, 2, (1, 1), 40),
                                                         (72, 6, 0, 2, (3, 2), 16), (128, 12, 4, 4, (4, 3), 64)])
def test_gated_experts_and_identities(dtype, hidden, E, ident, top, groups, ff):
    """A few tokens (all experts' products) and many (the chosen experts' alone, in bfloat16): the same sums, also for
    tokens whose every choice is an identity."""
    from lite_lang_b200 import ops
    from lite_lang_b200.parts.base import settled
    ops.configure_matmul_precision()
    g = torch.Generator().manual_seed(hidden + E)
    part, w = _routed(hidden, E, ident, top, groups, 1.7, ff, dtype, g)
    mlp = {"kind": "moe", "router": {"experts": E, "identity": ident, "top": top, "scale": 1.7,
                                     "groups": {"count": groups[0], "keep": groups[1]}}, "expert": {"ff": ff}}
    step = types.SimpleNamespace(captured=False)
    for n in (1, 9, 140):
        x = torch.randn(n, hidden, generator=g).to(dtype)
        out = settled(part.forward(x.to(dev()), step), torch.float32)
        out = (out.sum(0) if out.dim() == 3 else out).float().cpu()
        margins = []
        want = P.routed_ff(x.double(), mlp, w, "", margins)
        ok = margins[0] > 1e-4
        assert int(ok.sum()) >= 0.9 * n
        assert rel_err(out[ok].numpy(), want[ok].numpy()) <= (2e-5 if dtype == torch.float32 else 2.5e-2), n


# ---------------------------------------------------------------------------------------------------------
# GPU: the whole model through the runner, the cache manager, the replay tool and the scheduler
# ---------------------------------------------------------------------------------------------------------
def _case(name):
    if name not in _FOLDERS:
        folder = write_folder(name)
        cfg, w = P.read_model_folder(folder)
        rng = np.random.default_rng(CASES[name]["seed"])
        seqs = [[int(t) for t in rng.integers(0, cfg["vocab"], n)] for n in (150, 61, 97, 1, 34, 120)]
        refs, decided = [], []
        for s in seqs:
            margins = []
            refs.append(P.forward(cfg, w, s, margins=margins).numpy())
            decided.append(decided_rows(margins))
        _FOLDERS[name] = (folder, seqs, refs, decided)
    return _FOLDERS[name][:3]


def _strict(name, i, n=None):
    """The rows of sequence i (its first n) that bfloat16 is held to."""
    _case(name)
    n = len(_FOLDERS[name][1][i]) if n is None else n
    return np.arange(n) < _FOLDERS[name][3][i]


def _runner(folder, dtype, page_size, num_pages, slots=4, graphs=True, max_len=256):
    from lite_lang_b200.cache.manager import CacheManager
    from lite_lang_b200.config.base import load_config
    from lite_lang_b200.engine.model import CausalLM
    from lite_lang_b200.engine.runner import ModelRunner
    from lite_lang_b200.weights.loader import load_weights
    model = CausalLM(load_config(folder).model_spec())
    load_weights(model, folder, dtype, dev())
    n_paged = sum(1 for g in model.cache_groups if g.kind == "paged")
    mgr = CacheManager(model.cache_groups, [num_pages] * n_paged, page_size, slots, max_len)
    return mgr, ModelRunner(model, mgr, dev(), 512, cuda_graphs=graphs)


def _feed(runner, mgr, slot, toks, want=None):
    from lite_lang_b200.engine.batch import StepEntry
    assert runner.reserve(slot, len(toks))
    want = tuple(range(len(toks))) if want is None else want
    return runner.step([StepEntry(slot, toks, want)]).float().cpu().numpy().copy()


@gpu
def test_residual_after_every_layer_run():
    """The float32 residual stream after each layer run of a short prompt against the plain implementation's."""
    from lite_lang_b200.engine.batch import StepEntry
    from lite_lang_b200.parts.base import whole_output
    for name in ("P", "R", "W"):
        folder, seqs, _ = _case(name)
        cfg, w = P.read_model_folder(folder)
        layers = []
        P.forward(cfg, w, seqs[4], layers)
        mgr, runner = _runner(folder, torch.float32, CASES[name]["page_size"], 64, graphs=False)
        seen = []
        for block in runner.model.blocks:
            def wrapped(h, delta, step, caches, _f=block.forward):
                h, delta = _f(h, delta, step, caches)
                pending = 0 if delta is None else whole_output(delta, torch.float32).float()
                seen.append((h.float() + pending).cpu())
                return h, delta
            block.forward = wrapped
        s = mgr.open()
        assert runner.reserve(s, len(seqs[4]))
        runner.step([StepEntry(s, seqs[4], (0,))])
        assert len(seen) == len(layers) == len(runner.model.plan)
        for i, (a, b) in enumerate(zip(seen, layers)):
            assert float((a.double() - b).abs().max()) <= 2e-5 * float(b.abs().max()), (name, i)


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", ["P", "Q", "R", "W"])
def test_whole_decode_and_portions(name, dtype):
    folder, seqs, refs = _case(name)
    mgr, runner = _runner(folder, dtype, CASES[name]["page_size"], 256 // CASES[name]["page_size"])
    for i in (0, 3, 4):                                     # whole prompts (one of them a single token)
        s = mgr.open()
        assert close(_feed(runner, mgr, s, seqs[i]), refs[i], dtype, _strict(name, i)), f"{name} whole {i}"
        mgr.close(s)
    for i, tail in ((0, 120), (2, 40)):                     # a prompt, then many tokens one by one (captured steps):
        s, n = mgr.open(), len(seqs[i])                     # every window and chunk passes over decoded tokens
        head = n - tail
        got = [_feed(runner, mgr, s, seqs[i][:head])] + [_feed(runner, mgr, s, seqs[i][t:t + 1]) for t in range(head, n)]
        assert close(np.concatenate(got), refs[i], dtype, _strict(name, i)), f"{name} decode {i}"
        mgr.close(s)
    s, n = mgr.open(), len(seqs[1])                         # from the very first token on, one by one
    got = [_feed(runner, mgr, s, seqs[1][t:t + 1]) for t in range(n)]
    assert close(np.concatenate(got), refs[1], dtype, _strict(name, 1)), f"{name} token by token"
    mgr.close(s)
    sizes = [7, 2, 13, 2, 5, 31, 2, 3, 17, 2, 64, 2, 9]
    for i in (0, 5):                                        # portions of changing size, down to two tokens
        s, n, t, k, got = mgr.open(), len(seqs[i]), 0, 0, []
        while t < n:
            c = min(sizes[k % len(sizes)], n - t)
            got.append(_feed(runner, mgr, s, seqs[i][t:t + c]))
            t, k = t + c, k + 1
        assert close(np.concatenate(got), refs[i], dtype, _strict(name, i)), f"{name} portions {i}"
        mgr.close(s)
    runner.check_status()
    assert runner.graph_replays > 0


@gpu
def test_a_pool_smaller_than_the_prompt_serves_it_through_the_pages_given_back():
    """Every layer of this case has a window or chunks, so a request holds a bounded number of pages however long it
    grows: a prompt of several times the pool, fed in portions, and the logits are the whole prompt's."""
    folder = write_folder("W")
    ps = CASES["W"]["page_size"]
    cfg, w = P.read_model_folder(folder)
    toks = [int(t) for t in np.random.default_rng(21).integers(0, cfg["vocab"], 400)]
    ref = P.forward(cfg, w, toks).numpy()
    portion = 24
    pages = (20 + portion + ps - 1) // ps + 2
    assert pages * ps < len(toks) // 4
    mgr, runner = _runner(folder, torch.float32, ps, pages, slots=2, max_len=512)
    s, got = mgr.open(), []
    for t in range(0, 360, portion):
        got.append(_feed(runner, mgr, s, toks[t:t + portion]))
    got += [_feed(runner, mgr, s, toks[t:t + 1]) for t in range(360, 400)]
    assert close(np.concatenate(got), ref, torch.float32)
    mgr.close(s)
    mgr.check_invariants()
    runner.check_status()
    assert mgr.pages_reused > 0


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", ["P", "Q", "R", "W"])
def test_mixed_batches_with_pages_and_slots_used_again(name, dtype, monkeypatch):
    from lite_lang_b200.engine.batch import StepEntry
    monkeypatch.setenv("LITE_LANG_B200_CACHE_FILL", "nan")
    folder, seqs, refs = _case(name)
    ps = CASES[name]["page_size"]
    order = [0, 1, 2, 3, 4, 5, 1, 2, 0]
    need = sorted(((len(seqs[i]) + ps - 1) // ps for i in order), reverse=True)[:3]
    mgr, runner = _runner(folder, dtype, ps, sum(need) + 1, slots=3)
    rng = np.random.default_rng(3)
    waiting, live, all_got, all_ref, all_strict = list(enumerate(order)), {}, [], [], []
    while waiting or live:
        while waiting and len(live) < 3:
            k, i = waiting.pop(0)
            live[k] = [i, 0, mgr.open()]
        entries, expect, done = [], [], []
        for k, (i, t, slot) in list(live.items()):
            n = len(seqs[i])
            if len(live) > 1 and rng.random() < 0.2:
                continue                                    # left out of this step, goes on later
            c = min(int(rng.integers(2, 23)) if n - t > 20 else 1, n - t)
            assert runner.reserve(slot, c)
            want = tuple(range(c)) if rng.random() < 0.7 else (c - 1,)
            entries.append(StepEntry(slot, seqs[i][t:t + c], want))
            expect.append(refs[i][[t + w for w in want]])
            all_strict.append(_strict(name, i)[[t + w for w in want]])
            live[k][1] = t + c
            if t + c == n:
                done.append(k)
        if not entries:
            continue
        got = runner.step(entries).float().cpu().numpy()
        all_got.append(got.copy())
        all_ref.append(np.concatenate(expect))
        for k in done:
            mgr.close(live.pop(k)[2])
        mgr.check_invariants()
    runner.check_status()
    assert close(np.concatenate(all_got), np.concatenate(all_ref), dtype, np.concatenate(all_strict)), name
    assert mgr.pages_reused > 0


@gpu
def test_a_batch_gives_each_request_what_it_gets_alone():
    """In the attentions, the convolutions and the norms the order of every sum depends on the token's position only;
    what is left between a request alone and the same request beside others, in other pages and slots and cut
    otherwise, is the rounding of the matrix products, whose shapes differ (float32, where nothing else rounds)."""
    from lite_lang_b200.engine.batch import StepEntry
    folder, seqs, refs = _case("P")
    ps = CASES["P"]["page_size"]
    mgr, runner = _runner(folder, torch.float32, ps, 200, graphs=False)
    s = mgr.open()
    alone = _feed(runner, mgr, s, seqs[2])
    mgr.close(s)
    a, b, c = mgr.open(), mgr.open(), mgr.open()
    for slot, toks in ((a, seqs[1][:33]), (c, seqs[4][:9])):
        _feed(runner, mgr, slot, toks)
    got, t = [], 0
    for n in (5, 40, 2, 50):
        entries = [StepEntry(a, seqs[1][33 + len(got):34 + len(got)], (0,)), StepEntry(b, seqs[2][t:t + n], tuple(range(n)))]
        for e in entries:
            assert runner.reserve(e.slot, len(e.tokens))
        got.append(runner.step(entries).float().cpu().numpy()[1:].copy())
        t += n
    got = np.concatenate(got)
    assert float(np.abs(got - alone).max()) <= 5e-5 * float(np.abs(alone).max())


@gpu
def test_replay_tool_and_a_prompt_of_many_tokens_in_one_step():
    """The command-line replay on a folder: a prompt long enough for the prompt kernels, cut into three steps beside a
    short request that ends early."""
    folder = write_folder("Q")
    cfg, w = P.read_model_folder(folder)
    toks = [int(t) for t in np.random.default_rng(9).integers(0, cfg["vocab"], 260)]
    margins = []
    ref = P.forward(cfg, w, toks, margins=margins).numpy()
    ok = np.arange(260) < decided_rows(margins)
    for dtype in ("float32", "bfloat16"):
        tr = TraceRun(folder, dtype, max_tokens=384, page_size=16)
        try:
            a = tr.step([{"id": "a", "tokens": toks[:200], "want": list(range(0, 200, 7))}])
            b = tr.step([{"id": "a", "tokens": toks[200:259], "want": list(range(59))},
                         {"id": "b", "tokens": toks[:5], "want": [4]}], end=["b"])
            c = tr.step([{"id": "a", "tokens": toks[259:], "want": [0]}], end=["a"])
        finally:
            assert tr.close() == 0
        want = np.concatenate([ref[0:200:7], ref[200:259], ref[259:], ref[4:5]])
        assert close(np.concatenate([a, b[:59], c, b[59:]]), want, dtype,
                     np.concatenate([ok[0:200:7], ok[200:259], ok[259:], ok[4:5]]))


def _greedy_matches(cfg, w, prompt, out):
    seq = list(prompt)
    for tok in out:
        logits = P.forward(cfg, w, seq)[-1]
        top2 = torch.topk(logits, 2).values
        if float(top2[0] - top2[1]) < 1e-3:              # a near-tie: either token is right, stop comparing
            return
        assert int(torch.argmax(logits)) == tok, (len(prompt), len(seq))
        seq.append(tok)


@gpu
@pytest.mark.parametrize("name", ["R", "W"])
def test_greedy_generation_through_the_scheduler(name):
    """Engine.generate with more prompts than request slots: the tokens are the plain implementation's greedy
    continuation (float32, so that no near-tie decides)."""
    from lite_lang_b200 import Engine, EngineConfig, SamplingParams
    folder = write_folder(name)
    cfg, w = P.read_model_folder(folder)
    rng = np.random.default_rng(4)
    prompts = [[int(t) for t in rng.integers(0, cfg["vocab"], n)] for n in (9, 30, 1, 17, 44)]
    new = 12
    engine = Engine(folder, EngineConfig(dtype="float32", page_size=8, num_pages=40, max_batch_size=3,
                                         max_input_length=64, max_output_length=new, max_tokens_per_step=48))
    outs = engine.generate(prompts, SamplingParams(temperature=0.0, max_new_tokens=new, ignore_eos=True))
    for p, o in zip(prompts, outs):
        assert len(o) == new
        _greedy_matches(cfg, w, p, o)
    assert engine.stats()["graph_replays"] > 0


@gpu
def test_command_line_picks_the_model_by_its_configuration():
    folder = write_folder("P")
    cfg, w = P.read_model_folder(folder)
    prompt = [int(t) for t in np.random.default_rng(8).integers(0, cfg["vocab"], 11)]
    ids = os.path.join(folder, "prompt.json")
    with open(ids, "w") as fh:
        json.dump([prompt], fh)
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cmd = [sys.executable, "-m", "lite_lang_b200.cli", "--model_path", folder, "--prompt_ids", ids, "--dtype", "fp32",
           "--max_output_length", "6", "--page_size", "4", "--num_pages", "32", "--max_batch_size", "2",
           "--temperature", "0", "--ignore_eos"]
    res = subprocess.run(cmd, capture_output=True, text=True, cwd=root, timeout=600)
    assert res.returncode == 0, res.stderr[-2000:]
    out = json.loads(res.stdout.strip().splitlines()[-1])["outputs"][0]
    assert len(out) == 6
    _greedy_matches(cfg, w, prompt, out)
