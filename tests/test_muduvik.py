"""Muduvik through the engine against the plain implementation (tests/plain/muduvik_plain.py).

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
from muduvik_cases import CASES, write_folder
from plain import muduvik_plain as P

TOL = {torch.float32: 2e-4, torch.bfloat16: 6e-2}
gpu = pytest.mark.gpu


def dev():
    return torch.device("cuda:0")


def row_errors(got, ref):
    got, ref = np.asarray(got, dtype=np.float64), np.asarray(ref, dtype=np.float64)
    assert got.shape == ref.shape, (got.shape, ref.shape)
    return np.abs(got - ref).max(axis=-1) / np.abs(ref).max(axis=-1)


def close(got, ref, dtype) -> bool:
    """float32: every row within the tolerance.  bfloat16: where a token's gated table row or a head's read-out happens to be
    small, the norm behind it takes its direction from the rounding, and random weights give every few hundred tokens such
    a place; so 19 rows in 20 (all but three of a short sequence's) must be within the tolerance and the median row well inside it.  A wrong key, mask or state
    would move nearly all rows, and the float32 runs, on the same cache, excuse no row."""
    dtype = {"float32": torch.float32, "bfloat16": torch.bfloat16}.get(dtype, dtype)
    e = row_errors(got, ref)
    if dtype == torch.float32:
        return bool(e.max() <= TOL[dtype])
    return bool(np.isfinite(e).all() and (e > TOL[dtype]).sum() <= max(3, len(e) // 20) and np.median(e) <= 0.5 * TOL[dtype])


def kernel_tol(dtype):
    return 2e-5 if dtype == torch.float32 else 1.6e-2


_FOLDERS = {}


def _case(name):
    if name not in _FOLDERS:
        folder = write_folder(name)
        cfg, w = P.read_model_folder(folder)
        rng = np.random.default_rng(CASES[name]["seed"])
        seqs = [[int(t) for t in rng.integers(0, cfg["vocab"], n)] for n in (150, 61, 97, 1, 34, 120)]
        _FOLDERS[name] = (folder, seqs, [P.forward(cfg, w, s).numpy() for s in seqs])
    return _FOLDERS[name]


# ---------------------------------------------------------------------------------------------------------
# CPU
# ---------------------------------------------------------------------------------------------------------

def test_config_registry_and_round_trip():
    from lite_lang_b200.config import ConfigError, config_from_dict, known_architectures
    assert "Muduvik" in known_architectures()
    cfg = config_from_dict(CASES["P"]["config"])
    assert config_from_dict(cfg.to_dict()) == cfg
    spec = cfg.model_spec()
    full, short = "sandwich_token_side", "sandwich_token_side_mixer_only"
    assert [l.block for l in spec.layers] == [full, full, short, full, short]
    kinds = ["modulated_attention", "retention", "modulated_attention", "latent_attention", "retention"]
    assert [l.parts["mixer"].kind for l in spec.layers] == kinds
    a = spec.layers[0].parts["mixer"].params
    assert (a["num_heads"], a["num_kv_heads"], a["head_dim"], a["value_head_dim"]) == (6, 2, 12, 36)
    assert a["differential"] == {"diff": 0.35} and a["mask"] == "window" and a["mask_size"] == 23 and a["head_gate"]
    assert a["qk_norm"] == "head" and a["qkv_bias"] and a["scale"] == 0.35
    pos = a["position"].params
    assert pos["layout"] == "interleaved" and pos["rotary_dim"] == 8 and pos["scaling"]["high"] == 4.0
    ret = spec.layers[1].parts["mixer"].params
    assert ret["decay"] == [0.75, 0.96875, 0.9921875] and ret["key_scale"] == 10 ** -0.5
    assert ret["position"].params["layout"] == "half_split" and ret["position"].params["rotary_dim"] == 6
    lat = spec.layers[3].parts["mixer"].params
    assert lat["rot_dim"] == 0 and lat["q_rank"] == 19 and lat["kv_rank"] == 37 and lat["window"] is None
    assert spec.layers[0].parts["feed_forward"].params["activation"] == "gelu_tanh"
    side = [l.parts["token_side"].params for l in spec.layers]
    assert [s["index"] for s in side] == [0, 1, 2, 3, 4] and {s["layers"] for s in side} == {5} and side[0]["dim"] == 11
    assert spec.embedding.params["norm"]["tensor"] == "embed.norm" and "tied_to" not in spec.head.params
    # the range 1..2 runs three times, each pass with its own row; the parts of a layer are the same in every pass
    assert [(r.layer, r.add_row) for r in spec.order] == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None),
                                                         (3, None), (4, None)]
    assert spec.pass_rows.params["rows"] == 3
    r = config_from_dict(CASES["R"]["config"])
    assert [s.layer for s in r.run_order()] == [0, 1, 2, 3, 4] and r.model_spec().pass_rows is None
    assert r.model_spec().layers[3].parts["mixer"].params["position"] is None          # rot.dims 0
    assert config_from_dict(CASES["Q"]["config"]).model_spec().layers[4].parts["mixer"].params["mask"] == "causal"
    for path, value in ((("layers", 0, "type"), "attention_9"), (("layers", 0, "mixer", "kv_heads"), 4),
                        (("layers", 0, "mixer", "rot", "dims"), 14), (("layers", 1, "mixer", "rot", "dims"), 3),
                        (("layers", 0, "mlp", "kind"), "moe"), (("layers", 0, "mixer", "mask", "size"), 0),
                        (("layers", 1, "mixer", "decay"), [0.5, 0.5]), (("loop", "stop"), 6), (("loop", "times"), 0),
                        (("loop", "start"), 3), (("token_side", "dim"), 0), (("layers", 3, "mixer", "q_rank"), 0)):
        bad = cfg.to_dict()
        d = bad
        for key in path[:-1]:
            d = d[key]
        d[path[-1]] = value
        with pytest.raises(ConfigError):
            config_from_dict(bad)
    for key, sub in (("norm", None), ("token_side", None), ("diff", 0), ("scale", 0), ("kv_rank", 3), ("decay", 1), ("vdim", 4)):
        bad = cfg.to_dict()
        del (bad if sub is None else bad["layers"][sub]["mixer"])[key]
        with pytest.raises(ConfigError):
            config_from_dict(bad)


def test_cache_groups_and_declared_tensors():
    from lite_lang_b200.config import config_from_dict
    from lite_lang_b200.engine.model import CausalLM
    model = CausalLM(config_from_dict(CASES["P"]["config"]).model_spec())
    # a cached key is its two maps' parts side by side; a pass of a layer has a plane of its own
    paged = sorted((g.num_kv_heads, g.head_dim, g.value_dim, g.window, g.planes) for g in model.cache_groups if g.kind == "paged")
    assert paged == [(1, 37, 0, None, 1), (2, 24, 36, 23, 1), (4, 40, 28, 9, 3)]
    state = {g.shape: (g.planes, g.dtype) for g in model.cache_groups if g.kind == "state"}
    assert state == {(3 * 30 * 10,): (3, "float32"), (2 * 22 * 18,): (1, "float32")}
    names = model.declared_tensors()
    for n, shape in (("embed", (211, 88)), ("embed.norm", (88,)), ("loop.step", (3, 88)), ("side.embed", (211, 55)),
                     ("head", (211, 88)), ("final.norm", (88,)), ("l0.norm1", (88,)), ("l0.norm1b", (88,)), ("l0.norm2b", (88,)),
                     ("l0.ls1", (88,)), ("l0.ls2", (88,)), ("l0.mix.q", (144, 88)), ("l0.mix.q.b", (144,)), ("l0.mix.k", (48, 88)),
                     ("l0.mix.v.b", (72,)), ("l0.mix.q.norm", (12,)), ("l0.mix.lk2", (12,)), ("l0.mix.g", (6, 88)),
                     ("l0.mix.o", (88, 216)), ("l0.mlp.gate", (50, 88)), ("l0.side.gate", (11, 88)), ("l0.side.proj", (88, 11)),
                     ("l0.side.norm", (88,)), ("l1.mix.q", (30, 88)), ("l1.mix.g", (90, 88)), ("l1.mix.o", (88, 90)),
                     ("l2.ls1", (88,)), ("l3.mix.dq", (19, 88)), ("l3.mix.dq.norm", (19,)), ("l3.mix.uq", (60, 19)),
                     ("l3.mix.dkv", (37, 88)), ("l3.mix.dkv.norm", (37,)), ("l3.mix.uk", (60, 37)), ("l3.mix.uv", (36, 37))):
        assert tuple(names[n].shape) == shape, n
    for n in ("l2.norm2", "l2.norm2b", "l2.ls2", "l2.mlp.up", "l1.mix.q.b", "l1.mix.norm", "l3.mix.q", "l3.mix.g", "l0.mix.talk"):
        assert n not in names, n
    plain = CausalLM(config_from_dict(CASES["R"]["config"]).model_spec()).declared_tensors()
    assert "loop.step" not in plain and tuple(plain["side.embed"].shape) == (97, 35)


def test_what_blocks_hand_on_as_pending():
    from lite_lang_b200.parts.base import NormedOutput, Pending, settled, with_extra, with_row
    g = torch.Generator().manual_seed(1)
    y, extra = torch.randn(5, 8, generator=g), torch.randn(5, 8, generator=g)
    w, row, row2 = (torch.randn(8, generator=g) for _ in range(3))
    parts = torch.randn(3, 5, 8, generator=g)
    want = y / torch.sqrt((y * y).mean(-1, keepdim=True) + 0.5) * w
    assert torch.allclose(settled(NormedOutput(y, w, 0.5), torch.float32), want, atol=1e-6)
    assert settled(NormedOutput(None), torch.float32) is None
    s = parts.sum(0)
    want_parts = s / torch.sqrt((s * s).mean(-1, keepdim=True) + 0.5) * w
    assert torch.allclose(NormedOutput(parts, w, 0.5, row).gain(), want_parts + row, atol=1e-6)
    p = with_row(with_row(NormedOutput(y, w, 0.5), row, 5), row2, 5)
    assert isinstance(p, NormedOutput) and torch.allclose(p.gain(), want + row + row2, atol=1e-6)
    assert torch.equal(with_row(None, row, 5).gain(), row[None])
    both = with_row(Pending(y=y), row, 5)               # (a pending output without a norm of its own)
    assert torch.allclose(settled(both, torch.float32), y + row)
    assert torch.allclose(settled(with_extra(p, extra), torch.float32), want + row + row2 + extra, atol=1e-6)


def test_parts_refuse_what_is_not_built():
    from lite_lang_b200.config.spec import ModelSpec, PartSpec, RunStep
    from lite_lang_b200.engine.model import CausalLM
    from lite_lang_b200.parts import build_part
    att = {"hidden_size": 16, "num_heads": 2, "num_kv_heads": 1, "head_dim": 8, "differential": {"diff": 0.5}}
    for bad in ({"head_mix": True}, {"sink": True}, {"conv": 3}, {"channel_gate": True}, {"qk_norm": "projection"},
                {"distance_slopes": (0.5, 0.2)}, {"head_temperature": True}, {"distance_bias": {"max": 8}}):
        with pytest.raises(ValueError):
            build_part("mixer", PartSpec("modulated_attention", {**att, **bad}))
    ret = {"hidden_size": 16, "heads": 2, "key_dim": 8, "value_dim": 8, "decay": [0.5, 0.5], "eps": 1e-6}
    stretched = PartSpec("rope_computed", {"rotary_dim": 8, "theta": 100.0,
                                           "scaling": {"factor": 4.0, "original": 64, "fast": 32.0, "slow": 1.0}})
    for bad in ({"decay": [0.5]}, {"key_dim": 300}, {"position": stretched}):
        with pytest.raises(ValueError):
            build_part("mixer", PartSpec("retention", {**ret, **bad}))
    with pytest.raises(ValueError):
        build_part("feed_forward", PartSpec("token_side", {"hidden_size": 8, "vocab_size": 9, "dim": 2, "index": 3, "layers": 3}))
    with pytest.raises(ValueError):
        build_part("embedding", PartSpec("token_embedding", {"vocab_size": 9, "hidden_size": 8, "scale": 2.0, "residual": "float32",
                                                            "norm": {"tensor": "n", "eps": 1e-6}}))
    norm = PartSpec("rms_norm_f32_sandwich", {"hidden_size": 8, "eps": 1e-6})
    with pytest.raises(ValueError, match="pass_rows"):
        CausalLM(ModelSpec("X", 8, 9, 64, PartSpec("token_embedding", {"vocab_size": 9, "hidden_size": 8}), (),
                           (RunStep(0, add_row=1),), norm, PartSpec("lm_head", {"vocab_size": 9, "hidden_size": 8})))


def test_frequencies_by_wavelength():
    """Kept, divided and in between, on both sides of both bounds and on them."""
    from lite_lang_b200.config.spec import PartSpec
    from lite_lang_b200.parts import build_part
    for base, dims, sc in ((900.0, 8, (4.0, 1.0, 4.0, 64)), (250.0, 64, (8.0, 1.0, 4.0, 512)), (1e6, 128, (32.0, 0.5, 3.0, 8192)),
                           (10.0, 2, (2.0, 1.0, 2.0, 2 * math.pi))):
        keys = dict(zip(("factor", "low", "high", "original"), sc))
        part = build_part("position", PartSpec("rope_computed", {"rotary_dim": dims, "theta": base, "scaling": keys}))
        want = P.frequencies({"dims": dims, "base": base, "scaling": keys})
        assert torch.allclose(part.frequencies(), want, rtol=1e-12, atol=0) and part.amplitude == 1.0
        plain = P.frequencies({"dims": dims, "base": base})
        ratio = want / plain
        assert float(ratio.max()) <= 1 + 1e-12 and float(ratio.min()) >= 1 / sc[0] - 1e-12
        if dims > 8:
            assert float(ratio[0]) == 1.0 and abs(float(ratio[-1]) - 1 / sc[0]) < 1e-12
            assert ((ratio > 1.01 / sc[0]) & (ratio < 0.99)).any()
    for bad in ({"factor": 2.0, "low": 2.0, "high": 2.0, "original": 64}, {"factor": 0.0, "low": 1.0, "high": 4.0, "original": 64}):
        with pytest.raises(ValueError):
            build_part("position", PartSpec("rope_computed", {"rotary_dim": 8, "theta": 10.0, "scaling": bad}))


def test_plain_pieces_against_closed_forms():
    g = torch.Generator().manual_seed(0)
    # retention: a decay of 1 and equal keys sum all values; a small one forgets
    q = k = torch.ones(5, 2, 1, dtype=P.F)
    v = torch.arange(1, 6, dtype=P.F)[:, None, None].repeat(1, 2, 1)
    o = P.decayed_sums(q, k, v, torch.tensor([1.0, 0.5], dtype=P.F))
    assert o[:, 0, 0].tolist() == [1, 3, 6, 10, 15] and o[2, 1, 0].item() == 1 * 0.25 + 2 * 0.5 + 3
    # two maps: equal maps leave (1 - lambda) of either, whose size the norm takes out again
    a = torch.randn(3, 2, 8, generator=g, dtype=P.F)
    z = P.combine_maps(a, a, 0.25, 0.4, 0.0)
    assert torch.allclose(z, 0.6 * a / torch.sqrt((a * a).mean(-1, keepdim=True)))
    assert torch.allclose(P.combine_maps(a, a, 2.0, 0.4, 0.0), -z)
    w = {"lq1": torch.tensor([1.0, 2.0]), "lk1": torch.tensor([0.5, 0.0]), "lq2": torch.zeros(2), "lk2": torch.ones(2)}
    assert abs(P.map_weight({"diff": 0.3}, w, "") - (math.exp(0.5) - 1.0 + 0.3)) < 1e-6
    # rotations: neighbours and halves
    t = P.rotate_neighbours(torch.tensor([[[1.0, 0.0, 1.0, 0.0, 7.0]]], dtype=P.F), torch.tensor([3]), {"dims": 4, "base": 100.0})
    assert torch.allclose(t[0, 0], torch.tensor([math.cos(3), math.sin(3), math.cos(0.3), math.sin(0.3), 7.0], dtype=P.F))
    t = P.rotate_halves(torch.tensor([[[1.0, 1.0, 0.0, 0.0, 7.0]]], dtype=P.F), torch.tensor([3]), {"dims": 4, "base": 100.0})
    assert torch.allclose(t[0, 0], torch.tensor([math.cos(3), math.cos(0.3), math.sin(3), math.sin(0.3), 7.0], dtype=P.F))
    vis = P.visible(10, 4)
    assert vis[9].tolist() == [False] * 6 + [True] * 4 and vis[2].tolist() == [True] * 3 + [False] * 7
    assert torch.allclose(P.gelu_tanh(torch.tensor([0.7], dtype=P.F)),
                          torch.nn.functional.gelu(torch.tensor([0.7], dtype=P.F), approximate="tanh"))
    table = {"side.embed": torch.arange(12, dtype=P.F).view(2, 6)}
    assert P.side_slice(torch.tensor([1, 0]), 1, 2, table).tolist() == [[8, 9], [2, 3]]
    assert P.run_order({"layers": [0] * 4, "loop": {"start": 1, "stop": 3, "times": 2}}) == \
        [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]


MISTAKES = {
    "window": ("visible", lambda f: lambda T, W: f(T, None if W is None else W + 1)),
    "second map's weight": ("map_weight", lambda f: lambda m, w, p: float(m["diff"])),
    "no second map": ("combine_maps", lambda f: lambda a1, a2, lam, diff, eps: f(a1, 0.0 * a2, lam, diff, eps)),
    "no norm a head": ("normed_parts", lambda f: lambda z, w, eps: z),
    "unscaled frequencies": ("frequencies", lambda f: lambda rot: f({**rot, "scaling": None})),
    "neighbours as halves": ("rotate_neighbours", lambda f: P.rotate_halves),
    "halves as neighbours": ("rotate_halves", lambda f: P.rotate_neighbours),
    "decay": ("decayed_sums", lambda f: lambda q, k, v, d: f(q, k, v, d * 0.97)),
    "layer scale": ("output_norm", lambda f: lambda y, w, ls, eps: P.norm(y, w, eps)),
    "passes without rows": ("run_order", lambda f: lambda cfg: [(i, None) for i, _ in f(cfg)]),
    "first pass without its row": ("run_order", lambda f: lambda cfg: [(i, r or None) for i, r in f(cfg)]),
    "another layer's table": ("side_slice", lambda f: lambda ids, i, dim, w: f(ids, max(i - 1, 0), dim, w)),
    "gelu": ("gelu_tanh", lambda f: P.silu),
}


@pytest.mark.parametrize("mistake", sorted(MISTAKES))
def test_a_mistake_in_any_mechanism_would_show_in_the_logits(mistake, monkeypatch):
    """The cases' weights are such that a wrong mechanism, planted in the plain implementation, moves at least one row in
    twenty of the cases that have it by ten times what the float32 runs may differ by."""
    cases = {"unscaled frequencies": ("P", "Q"), "passes without rows": ("P", "Q", "W"),
             "first pass without its row": ("P", "Q", "W")}.get(mistake, ("P", "Q", "R", "W"))
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

def put(a):
    return torch.tensor(np.asarray(a), dtype=torch.int32, device=dev())


def _step(entries, ctx, slots):
    """The device arrays of a step whose entries bring ``entries[i]`` tokens after ``ctx[i]`` cached ones."""
    s = types.SimpleNamespace()
    s.req_slot = put(slots)
    s.token_req = put(np.repeat(np.arange(len(entries)), entries))
    s.positions = put(np.concatenate([np.arange(c, c + n) for n, c in zip(entries, ctx)]))
    s.cu_q = put(np.concatenate([[0], np.cumsum(entries)]))
    s.ctx_len = put(ctx)
    s.num_entries = len(entries)
    s.status = torch.zeros(1, dtype=torch.int32, device=dev())
    return s


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("W", [88, 90, 1, 320, 1536, 3584, 5000, 8192, 9000])
def test_output_norm_residual_sum_and_next_norm_in_one_pass(dtype, W):
    from lite_lang_b200 import ops
    from lite_lang_b200.parts.norm import OutputRMSNorm
    g = torch.Generator().manual_seed(W)
    for n in (1, 7, 400):
        res = torch.randn(n, W, generator=g) * 3
        y = torch.randn(n, W, generator=g).to(dtype)
        parts = torch.randn(3, n, W, generator=g)
        wa, wb, add = (torch.randn(W, generator=g) for _ in range(3))
        for form in ("y", "partial", "none"):
            for with_add in (False, True):
                delta = {"y": y, "partial": parts, "none": None}[form]
                x = res.double()
                if delta is not None:
                    d = delta.double() if form == "y" else delta.double().sum(0)
                    x = x + P.norm(d, wa.double(), 0.3)
                if with_add:
                    x = x + add.double()
                want = P.norm(x, wb.double(), 1e-5)
                args = (None if delta is None else delta.to(dev()), None if delta is None else wa.to(dev()), 0.3,
                        add.to(dev()) if with_add else None)
                r = res.to(dev())
                out = torch.full((n, W), float("nan"), dtype=dtype, device=dev())
                ops.sandwich_norm(out, r, *args, wb.to(dev()), 1e-5)
                assert rel_err(out.float().cpu().numpy(), want.numpy()) <= kernel_tol(dtype), (form, with_add)
                assert float((r.cpu().double() - x).abs().max()) <= 4e-6 * float(x.abs().max())
                r = res.to(dev())                            # the residual itself, rounded
                ops.sandwich_norm(out, r, *args, None, 0.0)
                assert torch.equal(out, r.to(dtype))
                assert float((r.cpu().double() - x).abs().max()) <= 4e-6 * float(x.abs().max())
                if n > 1:                                    # chosen rows, nothing written back
                    r = res.to(dev())
                    pick = put([n - 1, 0, 5, 5])
                    some = torch.empty(4, W, dtype=dtype, device=dev())
                    ops.sandwich_norm(some, r, *args, wb.to(dev()), 1e-5, pick)
                    assert rel_err(some.float().cpu().numpy(), want[[n - 1, 0, 5, 5]].numpy()) <= kernel_tol(dtype)
                    assert torch.equal(r.cpu(), res)
                if form == "y":                              # (what the parts hand to it)
                    from lite_lang_b200.parts.base import NormedOutput
                    r = res.to(dev())
                    copy = OutputRMSNorm.apply(r, NormedOutput(args[0], args[1], 0.3, args[3]), dtype)
                    assert copy.dtype == dtype and torch.equal(copy, r.to(dtype))


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("V,W,dim", [(50, 88, 8), (33, 90, 1), (200, 1536, 128), (17, 4099, 5), (9, 4096, 24)])
def test_embedding_norm_and_the_per_token_table(dtype, V, W, dim):
    from lite_lang_b200 import ops
    from lite_lang_b200.config.spec import PartSpec
    from lite_lang_b200.parts import build_part
    ops.configure_matmul_precision()
    g = torch.Generator().manual_seed(V)
    table, w = torch.randn(V, W, generator=g).to(dtype), torch.randn(W, generator=g)
    ids = torch.randint(0, V, (37,), generator=g, dtype=torch.int32)
    status = torch.zeros(1, dtype=torch.int32, device=dev())
    out = torch.full((37, W), float("nan"), device=dev())
    ops.embed_norm(out, table.to(dev()), ids.to(dev()), w.to(dev()), 1e-5, status)
    assert rel_err(out.cpu().numpy(), P.norm(table.double()[ids.long()], w.double(), 1e-5).numpy()) <= 2e-5
    part = build_part("feed_forward", PartSpec("token_side", {"hidden_size": W, "vocab_size": V, "dim": dim, "index": 2, "layers": 4}))
    t = {"gate": (torch.randn(dim, W, generator=g) * 1.5 / math.sqrt(W)), "proj": torch.randn(W, dim, generator=g),
         "table": torch.randn(V, 4 * dim, generator=g)}
    t = {k: v.to(torch.bfloat16) for k, v in t.items()}
    part.load(lambda n: t[n], dtype, dev())
    for n in (1, 37, 300):
        ids = torch.randint(0, V, (n,), generator=g, dtype=torch.int32)
        x = torch.randn(n, W, generator=g).to(dtype)
        step = types.SimpleNamespace(token_ids=ids.to(dev()), status=status)
        y = part.forward(x.to(dev()), step)
        y = (y.sum(0) if y.dim() == 3 else y).float().cpu()
        ww = {f"l2.side.{k}": v.double() for k, v in t.items()}
        e = P.side_slice(ids.long(), 2, dim, {"side.embed": t["table"].double()})
        want = (P.gelu_tanh(x.double() @ ww["l2.side.gate"].T) * e) @ ww["l2.side.proj"].T
        assert float((y.double() - want).abs().max()) <= (2e-5 if dtype == torch.float32 else 2e-2) * float(want.abs().max())
    assert int(status.item()) == 0
    ops.embed_norm(out[:1], table.to(dev()), put([V]), w.to(dev()), 1e-5, status)      # an id outside is reported, not read
    assert int(status.item()) == 1 and not out[0].any()


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("M,K,I", [(5, 128, 200), (3, 96, 40), (24, 256, 130), (40, 320, 256), (200, 88, 50), (300, 256, 512), (16, 90, 33)])
def test_gelu_gate_in_every_product(dtype, M, K, I):
    """Gates from far below zero to far above, in every kernel that makes the gated product."""
    from lite_lang_b200 import ops
    ops.configure_matmul_precision()
    g = torch.Generator().manual_seed(M + I)
    x = torch.randn(M, K, generator=g).to(dtype)
    w = (torch.randn(2 * I, K, generator=g) * (3.0 / math.sqrt(K))).to(dtype)
    got = ops.gated_linear(x.to(dev()), w.to(dev()), "gelu_tanh").float().cpu()
    want = P.gelu_tanh(x.double() @ w[:I].double().T) * (x.double() @ w[I:].double().T)
    assert rel_err(got.numpy(), want.numpy()) <= (2e-5 if dtype == torch.float32 else 2.5e-2)


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,K,d,vd,rot,interleaved,ps", [(4, 2, 32, 64, 32, True, 16), (6, 2, 12, 20, 8, True, 4),
                                                         (3, 3, 64, 128, 48, True, 32), (2, 1, 16, 24, 16, False, 4),
                                                         (9, 1, 8, 24, 0, True, 8), (1, 1, 128, 64, 64, True, 16)])
def test_heads_of_two_maps_are_normed_rotated_and_cached(dtype, H, K, d, vd, rot, interleaved, ps):
    """Bias, a norm a head and map with one weight, then the rotation; a key's two parts side by side in the cache; the
    queries beside zeros.  And the same norm for heads of one map."""
    from lite_lang_b200 import ops
    g = torch.Generator().manual_seed(H + d)
    pos = torch.tensor([0, 1, 2, 17, 511, 512, 1000, 1001, 40], dtype=torch.int32)
    n = len(pos)
    rotate = P.rotate_neighbours if interleaved else P.rotate_halves
    rc = {"dims": rot, "base": 700.0}
    freq = P.frequencies(rc).float().to(dev()) if rot else None
    qw, kw = 1 + 0.3 * torch.randn(d, generator=g), 1 + 0.3 * torch.randn(d, generator=g)
    for maps in (2, 1):
        width = maps * (H + K) * d + K * vd
        proj = torch.randn(n, (width + 7) // 8 * 8, generator=g).to(dtype)
        bias = torch.randn(width, generator=g)
        kc = torch.full((4, K, ps, maps * d), float("nan"), dtype=dtype, device=dev())
        vc = torch.full((4, K, ps, vd), float("nan"), dtype=dtype, device=dev())
        slots = np.random.default_rng(1).permutation(4 * ps)[:n]
        status = torch.zeros(1, dtype=torch.int32, device=dev())
        buf = proj.to(dev())
        paired = torch.full((n, H * 2 * 2 * d), float("nan"), dtype=dtype, device=dev()) if maps == 2 else None
        ops.qkv_norm_rotate_store(buf, bias.to(dev()), pos.to(dev()), freq, 1.0, interleaved, maps * H, maps * K, d, vd, "head",
                                  qw.to(dev()), kw.to(dev()), False, 1e-5, put(slots), kc, vc, ps, status, paired_q=paired)
        assert int(status.item()) == 0
        x = proj[:, :width].double() + bias.double()
        q = rotate(P.norm(x[:, :maps * H * d].view(n, maps * H, d), qw.double(), 1e-5), pos, rc)
        k = rotate(P.norm(x[:, maps * H * d:maps * (H + K) * d].view(n, maps * K, d), kw.double(), 1e-5), pos, rc)
        v = x[:, maps * (H + K) * d:].view(n, K, vd)
        tol = 2e-4 if dtype == torch.float32 else 1.6e-2          # (float32 angles of positions in the hundreds)
        page, place = slots // ps, slots % ps
        assert float((kc.cpu()[page, :, place].double() - k.reshape(n, K, maps * d)).abs().max()) <= tol * float(k.abs().max())
        assert float((vc.cpu()[page, :, place].double() - v).abs().max()) <= tol * float(v.abs().max())
        if maps == 1:
            got = buf[:, :H * d].float().cpu().view(n, H, d).double()
            assert float((got - q).abs().max()) <= tol * float(q.abs().max())
            continue
        got = paired.float().cpu().view(n, H, 2, 2, d).double()
        assert not got[:, :, 0, 1].any() and not got[:, :, 1, 0].any()
        want = q.view(n, H, 2, d)
        for m in (0, 1):
            assert float((got[:, :, m, m] - want[:, :, m]).abs().max()) <= tol * float(q.abs().max())


def _paged(dtype, seqs_k, seqs_v, ps, nkv, hd, vd, rng, live):
    """Keys/values of several requests scattered over a pool whose other slots hold NaN; pages that ``live(r, page)`` denies
    are not in the table, as when a window has given them back."""
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


def _two_map_case(dtype, H, K, d, vd, ps, size, lens, new, kernel):
    """Prompt portions and single tokens of several requests in one launch; pages no query sees are not there.  The last
    queries of every request are aimed (a large dot product with one key) by their first map at the keys on both sides of
    the window's edge (without a window at a key far back), by their second at the token itself."""
    from lite_lang_b200 import ops
    if kernel == "tc":
        keep = [r for r in range(len(lens)) if new[r] > 1]
        lens, new = [lens[r] for r in keep], [new[r] for r in keep]
    elif kernel == "shaped":
        order = sorted(range(len(lens)), key=lambda r: new[r] != 1)
        lens, new = [lens[r] for r in order], [new[r] for r in order]
    rng, g = np.random.default_rng(d), torch.Generator().manual_seed(d + H)
    R, group = len(lens), H // K
    ks = [torch.randn(n, K, 2, d, generator=g) for n in lens]
    ks = [k / k.norm(dim=-1, keepdim=True) * math.sqrt(d) for k in ks]
    vs = [torch.randn(n, K, vd, generator=g) for n in lens]
    qs = [torch.randn(c, H, 2, d, generator=g) for c in new]
    lam, diff, eps, scale = 0.37, 0.45, 1e-5, 0.9 / math.sqrt(d)

    def first(p):
        return 0 if size is None else max(0, p - size + 1)

    aimed = []
    for r in range(R):
        targets = [("far", lambda p: 1)] if size is None else [("in", first), ("out", lambda p: first(p) - 1)]
        for back, (which, where) in enumerate(targets):
            row, p = new[r] - 1 - back, lens[r] - 1 - back
            if row < 0 or not 0 <= where(p) <= p:
                continue
            for h in range(H):
                qs[r][row, h, 0] = 6.0 * ks[r][where(p), h // group, 0]
                qs[r][row, h, 1] = 6.0 * ks[r][p, h // group, 1]
            aimed.append((r, row, p, where(p), which))
    ks, vs, qs = ([t.to(dtype).float() for t in ts] for ts in (ks, vs, qs))
    kc, vc, bt = _paged(dtype, [k.reshape(len(k), K, 2 * d) for k in ks], vs, ps, K, 2 * d, vd, rng,
                        lambda r, page: page >= first(lens[r] - new[r]) // ps)
    step = _step(new, [n - c for n, c in zip(lens, new)], list(range(R)))
    n_tok = sum(new)
    q = torch.zeros(n_tok, H, 2, 2, d)
    q[:, :, 0, 0] = torch.cat(qs)[:, :, 0]
    q[:, :, 1, 1] = torch.cat(qs)[:, :, 1]
    q = q.reshape(n_tok, H * 4 * d).to(dtype).to(dev())
    gate = torch.randn(n_tok, H + 5, generator=g).to(dtype)
    gate_d = gate.to(dev())[:, 2:2 + H]
    pairs = ops.MapPairs(lam, 1.0 - diff, eps)
    out = torch.full((n_tok, H * vd), float("nan"), dtype=dtype, device=dev())
    mask = "causal" if size is None else "window"
    if kernel == "blocks":
        ops.attention_modulated(out, q, q.stride(0), gate_d, kc, vc, bt, step.token_req, step.req_slot, step.positions,
                                n_tok, 2 * H, K, 2 * d, vd, ps, mask, size, False, scale, None, None, step.status, pairs=pairs)
    elif kernel == "shaped":
        n_single = sum(1 for c in new if c == 1)
        tail = (2 * H, K, 2 * d, vd, ps, mask, size, False, scale, step.status)
        head = (out, q, q.stride(0), False, gate_d, None, kc, vc, bt)
        stages = (max(lens) + 63) // 64 + 1 if size is None else (size + 62) // 64 + 1
        for want_parts in (32, 2, 1):
            span = (stages + want_parts - 1) // want_parts
            ops.attn_shaped(*head, step.cu_q, step.ctx_len, step.req_slot, n_single, n_single * ((2 * group + 127) // 128),
                            *tail, nsplit=(stages + span - 1) // span, span=span, pairs=pairs)
        ops.attn_shaped(*head, step.cu_q[n_single:], step.ctx_len[n_single:], step.req_slot[n_single:], R - n_single,
                        ops.attn_shaped_blocks(new[n_single:], 2 * group), *tail, pairs=pairs)
    else:
        blocks = ops.attn_prefill_tc_blocks(new, 2 * group)
        for nsplit, length in ((4, 1), (1, 8)):
            ops.attn_prefill_tc(out, q, q.stride(0), kc, vc, bt, step.cu_q, step.ctx_len, step.req_slot, R, blocks, 2 * H, K,
                                2 * d, ps, size, scale, step.status, nsplit=nsplit, split_len=length, gate=gate_d, pairs=pairs)
    assert int(step.status.item()) == 0
    got, at = out.float().cpu(), 0
    for r in range(R):
        T, c = lens[r], new[r]
        full = torch.cat([torch.zeros(T - c, H, 2, d, dtype=P.F), qs[r].double()])
        a = [P.softmax_attention(full[:, :, m], ks[r][:, :, m].double(), vs[r].double(), scale, P.visible(T, size))[-c:] for m in (0, 1)]
        z = P.combine_maps(a[0], a[1], lam, diff, eps)
        o = (z * P.sigmoid(gate[at:at + c, 2:2 + H].double())[:, :, None]).reshape(c, H * vd)
        assert rel_err(got[at:at + c].numpy(), o.numpy()) <= kernel_tol(dtype), (kernel, size, r)
        for rr, row, p, j, which in aimed:
            if rr == r:                # the head reads the key it is aimed at exactly if the window shows it
                h = H - 1
                hit = P.combine_maps(vs[r][j, h // group].double(), vs[r][p, h // group].double(), lam, diff, eps)
                hit = hit * P.sigmoid(gate[at + row, 2 + h].double())
                near = float((got[at + row].view(H, vd)[h].double() - hit).abs().max()) < 0.15 * float(hit.abs().max())
                assert near == (which != "out"), (kernel, size, r, row, j, which)
        at += c
    return {w for *_, w in aimed}


LENS, NEW = [150, 61, 97, 300, 34, 700], [40, 1, 97, 1, 5, 1]


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,K,d,vd,ps", [(6, 2, 12, 20, 4), (9, 1, 16, 24, 8), (1, 1, 18, 20, 4), (4, 2, 32, 64, 16), (2, 1, 64, 128, 64)])
def test_two_maps_a_block_a_token(dtype, H, K, d, vd, ps):
    seen = set()
    for size in (23, 64, 9, 100, 1000, None):
        seen |= _two_map_case(dtype, H, K, d, vd, ps, size, LENS[:5], NEW[:5], "blocks")
    assert seen == {"in", "out", "far"}


@gpu
@pytest.mark.parametrize("H,K,d,vd,ps", [(4, 2, 32, 64, 16), (4, 4, 64, 128, 16), (2, 1, 64, 64, 64), (8, 4, 32, 128, 32), (7, 1, 64, 128, 16)])
def test_two_maps_on_tensor_cores_with_parts_joined(H, K, d, vd, ps):
    seen = set()
    for size in (44, 64, 77, 128, 130, 5, 1000, None):
        seen |= _two_map_case(torch.bfloat16, H, K, d, vd, ps, size, LENS, NEW, "shaped")
    assert seen == {"in", "out", "far"}


@gpu
@pytest.mark.parametrize("H,K,d,ps", [(4, 2, 32, 16), (4, 4, 64, 16), (2, 1, 64, 64), (6, 2, 32, 32), (7, 1, 64, 16), (12, 2, 64, 16)])
def test_two_maps_of_prompt_portions_in_tensor_memory(H, K, d, ps):
    seen = set()
    for size in (44, 64, 77, 128, 130, 5, 1000, None):
        seen |= _two_map_case(torch.bfloat16, H, K, d, 2 * d, ps, size, [150, 61, 97, 300, 34, 700], [40, 2, 97, 150, 5, 601], "tc")
    assert seen == {"in", "out", "far"}


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,dk,dv,rot", [(3, 10, 14, 6), (4, 32, 48, 32), (1, 4, 6, 4), (2, 128, 128, 128), (2, 200, 72, 64), (5, 16, 8, 0)])
def test_retention_in_portions_with_records_used_again(dtype, H, dk, dv, rot):
    """Rotation, decayed sums and the heads' norms and gates for four requests fed in portions of unequal sizes, through
    records that other requests held before, against the plain formulas on the whole sequences."""
    from lite_lang_b200 import ops
    g = torch.Generator().manual_seed(H + dk)
    lens, cuts = [37, 9, 64, 300], [[5, 1, 2, 20, 9], [1, 1, 1, 1, 5], [64], [2, 1, 290, 1, 6]]
    rc = {"dims": rot, "base": 300.0}
    freq = P.frequencies(rc).float().to(dev()) if rot else None
    decay = torch.linspace(0.6, 1.0, H) if H > 1 else torch.tensor([0.97])
    cq, cv = H * dk, H * dv
    width = (2 * cq + 2 * cv + 7) // 8 * 8
    proj = [torch.randn(n, width, generator=g).to(dtype) for n in lens]
    state = torch.full((6, H * dv * dk), 7.0, device=dev())              # what another request left
    slots = [2, 0, 5, 3]
    for s in slots:
        state[s].zero_()                                                # a slot is zeroed when opened
    pad8 = lambda n: (n + 7) // 8 * 8
    row = (0, pad8(cq), 2 * pad8(cq))
    got, at = [[] for _ in lens], [0] * 4
    for k in range(max(len(c) for c in cuts)):
        who = [(r, at[r], cuts[r][k]) for r in range(4) if k < len(cuts[r])]
        step = _step([c for *_, c in who] + [1], [a for _, a, _ in who] + [0], [slots[r] for r, *_ in who] + [-1])   # (+ padding)
        x = torch.cat([proj[r][a:a + c] for r, a, c in who] + [torch.zeros(1, width, dtype=dtype)]).to(dev())
        rows = torch.full((x.shape[0], row[2] + pad8(cv)), float("nan"), device=dev())
        ops.rotate_rows_f32(rows, row, x, (0, cq, 2 * cq), step.positions, freq, False, H, dk, cv, 1.0, dk ** -0.5)
        o = torch.full((x.shape[0], cv), float("nan"), device=dev())
        ops.decay_scan(rows, *row, decay.to(dev()), state, step, o, H, dk, dv)
        y = torch.full((x.shape[0], cv), float("nan"), dtype=dtype, device=dev())
        ops.head_norm_gate_out(y, o, x[:, 2 * cq + cv:2 * cq + 2 * cv], 1e-5, H, dv, "silu")
        assert int(step.status.item()) == 0
        y = y.float().cpu()
        for r, _, c in who:
            got[r].append(y[:c])
            y = y[c:]
            at[r] += c
    for r, n in enumerate(lens):
        x, pos = proj[r].double(), torch.arange(n)
        q = P.rotate_halves(x[:, :cq].view(n, H, dk), pos, rc)
        k = P.rotate_halves(x[:, cq:2 * cq].view(n, H, dk), pos, rc) * dk ** -0.5
        o = P.unit_rms(P.decayed_sums(q, k, x[:, 2 * cq:2 * cq + cv].view(n, H, dv), decay.double()), 1e-5)
        want = o.reshape(n, cv) * P.silu(x[:, 2 * cq + cv:2 * cq + 2 * cv])
        assert rel_err(torch.cat(got[r]).numpy(), want.numpy()) <= (1e-4 if dtype == torch.float32 else 1.6e-2), r
    assert float(state[1].min()) == 7.0 and float(state[4].max()) == 7.0                  # nobody's records are untouched


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_rotation_of_rows_in_both_layouts(dtype):
    from lite_lang_b200 import ops
    g = torch.Generator().manual_seed(3)
    pos = torch.tensor([0, 1, 2, 77, 1000], dtype=torch.int32)
    for H, dk, rot in ((2, 16, 16), (3, 10, 4), (1, 64, 32)):
        for interleaved in (True, False):
            x = torch.randn(5, 3 * H * dk, generator=g).to(dtype)
            rows = torch.full((5, 3 * H * dk), float("nan"), device=dev())
            offs = (0, H * dk, 2 * H * dk)
            rc = {"dims": rot, "base": 40.0}
            ops.rotate_rows_f32(rows, offs, x.to(dev()), offs, pos.to(dev()), P.frequencies(rc).float().to(dev()), interleaved,
                                H, dk, H * dk, 2.0, 0.5)
            turn = P.rotate_neighbours if interleaved else P.rotate_halves
            xd = x.double().view(5, 3, H, dk)
            want = torch.stack([2.0 * turn(xd[:, 0], pos, rc), 0.5 * turn(xd[:, 1], pos, rc), xd[:, 2]], dim=1).reshape(5, -1)
            assert float((rows.cpu().double() - want).abs().max()) <= 3e-4 * float(want.abs().max())


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,d,dv,R,qr", [(3, 20, 12, 37, 19), (5, 48, 64, 64, 48), (6, 24, 16, 96, 40), (1, 8, 8, 100, 8)])
def test_latent_attention_without_a_rotated_part_finds_a_far_key(dtype, H, d, dv, R, qr):
    """The whole mixer with nothing but the latent cached: prompts in portions (through the products and the walking
    kernel), single tokens alone and split, a query aimed at a token far back across page and tile borders."""
    from lite_lang_b200 import ops
    from lite_lang_b200.cache.storage import PagedKVView
    from lite_lang_b200.config.spec import PartSpec
    from lite_lang_b200.engine.batch import StepEntry
    from lite_lang_b200.parts import build_part
    ops.configure_matmul_precision()
    hidden, ps, T = 64, 4, 150
    g = torch.Generator().manual_seed(R)
    part = build_part("mixer", PartSpec("latent_attention", {
        "hidden_size": hidden, "heads": H, "dim": d, "rot_dim": 0, "vdim": dv, "kv_rank": R, "q_rank": qr, "scale": 0.5 / math.sqrt(d),
        "eps": 1e-5}))
    t = {n: torch.randn(decl.shape, generator=g) * (0.1 if len(decl.shape) == 1 else decl.shape[1] ** -0.5) + (1.0 if len(decl.shape) == 1 else 0.0)
         for n, decl in part.tensors().items()}
    assert set(t) == {"dq", "dq.norm", "uq", "dkv", "dkv.norm", "uk", "uv", "o"}
    t = {n: v.to(torch.bfloat16) for n, v in t.items()}
    w = {n: v.double() for n, v in t.items()}
    x = torch.randn(T, hidden, generator=g)
    # the last token's query of head 0 is aimed at token 5: its input is moved until that key's score stands out
    c = P.norm(x.double() @ w["dkv"].T, w["dkv.norm"], 1e-5)
    far = (c @ w["uk"].T).view(T, H, d)[5, 0]
    aim = torch.linalg.lstsq((w["uq"] @ (w["dq.norm"][:, None] * w["dq"]))[:d], far[:, None]).solution[:, 0]
    x[T - 1] = (aim / aim.norm() * math.sqrt(hidden)).float()
    x = x.to(dtype)
    part.load(lambda n: t[n], dtype, dev())
    m = {"heads": H, "dim": d, "vdim": dv, "scale": 0.5 / math.sqrt(d)}
    want = P.mixer_latent_attention(x.double(), None, m, w, "", 1e-5)
    pages = (T + ps - 1) // ps
    perm = np.random.default_rng(2).permutation(pages + 2)[:pages]
    table = torch.full((2, pages), -1, dtype=torch.int32)
    table[1] = torch.tensor(perm.astype(np.int32))
    for cuts in ([T - 1, 1], [50, 2, 31, 64, 1, 1, 1], [1] * 40 + [T - 40]):
        cache = torch.full((pages + 2, 1, ps, R), float("nan"), dtype=dtype, device=dev())
        got, at = [], 0
        for n in cuts:
            step = _step([n], [at], [1])
            step.entries, step.entry_ctx, step.max_kv_len = [StepEntry(1, [0] * n)], [at], at + n
            p = np.arange(at, at + n)
            view = PagedKVView(cache, None, table.to(dev()), put(perm[p // ps] * ps + p % ps), ps, True, 0, 0)
            y = part.forward(x[at:at + n].to(dev()), step, view)
            got.append((y.sum(0) if y.dim() == 3 else y).float().cpu())
            at += n
            assert int(step.status.item()) == 0
        assert at == T
        assert rel_err(torch.cat(got).numpy(), want.numpy()) <= (1e-4 if dtype == torch.float32 else 3e-2), cuts[0]


# ---------------------------------------------------------------------------------------------------------
# GPU: the whole model through the runner, the cache manager, the replay tool and the scheduler
# ---------------------------------------------------------------------------------------------------------
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
    for name in ("P", "Q", "R", "W"):
        folder, seqs, _ = _case(name)
        cfg, w = P.read_model_folder(folder)
        layers = []
        P.forward(cfg, w, seqs[4], layers)
        mgr, runner = _runner(folder, torch.float32, CASES[name]["page_size"], 64, graphs=False)
        seen = []
        for block in runner.model.blocks:
            def wrapped(h, delta, step, caches, _f=block.forward):
                h, delta = _f(h, delta, step, caches)
                seen.append((h + delta.gain()).cpu())
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
        assert close(_feed(runner, mgr, s, seqs[i]), refs[i], dtype), f"{name} whole {i}"
        mgr.close(s)
    for i, tail in ((0, 120), (2, 40)):                     # a prompt, then many tokens one by one (captured steps):
        s, n = mgr.open(), len(seqs[i])                     # every window passes over decoded tokens
        head = n - tail
        got = [_feed(runner, mgr, s, seqs[i][:head])] + [_feed(runner, mgr, s, seqs[i][t:t + 1]) for t in range(head, n)]
        assert close(np.concatenate(got), refs[i], dtype), f"{name} decode {i}"
        mgr.close(s)
    s, n = mgr.open(), len(seqs[1])                         # from the very first token on, one by one
    got = [_feed(runner, mgr, s, seqs[1][t:t + 1]) for t in range(n)]
    assert close(np.concatenate(got), refs[1], dtype), f"{name} token by token"
    mgr.close(s)
    sizes = [7, 2, 13, 2, 5, 31, 2, 3, 17, 2, 64, 2, 9]
    for i in (0, 5):                                        # portions of changing size, down to two tokens
        s, n, t, k, got = mgr.open(), len(seqs[i]), 0, 0, []
        while t < n:
            c = min(sizes[k % len(sizes)], n - t)
            got.append(_feed(runner, mgr, s, seqs[i][t:t + c]))
            t, k = t + c, k + 1
        assert close(np.concatenate(got), refs[i], dtype), f"{name} portions {i}"
        mgr.close(s)
    runner.check_status()
    assert runner.graph_replays > 0


@gpu
def test_a_pool_smaller_than_the_prompt_serves_it_through_the_pages_given_back():
    """Every layer of this case has a window or a state, so a request holds a bounded number of pages however long it grows:
    a prompt of several times the pool, fed in portions and then decoded, and the logits are the whole prompt's."""
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
    for t in range(0, 264, portion):
        got.append(_feed(runner, mgr, s, toks[t:t + portion]))
    got += [_feed(runner, mgr, s, toks[t:t + 1]) for t in range(264, 400)]
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
    waiting, live, all_got, all_ref = list(enumerate(order)), {}, [], []
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
            live[k][1] = t + c
            if t + c == n:
                done.append(k)
        if not entries:
            continue
        all_got.append(runner.step(entries).float().cpu().numpy().copy())
        all_ref.append(np.concatenate(expect))
        for k in done:
            mgr.close(live.pop(k)[2])
        mgr.check_invariants()
    runner.check_status()
    assert close(np.concatenate(all_got), np.concatenate(all_ref), dtype), name
    assert mgr.pages_reused > 0


@gpu
def test_a_batch_gives_each_request_what_it_gets_alone():
    """What is left between a request alone and the same request beside others, in other pages and slots and cut otherwise,
    is the rounding of the matrix products, whose shapes differ (float32, where nothing else rounds)."""
    from lite_lang_b200.engine.batch import StepEntry
    folder, seqs, refs = _case("P")
    mgr, runner = _runner(folder, torch.float32, CASES["P"]["page_size"], 200, graphs=False)
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
    ref = P.forward(cfg, w, toks).numpy()
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
        assert close(np.concatenate([a, b[:59], c, b[59:]]), want, dtype)


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
@pytest.mark.parametrize("name", ["P", "R", "W"])
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
