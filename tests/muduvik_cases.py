"""Small Muduvik configurations for the tests, and a helper that writes them as model folders."""

from __future__ import annotations

import json
import os
import tempfile
from typing import Optional


def _rot(base, dims, scaling=None):
    rot = {"base": base, "dims": dims}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return rot


def _attention(heads, kv_heads, dim, vdim, scale, diff, rot, size=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff, "rot": rot}
    if size is not None:
        m["mask"] = {"size": size}
    return m


def _latent(heads, dim, vdim, kv_rank, q_rank, scale):
    return {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale}


def _retention(heads, dim, vdim, rot, decay):
    return {"heads": heads, "dim": dim, "vdim": vdim, "rot": rot, "decay": decay}


def _layer(kind, mixer, ff=None):
    return {"type": kind, "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


CASES = {
    # odd sizes: no width or head size a power of two or a multiple of 8, values wider and narrower than keys, rotation on a
    # part of the channels, a window that is no multiple of the page, a table of 11 numbers a layer; a range in the middle
    # that runs three times (with a layer without a feed-forward and a recurrent one inside it)
    "P": {
        "config": {"architecture": "Muduvik", "vocab": 211, "width": 88, "norm": {"eps": 3e-6}, "token_side": {"dim": 11},
                   "loop": {"start": 1, "stop": 3, "times": 3},
                   "layers": [
                       _layer("attention", _attention(6, 2, 12, 36, 0.35, 0.35, _rot(900.0, 8, (4.0, 1.0, 4.0, 64)), 23), 50),
                       _layer("retention", _retention(3, 10, 30, _rot(500.0, 6), [0.75, 0.96875, 0.9921875]), 36),
                       _layer("attention", _attention(4, 4, 20, 28, 0.25, 0.4, _rot(10000.0, 20), 9)),
                       _layer("latent_attention", _latent(3, 20, 12, 37, 19, 0.35), 44),
                       _layer("retention", _retention(2, 18, 22, _rot(77.0, 2), [0.75, 0.984375])),
                   ]},
        "seed": 5, "page_size": 4},
    # two maps of 32 and 64 beside values as wide as both maps together (all tensor-core kernels in bfloat16) and not, pages
    # of 16, windows beside the kernels' key tiles, an attention without a window, a range from the first layer on
    "Q": {
        "config": {"architecture": "Muduvik", "vocab": 300, "width": 128, "norm": {"eps": 2e-5}, "token_side": {"dim": 24},
                   "loop": {"start": 0, "stop": 2, "times": 2},
                   "layers": [
                       _layer("attention", _attention(4, 2, 32, 64, 0.3, 0.5, _rot(5000.0, 32, (8.0, 1.0, 4.0, 256)), 44), 96),
                       _layer("retention", _retention(4, 32, 48, _rot(10000.0, 32), [0.875, 0.9375, 0.984375, 0.99609375])),
                       _layer("attention", _attention(2, 1, 64, 128, 0.2, 0.2, _rot(10000.0, 64), 77), 160),
                       _layer("latent_attention", _latent(5, 48, 64, 64, 48, 0.3), 128),
                       _layer("attention", _attention(6, 2, 64, 64, 0.2, 0.8, _rot(300.0, 48))),
                       _layer("attention", _attention(3, 3, 32, 128, 0.3, 0.4, _rot(300.0, 16), 128), 72),
                   ]},
        "seed": 6, "page_size": 16},
    # values that other models make equal or 1: a width that is no multiple of 4, no loop
    # section, one head, nine heads on one key head, no second-map constant, no rotation, a window longer than any request,
    # a head that never forgets, a latent wider than the model
    "R": {
        "config": {"architecture": "Muduvik", "vocab": 97, "width": 90, "norm": {"eps": 1e-6}, "token_side": {"dim": 7},
                   "layers": [
                       _layer("attention", _attention(9, 1, 8, 28, 0.4, 0.0, _rot(100.0, 4, (2.0, 1.0, 8.0, 32)), 1000), 33),
                       _layer("latent_attention", _latent(1, 12, 20, 100, 14, 0.4)),
                       _layer("retention", _retention(1, 20, 26, _rot(50.0, 4), [1.0]), 20),
                       _layer("attention", _attention(1, 1, 4, 30, 0.9, 0.6, _rot(100.0, 0), 1), 28),
                       _layer("latent_attention", _latent(4, 12, 20, 24, 30, 0.35), 33),
                   ]},
        "seed": 7, "page_size": 8},
    # every layer forgets or is of fixed size, so a request holds a bounded number of pages however long it grows; a loop over
    # all layers
    "W": {
        "config": {"architecture": "Muduvik", "vocab": 120, "width": 64, "norm": {"eps": 1e-5}, "token_side": {"dim": 8},
                   "loop": {"start": 0, "stop": 2, "times": 2},
                   "layers": [
                       _layer("attention", _attention(4, 2, 16, 24, 0.4, 0.3, _rot(1000.0, 16), 20), 40),
                       _layer("retention", _retention(2, 16, 24, _rot(1000.0, 16), [0.9375, 0.99])),
                   ]},
        "seed": 8, "page_size": 4},
}


def write_folder(name: str, folder: Optional[str] = None) -> str:
    """Write the case as a model folder with random weights.  The latents' expansions, the vectors that weigh the second map
    and the passes' rows are multiplied up afterwards, so that a wrong key, map or pass shows in the logits.  The keys that
    only this package's own tools read are taken out of config.json."""
    from safetensors.torch import load_file, save_file

    from lite_lang_b200.config import config_from_dict
    from lite_lang_b200.weights import write_random_model

    case = CASES[name]
    cfg = config_from_dict(case["config"])
    folder = folder or tempfile.mkdtemp(prefix=f"ll_muduvik_{name}_")
    write_random_model(folder, cfg, case["seed"], {"matrix": 0.12, "bias": 0.15, "norm": 0.2})
    path = os.path.join(folder, "model.safetensors")
    t = load_file(path)
    up = {"uq": 1.6, "uk": 1.6, "lq1": 2.5, "lk1": 2.5, "lq2": 2.5, "lk2": 2.5, "step": 5.0, "gate": 1.5}
    for k in list(t):
        f = up.get(k.rsplit(".", 1)[-1])
        if f is not None:
            t[k] = (t[k].float() * f).to(t[k].dtype)
        elif k == "side.embed":
            t[k] = (t[k].float() * 8.0).to(t[k].dtype)
    save_file(t, path, metadata={"format": "pt"})
    path = os.path.join(folder, "config.json")
    d = json.load(open(path))
    for k in ("vocab_size", "initializer_range"):
        d.pop(k, None)
    json.dump(d, open(path, "w"))
    return folder
