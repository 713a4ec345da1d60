"""Small Tusipel configurations for the tests, and a helper that writes them as model folders."""

from __future__ import annotations

import os
import tempfile
from typing import Optional


def _attention(heads, kv_heads, dim, vdim, scale, conv, size=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "conv": conv}
    if size is not None:
        m["mask"] = {"size": size}
    return m


def _latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, size, base, scaling=None, dims=None):
    rot = {"base": base, "dims": rot_dim if dims is None else dims}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
         "scale": scale, "rot": rot}
    if size is not None:
        m["mask"] = {"size": size}
    return m


def _moe(experts, identity, top, groups, scale, ff):
    r = {"experts": experts, "identity": identity, "top": top, "scale": scale}
    if groups is not None:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "router": r, "expert": {"ff": ff}}


def _dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


# what write_folder multiplies the query and key matrices by
QK_UP = 1.3

CASES = {
    # odd sizes: no width or head size a power of two, values wider and narrower than keys, windows and chunks that are
    # no multiple of the page and shorter than the kernels' key tiles, rotation on a part of the rotated channels, a range
    # in the middle that runs three times (a layer without a feed-forward and one with identities inside it)
    "P": {
        "config": {"architecture": "Tusipel", "vocab": 211, "width": 88, "norm": {"eps": 3e-6}, "canon": {"taps": 3},
                   "embedding": {"scale": 2.5}, "loop": {"start": 1, "stop": 3, "times": 3},
                   "layers": [
                       {"type": "attention", "mixer": _attention(6, 2, 24, 40, 0.5, 4, 23), "mlp": _dense(50, 0.7)},
                       {"type": "latent_attention",
                        "mixer": _latent(3, 20, 6, 12, 37, 19, 0.6, 17, 10000.0, (4.0, 64, 32.0, 1.0), dims=4),
                        "mlp": _moe(5, 3, 3, (4, 2), 1.5, 20)},
                       {"type": "attention", "mixer": _attention(1, 1, 36, 20, 0.4, 2, 9), "mlp": None},
                       {"type": "attention", "mixer": _attention(4, 4, 20, 28, 0.5, 3, 64), "mlp": _moe(6, 0, 2, (3, 2), 0.8, 28)},
                   ]},
        "seed": 5, "page_size": 4},
    # heads of 64 and 128 with values as wide as keys and not (the tensor-core kernels in bfloat16), pages of 16, chunks
    # longer than a key tile and no multiple of one, a loop over the first layers, two taps
    "Q": {
        "config": {"architecture": "Tusipel", "vocab": 300, "width": 128, "norm": {"eps": 2e-5}, "canon": {"taps": 2},
                   "embedding": {"scale": 11.0}, "loop": {"start": 0, "stop": 2, "times": 2},
                   "layers": [
                       {"type": "attention", "mixer": _attention(8, 2, 64, 64, 0.2, 3, 44), "mlp": _moe(8, 4, 4, (4, 3), 2.0, 64)},
                       {"type": "latent_attention", "mixer": _latent(2, 48, 16, 32, 64, 48, 0.25, 70, 30000.0),
                        "mlp": _dense(96, 1.3)},
                       {"type": "attention", "mixer": _attention(2, 1, 128, 128, 0.12, 4, 77), "mlp": _dense(128, 0.5)},
                       {"type": "attention", "mixer": _attention(4, 2, 128, 64, 0.12, 2, 128), "mlp": None},
                   ]},
        "seed": 6, "page_size": 16},
    # values that other models make equal or 1: a width that is no multiple of 4, one tap everywhere (nothing of earlier
    # tokens enters), nine query heads on one key head, an attention without a mask section, a window longer than any
    # request, an unscaled embedding and no loop, every output of a router chosen, one group, no scaled frequencies
    "R": {
        "config": {"architecture": "Tusipel", "vocab": 97, "width": 90, "norm": {"eps": 1e-6}, "canon": {"taps": 1},
                   "embedding": {"scale": 1.0},
                   "layers": [
                       {"type": "attention", "mixer": _attention(9, 1, 20, 28, 0.5, 1), "mlp": _moe(3, 0, 3, None, 1.0, 20)},
                       {"type": "latent_attention", "mixer": _latent(1, 8, 4, 8, 16, 8, 0.9, 1000, 77.0, (2.0, 16, 2.0, 1.0)),
                        "mlp": _moe(2, 1, 1, (3, 1), 1.0, 16)},
                       {"type": "latent_attention", "mixer": _latent(4, 12, 8, 20, 24, 30, 0.6, None, 500.0), "mlp": _dense(33, 50.0)},
                       {"type": "attention", "mixer": _attention(4, 2, 32, 32, 0.4, 5, 1000), "mlp": _moe(4, 4, 2, (2, 1), 3.0, 12)},
                   ]},
        "seed": 7, "page_size": 8},
    # every layer forgets, so a request holds a bounded number of pages however long it grows; six taps (more than the
    # kernels' unrolled forms) and a loop over all layers
    "W": {
        "config": {"architecture": "Tusipel", "vocab": 120, "width": 64, "norm": {"eps": 1e-5}, "canon": {"taps": 6},
                   "embedding": {"scale": 4.0}, "loop": {"start": 0, "stop": 2, "times": 2},
                   "layers": [
                       {"type": "attention", "mixer": _attention(4, 2, 16, 16, 0.7, 6, 20), "mlp": _dense(40, 1.0)},
                       {"type": "latent_attention", "mixer": _latent(4, 16, 8, 16, 32, 24, 0.6, 20, 1000.0),
                        "mlp": _moe(4, 2, 2, (3, 1), 1.2, 16)},
                   ]},
        "seed": 8, "page_size": 4},
}


def write_folder(name: str, folder: Optional[str] = None) -> str:
    """Write the case as a model folder with random weights.  The query and key matrices are multiplied up afterwards so
    that the attention is peaked on few keys (a wrong key, slope or mask shows in the logits).  The keys that only this
    package's own tools read are taken out of config.json."""
    import json

    from lite_lang_b200.config import config_from_dict
    from lite_lang_b200.weights import write_random_model

    case = CASES[name]
    cfg = config_from_dict(case["config"])
    folder = folder or tempfile.mkdtemp(prefix=f"ll_tusipel_{name}_")
    write_random_model(folder, cfg, case["seed"], {"matrix": 0.12, "bias": 0.1, "norm": 0.1})
    from safetensors.torch import load_file, save_file
    path = os.path.join(folder, "model.safetensors")
    t = load_file(path)
    for k in list(t):
        if k.rsplit(".", 1)[-1] in ("q", "k", "uq", "uk"):
            t[k] = (t[k].float() * QK_UP).to(t[k].dtype)
        elif k.endswith(".correction"):     # (choices further apart, so that fewer of them hang on a rounding)
            t[k] = (t[k].float() * 8.0).to(t[k].dtype)
        elif k == "embed":
            t[k] = (t[k].float() * 5.0).to(t[k].dtype)
    save_file(t, path, metadata={"format": "pt"})
    path = os.path.join(folder, "config.json")
    d = json.load(open(path))
    for k in ("vocab_size", "initializer_range"):
        d.pop(k, None)
    if "loop" not in case["config"]:
        d.pop("loop")
    json.dump(d, open(path, "w"))
    return folder
