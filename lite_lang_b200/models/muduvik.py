"""Muduvik: a decoder over a float32 residual with a norm before and behind every sublayer, three kinds of mixer, a per-token
table that enters every layer and a range of layers that runs several times.

config.json (``"architecture": "Muduvik"``) gives ``vocab``, ``width``, ``norm.eps``, ``token_side.dim``, ``loop`` (``start``,
``stop``, ``times``; may be missing: nothing runs again) and ``layers``: a list whose entries name the layer's mixer
(``type``), the mixer's sizes and constants (``mixer``) and its feed-forward (``mlp``, or null for none).  Every size and
constant is read from there; nothing is fixed by this file but what the design itself fixes.

The residual starts as an RMS norm of the token's embedding.  A layer is h += s1 N1b(mixer(N1(h))); h += s2 N2b(ff(N2(h)));
h += N3(P (gelu(G h) * e)) with RMS norms N, a layer scale s a channel and e the layer's part of the token's row of
``side.embed``.  Every pass of the looped range begins with its row of ``loop.step`` added to h.  The output is the final
norm and a head of its own.

Mixers, by ``type``:
  ``attention``         two score maps a head over the same values (``diff``; ``heads``, ``kv_heads``, ``dim`` a map, ``vdim``,
                        ``scale``): biases on q, k, v, an RMS norm a head and map before the rotation, neighbouring rotary
                        pairs with ``rot.base`` and wavelength scaling (``rot.scaling``: ``factor``, ``low``, ``high``,
                        ``original``), a sliding window of ``mask.size``, a sigmoid gate a head on the output (``g``)
  ``latent_attention``  keys and values expanded from one cached latent (``kv_rank``) a token, without positions; the queries
                        go through a latent of their own (``q_rank``); causal
  ``retention``         linear attention with a decay a head (``decay``), half-split rotary pairs, every head's output
                        divided by its root mean square and a SiLU gate a channel (``g``)
Feed-forward, by ``mlp.kind``: ``dense``: down(gelu(gate x) * (up x)) of width ``ff``, gelu in its tanh form.

Tensor names: ``embed``, ``embed.norm``, ``loop.step``, ``side.embed``, ``l<i>.norm1|norm1b|norm2|norm2b``, ``l<i>.ls1|ls2``,
``l<i>.mix.*``, ``l<i>.mlp.*``, ``l<i>.side.gate|proj|norm``, ``final.norm``, ``head``.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, List, Mapping, Optional, Tuple

from ..config.base import ConfigError, ModelConfig, _require, register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec, RunStep

LAYER_TYPES = ("attention", "latent_attention", "retention")
# positions are float32 inside the rotation: every position below 2^24 is exact
MAX_POSITIONS = 1 << 24


def _sub(d: Mapping[str, Any], key: str, where: str) -> Mapping[str, Any]:
    v = d.get(key)
    if not isinstance(v, Mapping):
        raise ConfigError(f"Muduvik: {where} lacks the section {key!r}")
    return v


def _positive(d: Mapping[str, Any], keys, where: str) -> None:
    for key in keys:
        if int(_require(d, key, int, f"Muduvik {where}")) <= 0:
            raise ConfigError(f"Muduvik: {where}: {key} must be positive")


def _mask_size(m: Mapping[str, Any]) -> Optional[int]:
    mask = m.get("mask") or {}
    return None if mask.get("size") is None else int(mask["size"])


def _check_rotation(m: Mapping[str, Any], where: str) -> None:
    rot = m.get("rot")
    if rot is None:
        return
    _require(rot, "base", float, f"Muduvik {where} rot")
    dims = int(_require(rot, "dims", int, f"Muduvik {where} rot"))
    if dims > int(m["dim"]) or dims % 2 or dims < 0:
        raise ConfigError(f"Muduvik: {where}: rot.dims must be even and at most dim")
    if rot.get("scaling"):
        for key in ("factor", "low", "high", "original"):
            _require(rot["scaling"], key, float, f"Muduvik {where} rot.scaling")


def _rotation(m: Mapping[str, Any], layout: str) -> Optional[PartSpec]:
    rot = m.get("rot")
    if rot is None or int(rot["dims"]) == 0:
        return None
    return PartSpec("rope_computed", {"rotary_dim": int(rot["dims"]), "theta": float(rot["base"]), "layout": layout,
                                      "scaling": None if not rot.get("scaling") else dict(rot["scaling"])})


@dataclass(frozen=True)
class MuduvikConfig(ModelConfig):
    vocab: int
    width: int
    norm_eps: float
    side_dim: int
    layers: Tuple[Mapping[str, Any], ...]                  # as in config.json (validated)
    loop: Optional[Tuple[int, int, int]] = None            # layers start .. stop - 1 run so many times in a row
    eos_token_id: Tuple[int, ...] = ()
    initializer_range: float = 0.05

    architecture = "Muduvik"

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "MuduvikConfig":
        a = cls.architecture
        layers = d.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError(f"{a}: config.json lacks the list 'layers'")
        eos = d.get("eos_token_id")
        eos_ids = () if eos is None else tuple(int(e) for e in (eos if isinstance(eos, (list, tuple)) else [eos]))
        loop = None
        if d.get("loop") is not None:
            sec = _sub(d, "loop", "config.json")
            loop = tuple(int(_require(sec, k, int, f"{a} loop")) for k in ("start", "stop", "times"))
        cfg = cls(vocab=_require(d, "vocab", int, a), width=_require(d, "width", int, a),
                  norm_eps=float(_require(_sub(d, "norm", "config.json"), "eps", float, f"{a} norm")),
                  side_dim=int(_require(_sub(d, "token_side", "config.json"), "dim", int, f"{a} token_side")),
                  layers=tuple(copy.deepcopy(dict(l)) for l in layers), loop=loop, eos_token_id=eos_ids,
                  initializer_range=float(d.get("initializer_range", 0.05)))
        cfg.validate()
        return cfg

    def validate(self) -> None:
        a = self.architecture
        if self.vocab <= 0 or self.width <= 0 or self.norm_eps <= 0 or self.side_dim <= 0:
            raise ConfigError(f"{a}: vocab, width, norm.eps and token_side.dim must be positive")
        if self.loop is not None:
            start, stop, times = self.loop
            if not (0 <= start < stop <= len(self.layers)) or times < 1:
                raise ConfigError(f"{a}: loop must lie within the layers (start {start}, stop {stop}) and run at least once")
        for i, layer in enumerate(self.layers):
            where = f"layer {i}"
            kind = layer.get("type")
            if kind not in LAYER_TYPES:
                raise ConfigError(f"{a}: {where} has the type {kind!r}; built: {', '.join(LAYER_TYPES)}")
            m = _sub(layer, "mixer", where)
            if kind == "attention":
                _positive(m, ("heads", "kv_heads", "dim", "vdim"), where)
                _require(m, "scale", float, f"{a} {where}")
                _require(m, "diff", float, f"{a} {where}")
                if int(m["heads"]) % int(m["kv_heads"]):
                    raise ConfigError(f"{a}: {where}: heads is not a multiple of kv_heads")
                size = _mask_size(m)
                if size is not None and size <= 0:
                    raise ConfigError(f"{a}: {where}: mask.size must be positive")
                _check_rotation(m, where)
            elif kind == "latent_attention":
                _positive(m, ("heads", "dim", "vdim", "kv_rank", "q_rank"), where)
                _require(m, "scale", float, f"{a} {where}")
            else:
                _positive(m, ("heads", "dim", "vdim"), where)
                decay = m.get("decay")
                if not isinstance(decay, (list, tuple)) or len(decay) != int(m["heads"]):
                    raise ConfigError(f"{a}: {where}: decay must give one number a head")
                _check_rotation(m, where)
            mlp = layer.get("mlp")
            if mlp is not None:
                if mlp.get("kind") != "dense":
                    raise ConfigError(f"{a}: {where} has a feed-forward of kind {mlp.get('kind')!r}; built: 'dense'")
                _positive(mlp, ("ff",), f"{where} mlp")

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {
            "architecture": self.architecture,
            "layers": [copy.deepcopy(dict(l)) for l in self.layers],
            "norm": {"eps": self.norm_eps},
            "token_side": {"dim": self.side_dim},
            "vocab": self.vocab,
            "width": self.width,
            # (read by this package's own tools: the tests' trace helper and the random-weights writer)
            "vocab_size": self.vocab,
            "initializer_range": self.initializer_range,
        }
        if self.loop is not None:
            d["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        if self.eos_token_id:
            d["eos_token_id"] = list(self.eos_token_id)
        return d

    def init_scales(self) -> Dict[str, float]:
        s = self.initializer_range
        return {"matrix": s, "bias": s, "norm": s}

    # ------------------------------------------------------------------
    def _mixer_spec(self, i: int, layer: Mapping[str, Any]) -> PartSpec:
        m, kind, prefix = layer["mixer"], layer["type"], f"l{i}.mix."
        if kind == "attention":
            size = _mask_size(m)
            return PartSpec("modulated_attention", {
                "hidden_size": self.width, "num_heads": int(m["heads"]), "num_kv_heads": int(m["kv_heads"]),
                "head_dim": int(m["dim"]), "value_head_dim": int(m["vdim"]), "scale": float(m["scale"]),
                "eps": self.norm_eps, "qkv_bias": True, "qk_norm": "head", "differential": {"diff": float(m["diff"])},
                "position": _rotation(m, "interleaved"), "mask": "causal" if size is None else "window", "mask_size": size,
                "head_gate": True}, prefix)
        if kind == "latent_attention":
            return PartSpec("latent_attention", {
                "hidden_size": self.width, "heads": int(m["heads"]), "dim": int(m["dim"]), "rot_dim": 0,
                "vdim": int(m["vdim"]), "kv_rank": int(m["kv_rank"]), "q_rank": int(m["q_rank"]), "window": None,
                "scale": float(m["scale"]), "eps": self.norm_eps}, prefix)
        return PartSpec("retention", {
            "hidden_size": self.width, "heads": int(m["heads"]), "key_dim": int(m["dim"]), "value_dim": int(m["vdim"]),
            "decay": [float(x) for x in m["decay"]], "key_scale": float(m["dim"]) ** -0.5, "eps": self.norm_eps,
            "position": _rotation(m, "half_split")}, prefix)

    def run_order(self) -> Tuple[RunStep, ...]:
        if self.loop is None:
            return tuple(RunStep(i) for i in range(len(self.layers)))
        start, stop, times = self.loop
        order: List[RunStep] = [RunStep(i) for i in range(start)]
        for t in range(times):
            order += [RunStep(i, add_row=t if i == start else None) for i in range(start, stop)]
        return tuple(order + [RunStep(i) for i in range(stop, len(self.layers))])

    def model_spec(self) -> ModelSpec:
        base = {"hidden_size": self.width, "eps": self.norm_eps}
        layers: List[LayerSpec] = []
        for i, layer in enumerate(self.layers):
            p = f"l{i}."

            def norm(name):
                return PartSpec("rms_norm_f32_sandwich", {**base, "tensor": ""}, p + name)

            def out_norm(name, scale=None):
                return PartSpec("rms_norm_out", {**base, "tensor": name, "scale_tensor": scale}, p)

            parts = {"mixer_norm": norm("norm1"), "mixer": self._mixer_spec(i, layer), "mixer_out_norm": out_norm("norm1b", "ls1"),
                     "token_side": PartSpec("token_side", {
                         "hidden_size": self.width, "vocab_size": self.vocab, "dim": self.side_dim, "index": i,
                         "layers": len(self.layers),
                         "tensor_names": {"gate": p + "side.gate", "proj": p + "side.proj", "table": "side.embed"}}),
                     "token_side_out_norm": out_norm("side.norm")}
            if layer.get("mlp") is None:
                layers.append(LayerSpec("sandwich_token_side_mixer_only", parts))
                continue
            parts["feed_forward_norm"] = norm("norm2")
            parts["feed_forward"] = PartSpec("gated_mlp", {
                "hidden_size": self.width, "intermediate_size": int(layer["mlp"]["ff"]), "activation": "gelu_tanh",
                "tensor_names": ("gate", "up", "down")}, p + "mlp.")
            parts["feed_forward_out_norm"] = out_norm("norm2b", "ls2")
            layers.append(LayerSpec("sandwich_token_side", parts))
        return ModelSpec(
            architecture=self.architecture, hidden_size=self.width, vocab_size=self.vocab, max_positions=MAX_POSITIONS,
            embedding=PartSpec("token_embedding", {
                "vocab_size": self.vocab, "hidden_size": self.width, "residual": "float32", "tensor": "embed",
                "norm": {"tensor": "embed.norm", "eps": self.norm_eps}}),
            layers=tuple(layers), order=self.run_order(),
            final_norm=PartSpec("rms_norm_f32_sandwich", {**base, "tensor": ""}, "final.norm"),
            head=PartSpec("lm_head", {"vocab_size": self.vocab, "hidden_size": self.width, "tensor": ""}, "head"),
            eos_token_ids=self.eos_token_id,
            pass_rows=None if self.loop is None else PartSpec("pass_rows", {
                "rows": self.loop[2], "hidden_size": self.width, "tensor": ""}, "loop.step"))


register_architecture(MuduvikConfig.architecture, MuduvikConfig)
