"""Tusipel: a pre-norm decoder over a float32 residual with a short convolution behind every norm, two kinds of
attention, dense or routed feed-forwards and a range of layers that runs several times.

config.json (``"architecture": "Tusipel"``) gives ``vocab``, ``width``, ``embedding.scale``, ``norm.eps``,
``canon.taps``, ``loop`` (``start``, ``stop``, ``times``; may be missing: nothing runs again) and ``layers``: a list whose
entries name the layer's mixer (``type``), the mixer's sizes and constants (``mixer``) and its feed-forward (``mlp``, or
null for none).  Every size and constant is read from there; nothing is fixed by this file but what the design itself
fixes.

A layer is h += mixer(C1(N1(h))); h += feed_forward(C2(N2(h))) with N an RMS norm whose weight is stored around zero
and C(u) = u + a causal convolution of u over time (``canon.taps`` weights a channel).  The embedding's output is its row
times ``embedding.scale``; it is added to the residual again before every further pass of the looped range.  The output
is the final norm and a head of its own.

Mixers, by ``type``:
  ``latent_attention``  keys and values expanded from one cached latent (``kv_rank``) and one rotated key part
                        (``rot_dim``) a token; the queries go through a latent of their own (``q_rank``); half-split
                        rotary pairs with stretched slow frequencies (``rot``); a sliding window of ``mask.size``; a
                        sigmoid gate a channel on the heads' outputs (``g``)
  ``attention``         grouped-query attention without rotation (``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``): q,
                        k and v each pass a causal convolution (``conv`` taps), scores lose slope_h times the distance
                        (slopes 2^(-8 (h + 1) / heads)), a token sees its own chunk of ``mask.size`` positions
Feed-forward, by ``mlp.kind``: ``dense``: gated, down(a sigmoid(1.702 a) (c + 1)), a = min(gate x, ``limit``), c = clamp(up
x, -limit, limit), of width ``ff``; ``moe``: ``router.experts`` experts down(silu(gate x) * (up x)) of width ``expert.ff`` and
``router.identity`` that return their input; softmax scores over all of them, chosen by the scores plus a correction
within the best ``router.groups.keep`` of ``router.groups.count`` groups, ``router.top`` of them, weighted by their scores
times ``router.scale``.

Tensor names: ``embed``, ``l<i>.norm1|norm2``, ``l<i>.canon1|canon2``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, List, Mapping, Optional, Tuple

from ..config.base import ConfigError, ModelConfig, _require, register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec, RunStep
from ..parts.modulated_attention import geometric_slopes

LAYER_TYPES = ("attention", "latent_attention")
MLP_KINDS = ("dense", "moe")
SWISH_ALPHA = 1.702
SLOPE_EXPONENT = 8.0
# positions are float32 inside the rotation: every position below 2^24 is exact
MAX_POSITIONS = 1 << 24


def _sub(d: Mapping[str, Any], key: str, where: str) -> Mapping[str, Any]:
    v = d.get(key)
    if not isinstance(v, Mapping):
        raise ConfigError(f"Tusipel: {where} lacks the section {key!r}")
    return v


def _positive(d: Mapping[str, Any], keys, where: str) -> None:
    for key in keys:
        if int(_require(d, key, int, f"Tusipel {where}")) <= 0:
            raise ConfigError(f"Tusipel: {where}: {key} must be positive")


def _mask_size(m: Mapping[str, Any]) -> Optional[int]:
    mask = m.get("mask") or {}
    return None if mask.get("size") is None else int(mask["size"])


@dataclass(frozen=True)
class TusipelConfig(ModelConfig):
    vocab: int
    width: int
    embedding_scale: float
    norm_eps: float
    canon_taps: int
    layers: Tuple[Mapping[str, Any], ...]      # as in config.json (validated)
    loop: Tuple[int, int, int] = (0, 0, 1)     # layers start .. stop - 1 run so many times in a row
    eos_token_id: Tuple[int, ...] = ()
    initializer_range: float = 0.05

    architecture = "Tusipel"

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "TusipelConfig":
        a = cls.architecture
        layers = d.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError(f"{a}: config.json lacks the list 'layers'")
        eos = d.get("eos_token_id")
        eos_ids = () if eos is None else tuple(int(e) for e in (eos if isinstance(eos, (list, tuple)) else [eos]))
        loop = (0, 0, 1)
        if d.get("loop") is not None:
            sec = _sub(d, "loop", "config.json")
            loop = tuple(int(_require(sec, k, int, f"{a} loop")) for k in ("start", "stop", "times"))
        cfg = cls(vocab=_require(d, "vocab", int, a), width=_require(d, "width", int, a),
                  embedding_scale=float(_require(_sub(d, "embedding", "config.json"), "scale", float, f"{a} embedding")),
                  norm_eps=float(_require(_sub(d, "norm", "config.json"), "eps", float, f"{a} norm")),
                  canon_taps=int(_require(_sub(d, "canon", "config.json"), "taps", int, f"{a} canon")),
                  layers=tuple(copy.deepcopy(dict(l)) for l in layers), loop=loop, eos_token_id=eos_ids,
                  initializer_range=float(d.get("initializer_range", 0.05)))
        cfg.validate()
        return cfg

    def validate(self) -> None:
        a = self.architecture
        if self.vocab <= 0 or self.width <= 0 or self.norm_eps <= 0 or self.canon_taps <= 0:
            raise ConfigError(f"{a}: vocab, width, norm.eps and canon.taps must be positive")
        start, stop, times = self.loop
        if not (0 <= start <= stop <= len(self.layers)) or times < 1:
            raise ConfigError(f"{a}: loop must lie within the layers (start {start}, stop {stop}) and run at least once")
        for i, layer in enumerate(self.layers):
            where = f"layer {i}"
            kind = layer.get("type")
            if kind not in LAYER_TYPES:
                raise ConfigError(f"{a}: {where} has the type {kind!r}; built: {', '.join(LAYER_TYPES)}")
            m = _sub(layer, "mixer", where)
            _require(m, "scale", float, f"{a} {where}")
            size = _mask_size(m)
            if size is not None and size <= 0:
                raise ConfigError(f"{a}: {where}: mask.size must be positive")
            if kind == "attention":
                _positive(m, ("heads", "kv_heads", "dim", "vdim", "conv"), where)
                if int(m["heads"]) % int(m["kv_heads"]):
                    raise ConfigError(f"{a}: {where}: heads is not a multiple of kv_heads")
            else:
                _positive(m, ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank"), where)
                rot = _sub(m, "rot", where)
                _require(rot, "base", float, f"{a} {where} rot")
                dims = int(_require(rot, "dims", int, f"{a} {where} rot"))
                if dims > int(m["rot_dim"]) or dims % 2 or dims < 0:
                    raise ConfigError(f"{a}: {where}: rot.dims must be even and at most rot_dim")
                if rot.get("scaling"):
                    for key in ("factor", "original", "fast", "slow"):
                        _require(rot["scaling"], key, float, f"{a} {where} rot.scaling")
            mlp = layer.get("mlp")
            if mlp is None:
                continue
            if mlp.get("kind") == "dense":
                _positive(mlp, ("ff",), f"{where} mlp")
                if float(_require(mlp, "limit", float, f"{a} {where} mlp")) <= 0:
                    raise ConfigError(f"{a}: {where}: mlp.limit must be positive")
            elif mlp.get("kind") == "moe":
                r = _sub(mlp, "router", where)
                _positive(r, ("experts", "top"), f"{where} router")
                _require(r, "scale", float, f"{a} {where} router")
                _positive(_sub(mlp, "expert", where), ("ff",), f"{where} expert")
                outputs = int(r["experts"]) + int(r.get("identity") or 0)
                count, keep = self._groups(r)
                if count < 1 or outputs % count or not (1 <= keep <= count):
                    raise ConfigError(f"{a}: {where}: router.groups.count must divide experts + identity, keep be 1 to count")
                if int(r["top"]) > keep * (outputs // count):
                    raise ConfigError(f"{a}: {where}: router.top is more than the kept groups hold")
            else:
                raise ConfigError(f"{a}: {where} has a feed-forward of kind {mlp.get('kind')!r}; "
                                  f"built: {', '.join(MLP_KINDS)}")

    @staticmethod
    def _groups(router: Mapping[str, Any]) -> Tuple[int, int]:
        g = router.get("groups")
        return (1, 1) if not g else (int(g["count"]), int(g["keep"]))

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {
            "architecture": self.architecture,
            "canon": {"taps": self.canon_taps},
            "embedding": {"scale": self.embedding_scale},
            "layers": [copy.deepcopy(dict(l)) for l in self.layers],
            "loop": dict(zip(("start", "stop", "times"), self.loop)),
            "norm": {"eps": self.norm_eps},
            "vocab": self.vocab,
            "width": self.width,
            # (read by this package's own tools: the tests' trace helper and the random-weights writer)
            "vocab_size": self.vocab,
            "initializer_range": self.initializer_range,
        }
        if self.eos_token_id:
            d["eos_token_id"] = list(self.eos_token_id)
        return d

    def init_scales(self) -> Dict[str, float]:
        s = self.initializer_range
        return {"matrix": s, "bias": s, "norm": s}

    # ------------------------------------------------------------------
    def _mixer_spec(self, i: int, layer: Mapping[str, Any]) -> PartSpec:
        m, prefix, size = layer["mixer"], f"l{i}.mix.", _mask_size(layer["mixer"])
        if layer["type"] == "attention":
            heads = int(m["heads"])
            return PartSpec("modulated_attention", {
                "hidden_size": self.width, "num_heads": heads, "num_kv_heads": int(m["kv_heads"]),
                "head_dim": int(m["dim"]), "value_head_dim": int(m["vdim"]), "scale": float(m["scale"]),
                "eps": self.norm_eps, "conv": int(m["conv"]),
                "distance_slopes": geometric_slopes(heads, SLOPE_EXPONENT),
                "mask": "causal" if size is None else "chunk", "mask_size": size}, prefix)
        rot = m["rot"]
        return PartSpec("latent_attention", {
            "hidden_size": self.width, "heads": int(m["heads"]), "dim": int(m["dim"]), "rot_dim": int(m["rot_dim"]),
            "vdim": int(m["vdim"]), "kv_rank": int(m["kv_rank"]), "q_rank": int(m["q_rank"]), "window": size,
            "scale": float(m["scale"]), "rot_base": float(rot["base"]), "rot_dims": int(rot["dims"]),
            "rot_layout": "half_split", "rot_scaling": None if not rot.get("scaling") else dict(rot["scaling"]),
            "channel_gate": True, "eps": self.norm_eps}, prefix)

    def _mlp_spec(self, i: int, mlp: Mapping[str, Any]) -> PartSpec:
        prefix = f"l{i}.mlp."
        if mlp["kind"] == "dense":
            return PartSpec("gated_mlp", {
                "hidden_size": self.width, "intermediate_size": int(mlp["ff"]), "activation": "clamped_swish",
                "limit": float(mlp["limit"]), "swish_alpha": SWISH_ALPHA, "tensor_names": ("gate", "up", "down")}, prefix)
        r = mlp["router"]
        return PartSpec("routed_experts", {
            "hidden_size": self.width, "experts": int(r["experts"]), "top": int(r["top"]),
            "expert_ff": int(mlp["expert"]["ff"]), "gated": True, "gate_form": "silu", "score": "softmax",
            "correction": True, "groups": self._groups(r), "weight_scale": float(r["scale"]),
            "identity": int(r.get("identity") or 0)}, prefix)

    def run_order(self) -> Tuple[RunStep, ...]:
        start, stop, times = self.loop
        order: List[RunStep] = [RunStep(i) for i in range(start)]
        for k in range(times):
            order += [RunStep(i, add_embedding=k > 0 and i == start) for i in range(start, stop)]
        return tuple(order + [RunStep(i) for i in range(stop, len(self.layers))])

    def model_spec(self) -> ModelSpec:
        norm = {"hidden_size": self.width, "eps": self.norm_eps, "offset": 1.0, "tensor": ""}
        conv = {"hidden_size": self.width, "taps": self.canon_taps, "tensor": ""}
        layers: List[LayerSpec] = []
        for i, layer in enumerate(self.layers):
            parts = {"mixer_norm": PartSpec("rms_norm_f32", norm, f"l{i}.norm1"),
                     "mixer_conv": PartSpec("short_conv", conv, f"l{i}.canon1"), "mixer": self._mixer_spec(i, layer)}
            mlp = layer.get("mlp")
            if mlp is None:
                layers.append(LayerSpec("pre_norm_conv_mixer_only", parts))
                continue
            parts["feed_forward_norm"] = PartSpec("rms_norm_f32", norm, f"l{i}.norm2")
            parts["feed_forward_conv"] = PartSpec("short_conv", conv, f"l{i}.canon2")
            parts["feed_forward"] = self._mlp_spec(i, mlp)
            layers.append(LayerSpec("pre_norm_conv", parts))
        return ModelSpec(
            architecture=self.architecture, hidden_size=self.width, vocab_size=self.vocab,
            max_positions=MAX_POSITIONS,
            embedding=PartSpec("token_embedding", {"vocab_size": self.vocab, "hidden_size": self.width,
                                                   "residual": "float32", "scale": self.embedding_scale,
                                                   "tensor": ""}, "embed"),
            layers=tuple(layers), order=self.run_order(), final_norm=PartSpec("rms_norm_f32", norm, "final.norm"),
            head=PartSpec("lm_head", {"vocab_size": self.vocab, "hidden_size": self.width, "tensor": ""}, "head"),
            eos_token_ids=self.eos_token_id)


register_architecture(TusipelConfig.architecture, TusipelConfig)
