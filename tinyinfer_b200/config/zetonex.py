"""Typed configuration of the Zetonex decoder, read from the keys of its own config.json.

config.json: ``architecture`` (the name), ``vocab``, ``width``, ``norm.eps``, ``logit_scale``, ``loop.{start, stop, times}`` and
``layers``, a list whose entries give ``type`` (which mixer), ``mixer`` (its sizes) and ``mlp`` (its feed-forward, or null).
Mixer types:
``attention``: ``heads, kv_heads, dim, vdim, scale, mask.{size, keep_first}, rot.{base, dims}``: the values are the keys before
their rotation, a sliding window of ``mask.size`` keys beside the first ``mask.keep_first`` positions, a sigmoid gate per output
feature;
``attention_2``: ``heads, kv_heads, dim, vdim, scale, softcap, diff, mask.size, rot.{base, dims, scaling}``: two attention maps a
head, the second one's output subtracted; per-map query and key norms; ``rot.scaling`` = ``{factor, low, high, original}`` slows
the rotation's slow pairs down by their wavelength.
Feed-forward: ``kind`` "dense" with ``ff`` (biases on all projections), or "moe" with ``expert.{ff, limit}`` and
``router.{experts, top}``, where a table names the experts of a token id. Every size and constant comes from there; tensors are
named ``embed``, ``head``, ``final.norm``, ``loop.in`` and ``l<i>.{norm1, mix.*, mlp.*}``. A key that is absent switches its
mechanism off where that means something (``loop``, ``mask``, ``keep_first``, ``rot``, ``scaling``, ``softcap``: none;
``logit_scale``: 1).
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import List, Optional, Tuple

from .specs import (AttentionSpec, ExecStep, ExpertsSpec, GatedMLPSpec, LayerSpec, ModelSpec, NormSpec, PositionSpec, TensorNames,
                    WavelengthBlend)

NAME = "Zetonex"
MAX_POSITIONS = 1 << 20             # the design sets no limit; the engine's tables need one
GLU_ALPHA = 1.702                   # the experts' gate: g * sigmoid(1.702 g)
_ATTENTION = ("heads", "kv_heads", "dim", "vdim", "scale")
_REQUIRED = {"attention": _ATTENTION, "attention_2": _ATTENTION + ("diff",)}


def _position(m: dict) -> PositionSpec:
    rot = m.get("rot")
    if not rot or not int(rot.get("dims", 0)):
        return PositionSpec(kind="none")
    s = rot.get("scaling")
    blend = None
    if s:
        blend = WavelengthBlend(factor=float(s["factor"]), low=float(s["low"]), high=float(s["high"]), original=float(s["original"]))
    return PositionSpec(kind="rope", theta=float(rot["base"]), rotary_dim=int(rot["dims"]), exact_frequencies=True, blend=blend)


def _mask(m: dict, key: str) -> Optional[int]:
    value = (m.get("mask") or {}).get(key)
    return None if value is None else int(value)


@dataclass
class ZetonexConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: List[dict]
    logit_scale: float = 1.0
    loop: Optional[dict] = None
    eos_token_id: Optional[int] = None
    torch_dtype: Optional[str] = None
    architectures: List[str] = field(default_factory=lambda: [NAME])

    # ------------------------------------------------------------------ parsing
    @classmethod
    def from_dict(cls, data: dict) -> "ZetonexConfig":
        missing = [k for k in ("vocab", "width", "layers", "norm") if k not in data]
        if missing:
            raise ValueError(f"config.json lacks required keys: {missing}")
        loop = data.get("loop")
        cfg = cls(vocab=int(data["vocab"]), width=int(data["width"]), norm_eps=float(data["norm"]["eps"]),
                  layers=copy.deepcopy(list(data["layers"])), logit_scale=float(data.get("logit_scale", 1.0)),
                  loop=dict(loop) if loop else None, eos_token_id=data.get("eos_token_id"),
                  torch_dtype=data.get("torch_dtype", data.get("dtype")))
        cfg.validate()
        return cfg

    def to_dict(self) -> dict:
        d = {"architecture": NAME, "layers": copy.deepcopy(self.layers), "logit_scale": self.logit_scale,
             "norm": {"eps": self.norm_eps}, "vocab": self.vocab, "width": self.width}
        if self.loop is not None:
            d["loop"] = dict(self.loop)
        if self.eos_token_id is not None:
            d["eos_token_id"] = self.eos_token_id
        return d

    # ------------------------------------------------------------------ checks
    def validate(self) -> None:
        if self.vocab <= 0 or self.width <= 0 or not self.layers:
            raise ValueError("vocab, width and the number of layers must be positive")
        if not self.norm_eps > 0:
            raise ValueError("norm.eps must be positive")
        if self.loop is not None:
            if any(k not in self.loop for k in ("start", "stop", "times")):
                raise ValueError("loop needs start, stop and times")
            start, stop, times = self._loop()
            if not (0 <= start < stop <= len(self.layers)) or times < 1:
                raise ValueError("loop must name a stretch of the layers and run it at least once")
        for i, layer in enumerate(self.layers):
            kind, m = layer.get("type"), layer.get("mixer")
            if kind not in _REQUIRED:
                raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
            if not isinstance(m, dict):
                raise ValueError(f"layer {i} has no mixer sizes")
            for key in _REQUIRED[kind]:
                if key not in m:
                    raise ValueError(f"layer {i} ({kind}) lacks mixer.{key}")
            if int(m["heads"]) % int(m["kv_heads"]):
                raise ValueError(f"layer {i}: heads must be a multiple of kv_heads")
            if kind == "attention" and int(m["vdim"]) != int(m["dim"]):
                raise ValueError(f"layer {i}: values that are the keys have the keys' size")
            rot = m.get("rot")
            if rot and int(rot.get("dims", 0)):
                if "base" not in rot or int(rot["dims"]) % 2 or int(rot["dims"]) > int(m["dim"]):
                    raise ValueError(f"layer {i}: rot needs a base, and dims even and at most dim")
                s = rot.get("scaling")
                if s and any(k not in s for k in ("factor", "low", "high", "original")):
                    raise ValueError(f"layer {i}: rot.scaling needs factor, low, high and original")
            size, keep = _mask(m, "size"), _mask(m, "keep_first")
            if (size is not None and size < 1) or (keep is not None and keep < 0):
                raise ValueError(f"layer {i}: mask.size must be at least 1, mask.keep_first not negative")
            if m.get("softcap") is not None and not float(m["softcap"]) > 0:
                raise ValueError(f"layer {i}: softcap must be positive")
            self._validate_feed_forward(i, layer.get("mlp"))

    @staticmethod
    def _validate_feed_forward(i: int, f: Optional[dict]) -> None:
        if f is None:
            return
        if f.get("kind") == "dense":
            if "ff" not in f:
                raise ValueError(f"layer {i}: a dense feed-forward needs ff")
            return
        if f.get("kind") != "moe":
            raise ValueError(f"layer {i}: unknown feed-forward kind {f.get('kind')!r}")
        router, expert = f.get("router") or {}, f.get("expert") or {}
        if any(k not in router for k in ("experts", "top")) or any(k not in expert for k in ("ff", "limit")):
            raise ValueError(f"layer {i}: a mixture of experts needs router.experts, router.top, expert.ff and expert.limit")
        if not 1 <= int(router["top"]) <= int(router["experts"]):
            raise ValueError(f"layer {i}: top must lie between 1 and the number of experts")
        if not float(expert["limit"]) > 0:
            raise ValueError(f"layer {i}: expert.limit must be positive")

    # ------------------------------------------------------------------ layers
    def _loop(self) -> Tuple[int, int, int]:
        n = len(self.layers)
        return tuple(int(self.loop[k]) for k in ("start", "stop", "times")) if self.loop else (n, n, 0)

    def execution(self) -> Tuple[ExecStep, ...]:
        """Every run of a layer has a cache entry of its own: a layer that runs twice keeps two caches. A pass of the loop
        starts with the projection of the residual beside the embedding's output."""
        start, stop, times = self._loop()
        order = [(i, False) for i in range(start)]
        order += [(i, i == start) for _ in range(times) for i in range(start, stop)]
        order += [(i, False) for i in range(stop, len(self.layers))]
        return tuple(ExecStep(layer=i, cache=e, writes_cache=True, projects_embedding=first) for e, (i, first) in enumerate(order))

    def _mixer(self, kind: str, m: dict) -> AttentionSpec:
        eps = float(self.norm_eps)
        size, keep = _mask(m, "size"), _mask(m, "keep_first")
        common = dict(hidden_size=self.width, num_heads=int(m["heads"]), num_kv_heads=int(m["kv_heads"]), head_dim=int(m["dim"]),
                      scale=float(m["scale"]), v_dim=int(m["vdim"]), position=_position(m), window=size, short_names=True)
        if kind == "attention":          # without a window every position is seen, first ones or not
            return AttentionSpec(values_are_keys=True, feature_gate=True, keep_first=keep or 0 if size else 0, **common)
        softcap = m.get("softcap")
        return AttentionSpec(qk_norm=NormSpec(int(m["dim"]), eps, tensor=""), softcap=float(softcap) if softcap is not None else None,
                             difference=float(m["diff"]), difference_eps=eps, **common)

    def _feed_forward(self, f: Optional[dict]):
        if f is None:
            return None
        if f["kind"] == "dense":
            return GatedMLPSpec(hidden_size=self.width, intermediate_size=int(f["ff"]), activation="silu", names=("gate", "up", "down"),
                                bias=True)
        router, expert = f["router"], f["expert"]
        return ExpertsSpec(hidden_size=self.width, num_experts=int(router["experts"]), top=int(router["top"]),
                           expert_size=int(expert["ff"]), activation="clamped_glu", glu_limit=float(expert["limit"]),
                           glu_alpha=GLU_ALPHA, table_rows=self.vocab)

    def model_spec(self) -> ModelSpec:
        norm = NormSpec(self.width, float(self.norm_eps), tensor="", offset=1.0)
        layers = tuple(LayerSpec(mixer=self._mixer(layer["type"], layer["mixer"]), feed_forward=self._feed_forward(layer.get("mlp")),
                                 mixer_norm=norm, feed_forward_norm=None, arrangement="parallel_residual") for layer in self.layers)
        names = TensorNames(embedding="embed", layer="l{i}.", mixer="mix.", feed_forward="mlp.", mixer_norm="norm1",
                            feed_forward_norm="norm2", final_norm="final.norm", head="head")
        return ModelSpec(architecture=NAME, vocab_size=self.vocab, hidden_size=self.width, layers=layers, execution=self.execution(),
                         final_norm=norm, tie_embeddings=False, max_positions=MAX_POSITIONS, names=names,
                         entry_projection="loop.in" if self.loop else None)
