"""Typed configuration of the Tarupel decoder, read from the keys of its own config.json.

config.json: ``architecture`` (the name), ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``, ``residual_mult``,
``loop.{start, stop, times}`` and ``layers``, a list whose entries give ``type`` (which mixer), ``mixer`` (its sizes) and
``mlp`` (its feed-forward, or null). Mixer types:
``attention``: ``heads, kv_heads, dim, vdim, scale, conv, mask.size, rot.{base, dims}``: convolved q, k and v, attention
within chunks of ``mask.size`` positions;
``attention_2``: ``heads, kv_heads, dim, vdim, scale, mask.size, rot.{base, dims}``: q and k normed as a whole, a sliding
window of ``mask.size`` keys;
``general_delta``: ``heads, dim`` (the inner size of the decay's two projections is the checkpoint's, or ``gate_rank`` for
random weights).
Feed-forward: ``kind`` "dense" with ``ff``, or "moe" with ``expert.ff``, ``router.{experts, top, scale,
groups.{count, keep}}`` and ``shared.ff``. Every size and constant comes from there; tensors are named ``embed``, ``head``,
``final.norm``, ``loop.step`` and ``l<i>.{norm1, norm2, ls1, ls2, shift, mix.*, mlp.*}``. A key that is absent switches its
mechanism off where that means something (``loop``, ``mask``, ``rot``, ``conv``, ``groups``, ``shared``: none;
``embedding.scale``, ``residual_mult``, ``router.scale``: 1).
"""
from __future__ import annotations

import copy
import math
from dataclasses import dataclass, field
from typing import List, Optional, Tuple

from .specs import (AttentionSpec, ExecStep, ExpertsSpec, GatedMLPSpec, GeneralDeltaSpec, LayerSpec, ModelSpec, NormSpec,
                    PositionSpec, TensorNames)

NAME = "Tarupel"
MAX_POSITIONS = 1 << 20             # the design sets no limit; the engine's tables need one
DECAY_SCALE = -math.exp(-0.5)       # the delta rule's decay: exp(-exp(-1/2) sigmoid(.))
UNIT_EPS = 1e-6                     # its unit key: k / sqrt(sum k^2 + 1e-6)
_ATTENTION = ("heads", "kv_heads", "dim", "vdim", "scale")
_REQUIRED = {"attention": _ATTENTION, "attention_2": _ATTENTION, "general_delta": ("heads", "dim")}


def _position(m: dict, interleaved: bool) -> PositionSpec:
    rot = m.get("rot")
    if not rot or not int(rot.get("dims", 0)):
        return PositionSpec(kind="none")
    return PositionSpec(kind="rope", theta=float(rot["base"]), rotary_dim=int(rot["dims"]), exact_frequencies=True,
                        interleaved=interleaved)


def _mask_size(m: dict) -> Optional[int]:
    size = (m.get("mask") or {}).get("size")
    return None if size is None else int(size)


@dataclass
class TarupelConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: List[dict]
    embedding_scale: float = 1.0
    residual_mult: float = 1.0
    loop: Optional[dict] = None
    eos_token_id: Optional[int] = None
    torch_dtype: Optional[str] = None
    architectures: List[str] = field(default_factory=lambda: [NAME])

    # ------------------------------------------------------------------ parsing
    @classmethod
    def from_dict(cls, data: dict) -> "TarupelConfig":
        missing = [k for k in ("vocab", "width", "layers", "norm") if k not in data]
        if missing:
            raise ValueError(f"config.json lacks required keys: {missing}")
        loop = data.get("loop")
        cfg = cls(vocab=int(data["vocab"]), width=int(data["width"]), norm_eps=float(data["norm"]["eps"]),
                  layers=copy.deepcopy(list(data["layers"])),
                  embedding_scale=float((data.get("embedding") or {}).get("scale", 1.0)),
                  residual_mult=float(data.get("residual_mult", 1.0)), loop=dict(loop) if loop else None,
                  eos_token_id=data.get("eos_token_id"), torch_dtype=data.get("torch_dtype", data.get("dtype")))
        cfg.validate()
        return cfg

    def to_dict(self) -> dict:
        d = {"architecture": NAME, "embedding": {"scale": self.embedding_scale}, "layers": copy.deepcopy(self.layers),
             "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult, "vocab": self.vocab, "width": self.width}
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
            start, stop, times = (int(self.loop[k]) for k in ("start", "stop", "times"))
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
            if kind != "general_delta":
                if int(m["heads"]) % int(m["kv_heads"]):
                    raise ValueError(f"layer {i}: heads must be a multiple of kv_heads")
                rot = m.get("rot")
                if rot and int(rot.get("dims", 0)) and ("base" not in rot or int(rot["dims"]) % 2
                                                        or int(rot["dims"]) > int(m["dim"])):
                    raise ValueError(f"layer {i}: rot needs a base, and dims even and at most dim")
                if _mask_size(m) is not None and _mask_size(m) < 1:
                    raise ValueError(f"layer {i}: mask.size must be at least 1")
                if int(m.get("conv", 0)) < 0:
                    raise ValueError(f"layer {i}: conv must not be negative")
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
        if any(k not in router for k in ("experts", "top")) or "ff" not in expert:
            raise ValueError(f"layer {i}: a mixture of experts needs router.experts, router.top and expert.ff")
        if f.get("shared") is not None and "ff" not in f["shared"]:
            raise ValueError(f"layer {i}: a shared expert needs shared.ff")
        experts, top, (count, keep) = int(router["experts"]), int(router["top"]), TarupelConfig._groups(router)
        if count < 1 or experts % count or not 1 <= keep <= count:
            raise ValueError(f"layer {i}: router.groups must cut the experts into equal groups and keep some of them")
        if not 1 <= top <= keep * (experts // count):
            raise ValueError(f"layer {i}: router.top exceeds the experts that can be chosen")

    @staticmethod
    def _groups(router: dict) -> Tuple[int, int]:
        groups = router.get("groups") or {}
        count = int(groups.get("count", 1))
        return count, int(groups.get("keep", count))

    # ------------------------------------------------------------------ layers
    def execution(self) -> Tuple[ExecStep, ...]:
        """Every run of a layer has a cache entry of its own: a layer that runs twice keeps two caches and two states. A
        pass of the loop starts with its row of ``loop.step``, every pass but the first also with the embedding."""
        n = len(self.layers)
        start, stop, times = (int(self.loop[k]) for k in ("start", "stop", "times")) if self.loop else (n, n, 0)
        order = [(i, None) for i in range(start)]
        order += [(i, t if i == start else None) for t in range(times) for i in range(start, stop)]
        order += [(i, None) for i in range(stop, n)]
        return tuple(ExecStep(layer=i, cache=e, writes_cache=True, adds_embedding=bool(t), adds_vector=t)
                     for e, (i, t) in enumerate(order))

    def _mixer(self, kind: str, m: dict):
        eps, width = float(self.norm_eps), self.width
        if kind == "general_delta":
            return GeneralDeltaSpec(hidden_size=width, num_heads=int(m["heads"]), key_dim=int(m["dim"]),
                                    value_dim=int(m["dim"]), decay_scale=DECAY_SCALE, norm_eps=eps, unit_eps=UNIT_EPS,
                                    gate_rank=int(m.get("gate_rank", 0)))
        common = dict(hidden_size=width, num_heads=int(m["heads"]), num_kv_heads=int(m["kv_heads"]), head_dim=int(m["dim"]),
                      scale=float(m["scale"]), v_dim=int(m["vdim"]), short_names=True, qkv_bias=True)
        if kind == "attention":
            return AttentionSpec(position=_position(m, interleaved=False), conv_taps=int(m.get("conv", 0)), qk_unit_norm=eps,
                                 chunk=_mask_size(m), **common)
        return AttentionSpec(position=_position(m, interleaved=True), qk_row_norm=NormSpec(0, eps, tensor=""),
                             window=_mask_size(m), **common)

    def _feed_forward(self, f: Optional[dict]):
        if f is None:
            return None
        if f["kind"] == "dense":
            return GatedMLPSpec(hidden_size=self.width, intermediate_size=int(f["ff"]), activation="gelu_tanh",
                                names=("gate", "up", "down"))
        router, shared = f["router"], f.get("shared")
        count, keep = self._groups(router)
        return ExpertsSpec(hidden_size=self.width, num_experts=int(router["experts"]), top=int(router["top"]),
                           expert_size=int(f["expert"]["ff"]), shared_size=int(shared["ff"]) if shared else 0,
                           activation="silu_glu", router_input="input", groups=count, keep_groups=keep,
                           weight_scale=float(router.get("scale", 1.0)), shared_gate=bool(shared))

    def model_spec(self) -> ModelSpec:
        norm = NormSpec(self.width, float(self.norm_eps), tensor="", single_gain=True)
        layers = []
        for layer in self.layers:
            ffn = self._feed_forward(layer.get("mlp"))
            layers.append(LayerSpec(mixer=self._mixer(layer["type"], layer["mixer"]), feed_forward=ffn, mixer_norm=norm,
                                    feed_forward_norm=norm if ffn is not None else None, arrangement="scaled_residual",
                                    residual_mult=float(self.residual_mult), mixer_scale="ls1", feed_forward_scale="ls2",
                                    token_shift="shift"))
        names = TensorNames(embedding="embed", layer="l{i}.", mixer="mix.", feed_forward="mlp.", mixer_norm="norm1",
                            feed_forward_norm="norm2", final_norm="final.norm", head="head")
        return ModelSpec(architecture=NAME, vocab_size=self.vocab, hidden_size=self.width, layers=tuple(layers),
                         execution=self.execution(), final_norm=norm, tie_embeddings=False, max_positions=MAX_POSITIONS,
                         names=names, step_vectors=("loop.step", int(self.loop["times"])) if self.loop else None)
