"""Tarupel: a pre-norm decoder whose layers mix two kinds of grouped-query attention (short convolutions on q, k and v,
q and k of unit root mean square after a half-split rotation, attention within chunks of positions; q and k normed as a
whole, an interleaved rotation, a sliding window) and the generalized delta rule (a decay and a removal rate per head and
key channel), each with a dense gelu-gated feed-forward, a mixture of experts chosen by groups with a gated shared expert, or
none. Norms have one gain, sublayers a scale per feature and a common factor, mixers read a token shift of their input; a
stretch of layers may run several times, each pass starting from its own vector and, after the first, from the embedding
once more. The blocks, cache and step function are the generic decoder's; the frame (scaled embedding into one float32
stream, what passes start with, final norm on the wanted rows, untied head) is the scaled-residual decoder's."""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.tarupel import NAME, TarupelConfig
from .decoder import ScaledResidualDecoderModel


class TarupelForCausalLM(ScaledResidualDecoderModel):
    def __init__(self, config: TarupelConfig, dtype, device):
        super().__init__(config.model_spec(), dtype, device, embedding_scale=config.embedding_scale)
        self.config = config


def _layers(pattern: str, chunked: dict, windowed: dict, delta: dict, dense: dict, moe: dict):
    """config.json layers from a pattern of letters: 'c' the chunked attention, 'w' the windowed one, 'd' the delta rule; a
    capital letter gives the layer the mixture of experts, a small one the dense feed-forward."""
    kinds = {"c": ("attention", chunked), "w": ("attention_2", windowed), "d": ("general_delta", delta)}
    return [dict(type=kinds[c.lower()][0], mixer=dict(kinds[c.lower()][1]), mlp=dict(moe) if c.isupper() else dict(dense))
            for c in pattern]


def _moe(experts: int, top: int, ff: int, groups: int, keep: int, shared: int):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top, scale=2.0, groups=dict(count=groups, keep=keep)),
                shared=dict(ff=shared))


# Sizes worth running with random weights (config.json keys): a toy, and two with the layer sizes of models of about
# one and of a few billion parameters, eight layer runs each (a benchmark runs as many layers as it lists).
PRESETS = {
    "tarupel-tiny": dict(
        vocab=256, width=64, norm=dict(eps=1e-5), embedding=dict(scale=4.0), residual_mult=0.7, loop=dict(start=1, stop=3, times=2),
        layers=_layers("cDwD",
                       dict(heads=4, kv_heads=2, dim=16, vdim=8, scale=0.25, conv=3, mask=dict(size=20), rot=dict(base=10000.0, dims=8)),
                       dict(heads=4, kv_heads=1, dim=16, vdim=16, scale=0.25, mask=dict(size=12), rot=dict(base=10000.0, dims=16)),
                       dict(heads=2, dim=16, gate_rank=8), dict(kind="dense", ff=96), _moe(6, 2, 32, 3, 2, 40))),
    "tarupel-1b": dict(
        vocab=102400, width=1024, norm=dict(eps=1e-6), embedding=dict(scale=32.0), residual_mult=1.0,
        layers=_layers("cDwD" * 2,
                       dict(heads=8, kv_heads=4, dim=128, vdim=128, scale=128 ** -0.5, conv=4, mask=dict(size=2048),
                            rot=dict(base=10000.0, dims=64)),
                       dict(heads=8, kv_heads=4, dim=128, vdim=128, scale=128 ** -0.5, mask=dict(size=1024),
                            rot=dict(base=1000000.0, dims=128)),
                       dict(heads=8, dim=128, gate_rank=64), dict(kind="dense", ff=3072), _moe(32, 4, 704, 4, 2, 704))),
    "tarupel-2b": dict(
        vocab=102400, width=2048, norm=dict(eps=1e-6), embedding=dict(scale=45.0), residual_mult=1.0,
        layers=_layers("cDwD" * 2,
                       dict(heads=16, kv_heads=8, dim=128, vdim=128, scale=128 ** -0.5, conv=4, mask=dict(size=2048),
                            rot=dict(base=10000.0, dims=64)),
                       dict(heads=16, kv_heads=8, dim=128, vdim=128, scale=128 ** -0.5, mask=dict(size=1024),
                            rot=dict(base=1000000.0, dims=128)),
                       dict(heads=16, dim=128, gate_rank=64), dict(kind="dense", ff=6144), _moe(64, 6, 1408, 8, 4, 1408))),
}

register_architecture(NAME, TarupelConfig, TarupelForCausalLM, presets=PRESETS)
