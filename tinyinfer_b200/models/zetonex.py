"""Zetonex: a decoder whose layers run mixer and feed-forward side by side on one norm of a float32 residual. Two kinds of
grouped-query attention (the values are the unrotated keys, a window that keeps a request's first positions and a gate per output
feature; differential attention with query and key norms, capped scores and a window) and two kinds of feed-forward (dense with
biases; a mixture whose experts are named by a table of token ids). A stretch of layers may run several times, each pass
starting from a projection of the residual beside the embedding. The blocks, cache and step function are the generic decoder's;
the frame (one float32 stream, what passes start with, final norm on the wanted rows, untied head with a constant factor) is
the scaled-residual decoder's."""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.zetonex import NAME, ZetonexConfig
from .decoder import ScaledResidualDecoderModel


class ZetonexForCausalLM(ScaledResidualDecoderModel):
    def __init__(self, config: ZetonexConfig, dtype, device):
        super().__init__(config.model_spec(), dtype, device, logit_scale=config.logit_scale)
        self.config = config


def _layers(pattern: str, kept: dict, difference: dict, dense: dict, moe: dict):
    """config.json layers from a pattern of letters: 'k' the attention that keeps first positions, 'd' the differential one; a
    capital letter gives the layer the mixture of experts, a small one the dense feed-forward."""
    kinds = {"k": ("attention", kept), "d": ("attention_2", difference)}
    return [dict(type=kinds[c.lower()][0], mixer=dict(kinds[c.lower()][1]), mlp=dict(moe) if c.isupper() else dict(dense))
            for c in pattern]


def _moe(experts: int, top: int, ff: int):
    return dict(kind="moe", expert=dict(ff=ff, limit=7.0), router=dict(experts=experts, top=top))


def _scaling(original: int):
    return dict(factor=8.0, low=1.0, high=4.0, original=original)


# Sizes worth running with random weights (config.json keys): a toy, and two with the layer sizes of models of about
# one and of a few billion parameters, eight layer runs each (a benchmark runs as many layers as it lists).
PRESETS = {
    "zetonex-tiny": dict(
        vocab=256, width=64, norm=dict(eps=1e-6), logit_scale=0.7, loop=dict(start=0, stop=2, times=2),
        layers=_layers("kDKd", dict(heads=4, kv_heads=2, dim=16, vdim=16, scale=0.25, mask=dict(size=12, keep_first=3),
                                    rot=dict(base=10000.0, dims=8)),
                       dict(heads=4, kv_heads=1, dim=8, vdim=16, scale=0.35, softcap=30.0, diff=0.4, mask=dict(size=20),
                            rot=dict(base=10000.0, dims=8, scaling=_scaling(64))),
                       dict(kind="dense", ff=96), _moe(6, 2, 32))),
    "zetonex-1b": dict(
        vocab=102400, width=1024, norm=dict(eps=1e-6), logit_scale=1.0, loop=dict(start=2, stop=4, times=2),
        layers=_layers("kD" * 3, dict(heads=8, kv_heads=4, dim=128, vdim=128, scale=128 ** -0.5, mask=dict(size=1024, keep_first=4),
                                      rot=dict(base=10000.0, dims=64)),
                       dict(heads=8, kv_heads=4, dim=64, vdim=128, scale=0.125, softcap=50.0, diff=0.3, mask=dict(size=2048),
                            rot=dict(base=500000.0, dims=64, scaling=_scaling(8192))),
                       dict(kind="dense", ff=3072), _moe(32, 4, 704))),
    "zetonex-2b": dict(
        vocab=102400, width=2048, norm=dict(eps=1e-6), logit_scale=1.0, loop=dict(start=2, stop=4, times=2),
        layers=_layers("kD" * 3, dict(heads=16, kv_heads=8, dim=128, vdim=128, scale=128 ** -0.5, mask=dict(size=1024, keep_first=4),
                                      rot=dict(base=10000.0, dims=64)),
                       dict(heads=16, kv_heads=8, dim=64, vdim=128, scale=0.125, softcap=50.0, diff=0.3, mask=dict(size=2048),
                            rot=dict(base=500000.0, dims=64, scaling=_scaling(8192))),
                       dict(kind="dense", ff=6144), _moe(64, 6, 1408))),
}

register_architecture(NAME, ZetonexConfig, ZetonexForCausalLM, presets=PRESETS)
