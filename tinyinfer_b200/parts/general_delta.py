"""The generalized delta rule with a decay and a removal rate per head and key channel. r, k and v are projections of the
input, heads side by side; with u = k / sqrt(k.k + eps) the unit key of a head,
    w = exp(decay_scale * sigmoid(W_w2 tanh(W_w1 h) + w0))        a = sigmoid(W_a h + b)        per head and key channel
    S <- diag(w) S - (a * u) (u^T S) + k v^T   (both terms read the old S)        o = S^T r
so what is taken away lies along the unit key, channel by channel at a rate of its own, and what is added is the key as it
is. Each head's o is divided by its root mean square; the heads side by side are multiplied by one weight of their length
and by sigmoid(W_g h), and projected.

Float32: the logits of the decay and of the rate (their products leave their kernels unrounded), tanh, sigmoids,
exponentials, unit keys, the state, the recurrence, its outputs and their norm. The state slot of a request holds S,
transposed, [heads, value_dim, key_dim].
"""
from __future__ import annotations

import torch

from .. import ops
from .base import Mixer, StateNeed, TensorSpec, register_mixer


class GeneralDelta(Mixer):
    graph_safe = True

    def __init__(self, spec, dtype, device):
        super().__init__(spec, dtype, device)
        self.w_in = self.w_gates = self.w_w2 = self.w_o = None
        self.decay_bias = self.rate_bias = self.norm_w = None

    @property
    def _sizes(self):
        s = self.spec
        return s.num_heads * s.key_dim, s.num_heads * s.value_dim

    def state_need(self):
        s = self.spec
        return StateNeed((s.num_heads * s.value_dim * s.key_dim,), torch.float32)

    def tensors(self):
        s = self.spec
        nk, nv = self._sizes
        rank = s.gate_rank if s.gate_rank > 0 else -1
        return {"r": TensorSpec((nk, s.hidden_size)), "k": TensorSpec((nk, s.hidden_size)), "v": TensorSpec((nv, s.hidden_size)),
                "g": TensorSpec((nv, s.hidden_size)), "a": TensorSpec((nk, s.hidden_size)),
                "a.b": TensorSpec((nk,), role="vector32"), "w1": TensorSpec((rank, s.hidden_size)),
                "w2": TensorSpec((nk, rank)), "w0": TensorSpec((nk,), role="vector32"),
                "norm": TensorSpec((nv,), role="vector32", init="ones_noise"), "o": TensorSpec((s.hidden_size, nv))}

    def load(self, tensors):
        if tensors["w1"].shape[0] != tensors["w2"].shape[1]:
            raise ValueError("the two projections of the decay do not fit each other")

        def packed(names):          # zero rows up to a multiple of eight, which the tensor-core product wants of its output's rows
            rows = [tensors[n] for n in names]
            fill = (-sum(r.shape[0] for r in rows)) % 8
            return torch.cat(rows + ([rows[0].new_zeros((fill, rows[0].shape[1]))] if fill else []), dim=0).contiguous()
        self.w_in = packed(["r", "k", "v", "g"])
        self.w_gates = packed(["a", "w1"])                  # both leave their product as float32
        self.rank = tensors["w1"].shape[0]
        self.w_w2, self.w_o = tensors["w2"].contiguous(), tensors["o"].contiguous()
        self.rate_bias, self.decay_bias, self.norm_w = tensors["a.b"], tensors["w0"], tensors["norm"]

    def _features(self, x, step, cache):
        s = self.spec
        nk, nv = self._sizes
        rkvg = ops.linear(x, self.w_in)                                                # [T, r | k | v | g]
        gates = ops.linear(x, self.w_gates, out_float32=True)                          # float32 [T, a | w1]
        decay = ops.linear(ops.tanh_rows(gates, nk, self.rank, self.dtype), self.w_w2, out_float32=True)
        state = cache.state.unflatten(1, (s.num_heads, s.value_dim, s.key_dim))
        o = ops.general_delta_scan(rkvg, rkvg, rkvg, decay, gates, decay_bias=self.decay_bias, rate_bias=self.rate_bias,
                                   decay_scale=s.decay_scale, state=state, heads=s.num_heads, key_dim=s.key_dim,
                                   value_dim=s.value_dim, r_offset=0, k_offset=nk, v_offset=2 * nk, unit_eps=s.unit_eps,
                                   cu_seqlens=step.cu_seqlens, state_slots=step.state_slots, num_seqs=step.num_seqs)
        return ops.gated_group_norm(o, rkvg, self.norm_w, group=s.value_dim, eps=s.norm_eps, gate_first=False,
                                    out_dtype=self.dtype, gate_offset=2 * nk + nv, gate_activation="sigmoid")

    def forward(self, x, step, cache):
        return ops.linear(self._features(x, step, cache), self.w_o)

    def forward_residual(self, x, residual, step, cache):
        return ops.linear(self._features(x, step, cache), self.w_o, residual=residual)


register_mixer("general_delta", GeneralDelta)
