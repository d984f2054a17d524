"""Dense gated feed-forward: down(act(gate(x)) * up(x)), act silu (SwiGLU) or the tanh form of gelu, with or without biases
(tinyinfer/models/qwen3.py:148-150,170-175 of the reference). Gate and up are packed as one
[2I, H] matrix so that one matrix product feeds the activation, which acts on the float32
accumulators as the reference's kernel does (tinyinfer/csrc/mlp.cu:116-141)."""
from __future__ import annotations

import torch

from .. import ops
from .base import FeedForward, TensorSpec, register_feed_forward


class GatedMLP(FeedForward):
    graph_safe = True
    def __init__(self, spec, dtype, device):
        super().__init__(spec, dtype, device)
        if spec.activation not in ops.GATED_ACTIVATIONS:
            raise ValueError(f"activation {spec.activation!r} is not supported ({', '.join(ops.GATED_ACTIVATIONS)})")
        self.w_gate_up = self.w_down = self.b_gate_up = self.b_down = None

    def tensors(self):
        s = self.spec
        gate, up, down = s.names
        biases = {name + ".b": TensorSpec((rows,), role="vector32") for name, rows in
                  ((gate, s.intermediate_size), (up, s.intermediate_size), (down, s.hidden_size))} if s.bias else {}
        return {
            **biases,
            gate: TensorSpec((s.intermediate_size, s.hidden_size)),
            up: TensorSpec((s.intermediate_size, s.hidden_size)),
            down: TensorSpec((s.hidden_size, s.intermediate_size)),
        }

    def load(self, tensors):
        gate, up, down = self.spec.names
        self.w_gate_up = torch.cat([tensors[gate], tensors[up]], dim=0).contiguous()
        self.w_down = tensors[down].contiguous()
        if self.spec.bias:
            self.b_gate_up = torch.cat([tensors[gate + ".b"], tensors[up + ".b"]]).contiguous()
            self.b_down = tensors[down + ".b"].contiguous()

    def runs_beside(self, num_tokens):
        return num_tokens < 16            # from 16 tokens on the units of a product's tile wait for each other's partial sums

    def _hidden(self, x, **link):
        return ops.gated_linear(x, self.w_gate_up, bias=self.b_gate_up, activation=self.spec.activation, **link)

    def forward(self, x, step=None):
        return ops.linear(self._hidden(x), self.w_down, bias=self.b_down)

    def forward_residual(self, x, residual, step=None):
        return ops.linear(self._hidden(x), self.w_down, bias=self.b_down, residual=residual)

    def forward_prenorm(self, x, norm, link, next_norm, step=None):
        rms = norm.as_rms()
        if rms is None or self.spec.bias or not ops.norm_link_ok(x):
            return super().forward_prenorm(x, norm, link, next_norm, step)
        if link is not None and link.weight is rms[0]:
            hidden = self._hidden(link.scaled, link=link, link_eps=rms[1])
        else:
            hidden = self._hidden(norm.forward(x))
        after = next_norm.as_rms() if next_norm is not None else None
        if after is None:
            return ops.linear(hidden, self.w_down, residual=x), None
        return ops.linear(hidden, self.w_down, residual=x, next_norm_weight=after[0])


class DenseMLP(FeedForward):
    """Dense feed-forward without a gate: down(act(up h + b_up)) + b_down, act the exact (erf) gelu or its tanh
    form, computed in float32 on the stored product and rounded once."""
    graph_safe = True

    def __init__(self, spec, dtype, device):
        super().__init__(spec, dtype, device)
        if spec.activation not in ("gelu", "gelu_tanh"):
            raise ValueError(f"activation {spec.activation!r} is not supported (gelu, gelu_tanh)")
        self.w_up = self.b_up = self.w_down = self.b_down = None

    def tensors(self):
        s = self.spec
        t = {"up": TensorSpec((s.intermediate_size, s.hidden_size)),
             "down": TensorSpec((s.hidden_size, s.intermediate_size))}
        if s.bias:
            t["up.b"] = TensorSpec((s.intermediate_size,), role="vector32")
            t["down.b"] = TensorSpec((s.hidden_size,), role="vector32")
        return t

    def load(self, tensors):
        self.w_up, self.w_down = tensors["up"].contiguous(), tensors["down"].contiguous()
        if self.spec.bias:
            self.b_up, self.b_down = tensors["up.b"], tensors["down.b"]

    def _hidden(self, x):
        up = ops.linear(x, self.w_up, bias=self.b_up)
        return ops.gelu(up, tanh=self.spec.activation == "gelu_tanh", out=up)

    def forward(self, x, step=None):
        return ops.linear(self._hidden(x), self.w_down, bias=self.b_down)

    def forward_residual(self, x, residual, step=None):
        return ops.linear(self._hidden(x), self.w_down, bias=self.b_down, residual=residual)


register_feed_forward("gated_mlp", GatedMLP)
register_feed_forward("dense_mlp", DenseMLP)
