"""The generic decoder: embedding, blocks run in the order the spec lists, final norm on the
wanted rows, output projection to float32 logits.

It plays the role of the reference's Qwen3ForCausalLM / Qwen3Model
(tinyinfer/models/qwen3.py:225-288) but knows no architecture: which mixer, feed-forward and
norm a layer has, and which layers run in which order on which cache entry, all come from the
``ModelSpec``. Only rows that want logits reach the final norm and the head, as in the
reference's runner (tinyinfer/engine/model_runner.py:381-395).
"""
from __future__ import annotations

from typing import Dict, List, Optional, Tuple

import torch

from .. import ops
from ..config.specs import ModelSpec
from ..parts.experts import TableRoutes
from ..parts import CacheNeed, StateNeed, TensorSpec, build_block, build_norm


class DecoderModel:
    def __init__(self, spec: ModelSpec, dtype: torch.dtype, device):
        if dtype not in (torch.float32, torch.bfloat16):
            raise ValueError(f"compute dtype must be float32 or bfloat16, got {dtype}")
        self.spec = spec
        self.dtype = dtype
        self.device = torch.device(device)
        self.blocks = [build_block(layer, dtype, self.device) for layer in spec.layers]
        self.final_norm = build_norm(spec.final_norm, dtype, self.device)
        self.embedding: Optional[torch.Tensor] = None
        self.head: Optional[torch.Tensor] = None
        self.entry_weight: Optional[torch.Tensor] = None      # of the entries that project [x; embedding]
        self.table_routes: Optional[TableRoutes] = None       # feed-forwards whose routing depends on the token ids alone
        self.step_vectors: Optional[torch.Tensor] = None      # float32 [rows, hidden]: what entries of the run order add

    # ------------------------------------------------------------------ tensors
    def _part_prefixes(self, i: int):
        n = self.spec.names
        number = self.spec.layers[i].index
        base = n.layer.format(i=i if number is None else number)
        block = self.blocks[i]
        parts = [(base + n.mixer, block.mixer), (base + n.feed_forward, block.feed_forward),
                 (base + n.mixer_norm, block.mixer_norm),
                 (base + n.feed_forward_norm, block.feed_forward_norm),
                 (base, block if block.tensors() else None)]     # tensors of the arrangement itself, if it has any
        return [(prefix, part) for prefix, part in parts if part is not None]     # a block may have a mixer only

    def expected_tensors(self) -> Dict[str, TensorSpec]:
        """Checkpoint name -> what the tensor must look like, in a fixed order."""
        spec = self.spec
        out: Dict[str, TensorSpec] = {
            spec.names.embedding: TensorSpec((spec.vocab_size, spec.hidden_size))}
        for i in range(len(self.blocks)):
            for prefix, part in self._part_prefixes(i):
                for local, ts in part.tensors().items():
                    out[prefix + local] = ts
        if spec.entry_projection:
            out[spec.entry_projection] = TensorSpec((spec.hidden_size, 2 * spec.hidden_size))
        if spec.step_vectors:
            out[spec.step_vectors[0]] = TensorSpec((spec.step_vectors[1], spec.hidden_size), role="vector32")
        for local, ts in self.final_norm.tensors().items():
            out[spec.names.final_norm + local] = ts
        if not spec.tie_embeddings:
            out[spec.names.head] = TensorSpec((spec.vocab_size, spec.hidden_size))
        return out

    def ignored_tensors(self) -> List[str]:
        """Names a checkpoint may carry that this model has no use for (a tied model's head,
        tinyinfer/utils/loader.py:103-105 of the reference)."""
        return [self.spec.names.head] if self.spec.tie_embeddings else []

    def load_tensors(self, tensors) -> None:
        """``tensors[name]``: the tensor of that name of ``expected_tensors()``, on the device, role
        applied. Every name is asked for once, in the order of ``expected_tensors()``, and a part's
        tensors are let go of as soon as the part has packed them: a mapping that makes each tensor
        when it is asked for (a reader of a file, a random draw) never has more than one part's
        tensors alive beside the model, which is what lets a model of 65 GB load into 180 GB."""
        spec = self.spec
        self.embedding = tensors[spec.names.embedding].contiguous()
        for i in range(len(self.blocks)):
            for prefix, part in self._part_prefixes(i):
                part.load({local: tensors[prefix + local] for local in part.tensors()})
        table_parts = [b.feed_forward for b in self.blocks if getattr(b.feed_forward, "table", None) is not None]
        self.table_routes = TableRoutes(table_parts) if table_parts else None
        if spec.entry_projection:
            self.load_entry_projection(tensors[spec.entry_projection])
        if spec.step_vectors:
            self.step_vectors = tensors[spec.step_vectors[0]].contiguous()
        self.final_norm.load({local: tensors[spec.names.final_norm + local]
                              for local in self.final_norm.tensors()})
        self.head = self.embedding if spec.tie_embeddings else tensors[spec.names.head].contiguous()

    def weight_bytes(self) -> int:
        total = 0
        for name, ts in self.expected_tensors().items():
            n = 1
            for s in ts.shape:
                n *= max(s, 0)        # a size only the checkpoint gives counts as nothing
            total += n * (self.dtype.itemsize if ts.role == "matrix" else 4)
        return total

    # ------------------------------------------------------------------ cache needs
    def cache_needs(self) -> List[Tuple[Optional[CacheNeed], Optional[StateNeed]]]:
        """For every cache entry of the run order: the pages and the state its writer wants."""
        needs: List[Tuple[Optional[CacheNeed], Optional[StateNeed]]] = \
            [(None, None)] * self.spec.num_cache_entries
        for step in self.spec.execution:
            if step.writes_cache:
                mixer = self.blocks[step.layer].mixer
                needs[step.cache] = (mixer.cache_need(), self.blocks[step.layer].state_need())
        return needs

    # ------------------------------------------------------------------ forward
    # The frame around the blocks is three methods, so that a model whose frame differs (an embedding
    # that is scaled, logits that are capped, a norm elsewhere) overrides one of them in a subclass and
    # registers that class for its architecture; blocks, cache and step function stay as they are.
    def forward(self, step) -> torch.Tensor:
        """Runs the tokens of ``step`` (a StepContext) and returns float32 logits [N, V] at
        ``step.logit_rows``."""
        if self.table_routes is not None:
            self.table_routes.route(step)
        x = self.run_blocks(self.embed(step), step)
        if step.num_logit_rows == 0:
            return torch.empty((0, self.spec.vocab_size), dtype=torch.float32, device=self.device)
        return self.logits(x, step)

    def embed(self, step) -> torch.Tensor:
        """The residual stream [T, hidden] the first block starts from."""
        return ops.embedding(step.token_ids, self.embedding)

    def run_blocks(self, x: torch.Tensor, step) -> torch.Tensor:
        """The blocks in the order the spec lists, each on its cache entry."""
        link = None        # what a block's last product leaves for the next block's first norm (see parts.base)
        order = self.spec.execution
        for i, entry in enumerate(order):
            if entry.adds_embedding or entry.projects_embedding or entry.adds_vector is not None:
                x, link = self.enter(x, entry, step), None
            after = self.blocks[order[i + 1].layer].mixer_norm if i + 1 < len(order) else None
            x, link = self.blocks[entry.layer].forward_linked(x, link, after, step, step.cache_view(entry))
        return x

    def load_entry_projection(self, weight: torch.Tensor) -> None:
        """``weight`` [hidden, 2 hidden] of the entries that project [x; embedding]."""
        self.entry_weight = weight.contiguous()

    def enter(self, x, entry, step=None):
        """What an entry of the run order does to the residual right before its layer."""
        raise NotImplementedError(f"{type(self).__name__} has no residual that an entry of the run order could add to")

    def logits(self, x: torch.Tensor, step) -> torch.Tensor:
        """Float32 logits [N, V] of the rows ``step.logit_rows`` (there is at least one) of the last
        block's output."""
        h = self.final_norm.forward_rows(x, step.logit_rows)
        return ops.linear(h, self.head, out_float32=True)


class StreamDecoderModel(DecoderModel):
    """The frame of the decoders whose blocks are 'multi_stream' blocks around ONE float32 residual stream: the
    embedding times a constant goes into the stream; at the end the last sublayer's update, the final norm and the
    choice of the wanted rows are one kernel, then the head and, if asked for, a smooth cap c * tanh(z / c) on the
    logits. What travels between the blocks is the pair (stream [1, T, width], update still to be applied)."""

    def __init__(self, spec: ModelSpec, dtype, device, *, embedding_scale: float = 1.0,
                 logit_softcap: Optional[float] = None):
        super().__init__(spec, dtype, device)
        self.embedding_scale = float(embedding_scale)
        self.logit_softcap = logit_softcap
        self._one = None

    def embed(self, step):
        return ops.streams_embed(step.token_ids, self.embedding, 1, self.embedding_scale), None

    def logits(self, x, step):
        stream, pending = x
        if self._one is None:
            self._one = torch.ones(1, dtype=torch.float32, device=self.device)
        rms = self.final_norm.as_rms()
        # the last sublayer's update and the final norm, for the wanted rows only
        h = ops.streams_step(stream, pending, self._one, rms[0], rms[1], self.dtype, rows=step.logit_rows)
        z = ops.linear(h, self.head, out_float32=True)
        return ops.soft_cap_(z, self.logit_softcap) if self.logit_softcap else z


class ScaledResidualDecoderModel(DecoderModel):
    """The frame of the decoders whose blocks are 'scaled_residual' blocks: the embedding times a constant starts one
    float32 stream [T, width]; what travels between the blocks is the pair (stream, update still to be applied). Entries of
    the run order may add the embedding's output and a row of the step vectors before their layer; both ride in the update.
    Entries may also replace the stream by W [x; x0], x0 being the embedding's output: one kernel applies the update and lays
    the operand rows out, a product makes the new stream. In a bfloat16 model x travels there as two halves, x = hi + lo, so
    that the residual never passes through 16 bits.
    At the end the last update, the final norm and the choice of the wanted rows are one kernel, then the head; a constant
    factor on the logits rides in the final norm's weight."""

    def __init__(self, spec: ModelSpec, dtype, device, *, embedding_scale: float = 1.0, logit_scale: float = 1.0):
        super().__init__(spec, dtype, device)
        self.embedding_scale = float(embedding_scale)
        self.logit_scale = float(logit_scale)
        self._logit_norm = None
        self._needs_start = any(e.adds_embedding for e in spec.execution)
        self._start = None

    def load_tensors(self, tensors) -> None:
        super().load_tensors(tensors)
        weight = self.final_norm.as_rms()[0]
        self._logit_norm = weight if self.logit_scale == 1.0 else (weight * self.logit_scale).contiguous()

    def load_entry_projection(self, weight):
        if self.dtype == torch.bfloat16:                  # the columns of x twice: for its upper and its lower half
            w = self.spec.hidden_size
            weight = torch.cat([weight[:, :w], weight], dim=1)
        super().load_entry_projection(weight)

    def embed(self, step):
        # the stream is updated in place: where later entries add what it started from, the kernel makes a second copy
        copies = ops.streams_embed(step.token_ids, self.embedding, 2 if self._needs_start else 1, self.embedding_scale)
        self._start = copies[1] if self._needs_start else None
        return copies[0], None

    def run_blocks(self, x, step):
        try:
            return super().run_blocks(x, step)
        finally:
            self._start = None

    def enter(self, x, entry, step=None):
        stream, pending = x
        if entry.projects_embedding:
            if entry.adds_embedding or entry.adds_vector is not None:
                raise ValueError("an entry projects the embedding or adds it, not both")
            rows = ops.residual_enter(stream, pending, self.embedding, step.token_ids, self.embedding_scale)
            return ops.linear(rows, self.entry_weight, out_float32=True), None
        pending = pending if pending is not None else ops.ResidualUpdate()
        pending.add_rows = self._start if entry.adds_embedding else None
        pending.add_vec = self.step_vectors[entry.adds_vector] if entry.adds_vector is not None else None
        return stream, pending

    def logits(self, x, step):
        stream, pending = x
        _, h = ops.residual_step(stream, pending, self._logit_norm, self.final_norm.as_rms()[1], self.dtype, rows=step.logit_rows)
        return ops.linear(h, self.head, out_float32=True)
