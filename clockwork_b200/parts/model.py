"""The decoder model: embedding, the layers in their run order, final norm, output head.

Reference: ``clockwork/engine/model.py:157-233`` (embedding, layer stack, final norm, logits
only at the requested rows, output head tied to the embedding when ``tie_word_embeddings``).
Built from a ``ModelSpec`` alone.  ``forward`` runs one flat batch of tokens (whatever mixture
of prompt portions and decoded tokens the step function assembled) and returns float32 logits
for the requested rows.
"""

from __future__ import annotations

import torch

from .. import ops
from ..config.model_spec import ModelSpec
from ..weights.decl import TensorDecl
from .base import PagedKVNeed, ResidualStream, SlotStateNeed, StepContext
from .linear import Linear
from .registry import build_block, build_part


class DecoderModel:
    def __init__(self, spec: ModelSpec, dtype: torch.dtype, device) -> None:
        spec.validate()
        if dtype not in (torch.float32, torch.bfloat16):
            raise ValueError(f"run dtype must be float32 or bfloat16, got {dtype}")
        self.spec = spec
        self.dtype = dtype
        self.device = torch.device(device)
        self.blocks = [build_block(layer, dtype, self.device) for layer in spec.layers]
        self.final_norm = build_part("norm", spec.final_norm, spec.final_norm_prefix, dtype, self.device)
        self.absolute_positions = None
        if spec.absolute_positions is not None:
            self.absolute_positions = build_part("position", spec.absolute_positions, "", dtype, self.device)
        # a part that adds a row chosen by (previous token, token): its state (the previous token of every request) lives in
        # a cache layer of its own, above every layer's
        self.pair_embedding = None
        self.pair_cache_layer = max([len(spec.layers)] + [s.resolved_cache_layer() + 1 for s in spec.schedule])
        if spec.pair_embedding is not None:
            self.pair_embedding = build_part("embedding", spec.pair_embedding, "", dtype, self.device)
        self.embedding: torch.Tensor | None = None
        self.head: Linear | None = None

    # ---- what the cache manager needs to know -------------------------------------------
    def cache_needs(self) -> dict[int, PagedKVNeed | SlotStateNeed]:
        """Per cache layer (a layer some schedule entry writes): what its mixer keeps."""
        needs: dict[int, PagedKVNeed | SlotStateNeed] = {}
        for step in self.spec.schedule:
            need = self.blocks[step.layer].mixer.cache_need()
            if need is None:
                continue
            cache_layer = step.resolved_cache_layer()
            if step.write_cache:
                needs[cache_layer] = need
            elif needs.get(cache_layer) != need:
                raise ValueError(
                    f"layer {step.layer} reads cache layer {cache_layer}, whose contents have another shape"
                )
        if self.pair_embedding is not None:
            needs[self.pair_cache_layer] = self.pair_embedding.cache_need()
        return needs

    def graph_safe(self) -> bool:
        """Whether a step of this model may be captured in a CUDA graph."""
        return (all(block.graph_safe for block in self.blocks) and self.final_norm.graph_safe
                and (self.absolute_positions is None or self.absolute_positions.graph_safe)
                and (self.pair_embedding is None or self.pair_embedding.graph_safe))

    def graph_safe_portions(self) -> bool:
        """Whether a step of this model that holds prompt portions may be captured in a CUDA graph."""
        return all(part.graph_safe_portions for part in self.all_parts())

    def all_parts(self):
        """Every part of every block, and the final norm."""
        for block in self.blocks:
            yield from block.parts()
        yield self.final_norm
        if self.absolute_positions is not None:
            yield self.absolute_positions
        if self.pair_embedding is not None:
            yield self.pair_embedding

    def step_scalars(self) -> dict:
        """The per-step device scalars that the model's parts declare (``Part.step_scalars``), by name."""
        scalars: dict = {}
        for part in self.all_parts():
            for name, rule in part.step_scalars().items():
                scalars.setdefault(name, rule)
        return scalars

    def step_arrays(self, max_tokens: int, max_seqs: int, page_size: int, max_portions: int | None = None,
                    max_ctx: int | None = None) -> dict:
        """The per-step device arrays that the model's parts declare (``Part.step_arrays``), by key."""
        arrays: dict = {}
        for part in self.all_parts():
            for key, decl in part.step_arrays(max_tokens, max_seqs, page_size, max_portions, max_ctx).items():
                arrays.setdefault(key, decl)
        return arrays

    def reserve_for_steps(self, max_seqs: int, max_ctx: int) -> None:
        for part in self.all_parts():
            part.reserve_for_steps(max_seqs, max_ctx)

    # ---- weights ---------------------------------------------------------------------------
    def tensor_decls(self) -> list[TensorDecl]:
        spec = self.spec
        decls = [TensorDecl(spec.embedding_name, (spec.vocab_size, spec.hidden_size), "table", "embedding")]
        if self.pair_embedding is not None:
            decls.extend(self.pair_embedding.tensor_decls())
        for block in self.blocks:
            decls.extend(block.tensor_decls())
        decls.extend(self.final_norm.tensor_decls())
        # a tied model's checkpoint may omit the head (clockwork/engine/loader.py:57-62)
        decls.append(TensorDecl(spec.head_name, (spec.vocab_size, spec.hidden_size), "matrix", "linear",
                                optional=spec.tie_word_embeddings))
        return decls

    def load_weights(self, fetch) -> None:
        self.embedding = fetch(self.spec.embedding_name)
        if self.pair_embedding is not None:
            self.pair_embedding.load_weights(fetch)
        for block in self.blocks:
            block.load_weights(fetch)
        self.final_norm.load_weights(fetch)
        self.head = Linear(self.embedding if self.spec.tie_word_embeddings else fetch(self.spec.head_name))

    def weight_bytes(self) -> int:
        """Bytes of distinct weight storage a step reads when every weight is used once."""
        seen: dict[int, int] = {}

        def visit(obj) -> None:
            if isinstance(obj, torch.Tensor):
                seen[obj.data_ptr()] = obj.numel() * obj.element_size()
            elif isinstance(obj, Linear):
                visit(obj.weight)
                visit(obj.bias)
            elif isinstance(obj, (list, tuple)):
                for o in obj:
                    visit(o)
            elif hasattr(obj, "__dict__") and not isinstance(obj, (ModelSpec, torch.dtype, torch.device)):
                for key, value in vars(obj).items():
                    if key in ("spec", "layer"):
                        continue
                    visit(value)

        visit(self.blocks)
        visit(self.pair_embedding)
        visit(self.final_norm)
        visit(self.head)
        return sum(seen.values())

    # ---- one step --------------------------------------------------------------------------
    def forward(self, ctx: StepContext, token_ids: torch.Tensor, logit_rows: torch.Tensor | None) -> torch.Tensor | None:
        """token_ids int32 [N]; logit_rows int32 [R] (rows of the flat batch whose logits are
        wanted).  Returns float32 [R, vocab], or None when no row is wanted."""
        # (kernels of a step read its inputs before they wait for their predecessors; when a kernel has
        # only just written those inputs, the first kernel here must not start before it has finished)
        # (a position part multiplies the rows by the embedding's scale itself; without one the gather does)
        scale = 1.0 if self.absolute_positions is not None else self.spec.embedding_scale
        schedule = self.spec.schedule
        planes = None
        if self.spec.keeps_layer_outputs:
            # the input rows and what every layer run leaves, a plane each: the embedding is gathered into plane 0
            planes = torch.empty((len(schedule) + 1, token_ids.shape[0], self.spec.hidden_size), dtype=torch.float32, device=self.device)
        stream = ResidualStream(ops.embed(self.embedding, token_ids, ctx.status, serial=ctx.inputs_from_device, scale=scale,
                                          out=None if planes is None else planes[0]))
        stream.layer_outputs = planes
        if self.absolute_positions is not None:
            self.absolute_positions.add_to_embedding(stream.residual, ctx.positions, self.spec.embedding_scale)
        if self.pair_embedding is not None:
            self.pair_embedding.add_to_embedding(ctx, stream.residual, token_ids, ctx.views[self.pair_cache_layer])
        input_rows = None
        if any(step.add_input for step in schedule):
            input_rows = torch.empty_like(stream.residual).copy_(stream.residual)  # (a device-to-device copy)
        for i, step in enumerate(schedule):
            if step.add_input:
                self._add_input(stream, input_rows, self.blocks[step.layer].first_norm())
            view = ctx.views.get(step.resolved_cache_layer())
            if view is not None and hasattr(view, "write"):
                view.write = step.write_cache
            block = self.blocks[step.layer]
            # the norm that reads the residual next, for blocks that can fuse its first half into their
            # last product (the final norm reads selected rows only and is left alone)
            # (input rows added in between come before that norm: a product must not begin it)
            following = None
            if i + 1 < len(schedule) and not schedule[i + 1].add_input:
                following = self.blocks[schedule[i + 1].layer].first_norm()
            if following is not None:
                block.forward(ctx, stream, view, following_norm=following)
            else:
                block.forward(ctx, stream, view)
        if logit_rows is None or logit_rows.numel() == 0:
            stream.flush()
            return None
        x = self.final_norm.forward_rows(stream, logit_rows, ctx.status)
        logits = self.head.to_float32(x)
        if self.spec.logit_softcap is not None or self.spec.logit_scale != 1.0:
            ops.softcap_(logits, self.spec.logit_softcap, self.spec.logit_scale)
        return logits

    @staticmethod
    def _add_input(stream: ResidualStream, rows: torch.Tensor, norm) -> None:
        """``residual += rows`` (float32): inside the kernel of the norm that reads the residual next, when that norm takes
        slabs and the width suits the kernel that adds them up."""
        n, w = rows.shape
        if getattr(norm, "takes_partial_sums", False) and w % 4 == 0 and w <= 4096:
            stream.push(ops.PartialSums(rows.view(1, n, w), n))
        else:
            ops.add_to_residual(stream.residual_after_flush(), rows)


def tensor_decls_for_spec(spec: ModelSpec) -> list[TensorDecl]:
    """Declarations without building anything on a GPU (parts are built on the meta-free CPU
    path: no tensor is allocated until weights load)."""
    return DecoderModel(spec, torch.float32, "cpu").tensor_decls()


def build_model(spec: ModelSpec, dtype: torch.dtype, device) -> DecoderModel:
    return DecoderModel(spec, dtype, device)
