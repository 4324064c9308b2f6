"""Parallel residual blocks: mixer and feed-forward read the same residual.

``parallel_residual``: a single norm feeds both, ``n = norm(h); h += mixer(n) + ffn(n)``.
``parallel_residual_two_norms``: each has a norm of its own, ``h += mixer(norm1(h)) + ffn(norm2(h))``; one kernel makes both
norms in one pass over the rows, and what of the feed-forward does not touch the residual (``FeedForward.begin``) runs on a
second stream beside the mixer, joined before its last product (or the experts' weighted sum) adds into the residual.

Tensor prefixes: ``<layer>.norm1`` (and ``<layer>.norm2``), ``<layer>.mix``, ``<layer>.mlp``.  A layer without a feed-forward
names the kind ``none`` (and has no second norm).  The sublayers' output
products add into the float32 residual in their epilogues, the mixer first, so the sum is
``(h + mixer) + ffn`` in float32 whatever the run precision.
"""

from __future__ import annotations

import torch

from ..config.model_spec import LayerSpec
from ..ops.library import serial_launch
from ..weights.decl import TensorDecl
from .base import Block, Norm, ResidualStream, StepContext
from .registry import build_part, register_block
from .side_by_side import side_stream


class ParallelResidualBlock(Block):
    def __init__(self, layer: LayerSpec, dtype, device) -> None:
        self.layer = layer
        self.prefix = layer.prefix
        self.dtype, self.device = dtype, device
        self.norm = build_part("norm", layer.mixer_norm, f"{layer.prefix}.norm1", dtype, device)
        self.mixer = build_part("mixer", layer.mixer, f"{layer.prefix}.mix", dtype, device)
        self.ffn = None if layer.ffn.kind == "none" else build_part("ffn", layer.ffn, f"{layer.prefix}.mlp", dtype, device)

    def parts(self):
        return (self.norm, self.mixer) + (() if self.ffn is None else (self.ffn,))

    @property
    def graph_safe(self) -> bool:
        return all(part.graph_safe for part in self.parts())

    def tensor_decls(self):
        for part in self.parts():
            yield from part.tensor_decls()

    def load_weights(self, fetch) -> None:
        for part in self.parts():
            part.load_weights(fetch)

    def first_norm(self):
        return self.norm

    def forward(self, ctx: StepContext, stream: ResidualStream, view, following_norm=None) -> None:
        x = self.norm.forward(stream, ctx.status)  # a plain tensor: two sublayers read it
        stream.next_norm = None if self.ffn is not None else following_norm
        stream.push(self.mixer.forward(ctx, x, view, stream))
        if self.ffn is not None:
            stream.next_norm = following_norm  # what the feed-forward's last product may begin or leave in parts
            stream.push(self.ffn.forward(ctx, x, stream))
        stream.next_norm = None


class NormPair(Norm):
    """Two norms of the same rows as one part: ``forward`` returns both.  (It takes the slabs of a product whose splits are
    kept apart like either of them, but no product can begin it: it has two weights.)"""

    graph_safe = True
    graph_safe_portions = True
    takes_partial_sums = True

    def __init__(self, first: Norm, second: Norm) -> None:
        self.first, self.second = first, second

    def tensor_decls(self):
        yield from self.first.tensor_decls()
        yield from self.second.tensor_decls()

    def load_weights(self, fetch) -> None:
        self.first.load_weights(fetch)
        self.second.load_weights(fetch)

    def forward(self, stream: ResidualStream, status, lazy: bool = False):
        return self.first.forward_with(self.second, stream, status)


class TwoNormParallelBlock(ParallelResidualBlock):
    concurrent = True  # the feed-forward on a second stream beside the mixer

    def __init__(self, layer: LayerSpec, dtype, device) -> None:
        super().__init__(layer, dtype, device)
        if self.ffn is not None:
            second = build_part("norm", layer.ffn_norm, f"{layer.prefix}.norm2", dtype, device)
            for norm in (self.norm, second):
                if not hasattr(norm, "forward_with"):
                    raise ValueError(f"norm kind {norm.spec.kind!r} cannot share a pass with another")
            self.norm = NormPair(self.norm, second)
        self._forked = self._joined = None  # events of the fork and the join (made at first use)

    def tensor_decls(self):
        yield from super().tensor_decls()
        if self.ffn is None:  # (a checkpoint may hold the second norm all the same; nothing reads it)
            yield TensorDecl(f"{self.prefix}.norm2", (int(self.layer.ffn_norm["size"]),), "vector", "norm", optional=True)

    def forward(self, ctx: StepContext, stream: ResidualStream, view, following_norm=None) -> None:
        if self.ffn is None:
            super().forward(ctx, stream, view, following_norm)
            return
        x, y = self.norm.forward(stream, ctx.status)
        stream.next_norm = None
        if not (self.concurrent and y.is_cuda and self.ffn.in_two_pieces):
            stream.push(self.mixer.forward(ctx, x, view, stream))
            stream.next_norm = following_norm
            stream.push(self.ffn.forward(ctx, y, stream))
            stream.next_norm = None
            return
        if self._forked is None:
            self._forked, self._joined = torch.cuda.Event(), torch.cuda.Event()
        main, side = torch.cuda.current_stream(y.device), side_stream(y.device)
        self._forked.record(main)
        side.wait_event(self._forked)  # the norms are ready (and everything the step's stream did before)
        with torch.cuda.stream(side):
            begun = self.ffn.begin(ctx, y)
            self._joined.record(side)
        stream.push(self.mixer.forward(ctx, x, view, stream))
        stream.flush()
        main.wait_event(self._joined)
        stream.next_norm = following_norm
        with serial_launch():  # (what reads the second stream's results starts when both streams have got here)
            stream.push(self.ffn.finish(ctx, y, begun, stream))
        stream.next_norm = None


register_block("parallel_residual", ParallelResidualBlock, replace=True)
register_block("parallel_residual_two_norms", TwoNormParallelBlock, replace=True)
