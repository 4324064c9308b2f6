"""Attention that caches a latent instead of keys and values.

Parameters: ``hidden_size, heads, dim, rot_dim, vdim, kv_rank, scale, rope_base, eps``, and the switches

* ``q_rank``: queries go through a normed latent of their own (None: straight from the input);
* ``sink``: the softmax denominator also holds ``exp(sink_h)``, a learned logit per head (by default it does; False: not);
* ``gate``: ``"entry"`` (the default): the heads' outputs are multiplied by ``sigmoid(g x)`` entry by entry; ``"head"``: head
  h's output by ``sigmoid(g x)_h``;
* ``pairing`` (``"half"`` by default, ``"interleaved"``) and ``scaling`` of the rotation, as in ``rotary.check_rotary``.

Tensors: with ``q_rank`` ``dq`` [q_rank, H], ``dq.norm`` [q_rank], ``uq`` [heads*(dim+rot_dim), q_rank], else ``q``
[heads*(dim+rot_dim), H]; ``dkv`` [kv_rank+rot_dim, H], ``dkv.norm`` [kv_rank], ``uk`` [heads*dim, kv_rank], ``uv`` [heads*vdim,
kv_rank], ``sink`` [heads], ``g`` [heads*vdim or heads, H], ``o`` [H, heads*vdim].

Queries: ``q = uq (rmsnorm(dq x) * dq.norm)`` or ``q x``, per head ``[dim plain | rot_dim rotated]``.
Keys and values: the first kv_rank rows of ``dkv x``, RMS-normed with ``dkv.norm``, are the latent c;
the last rot_dim are one rotated key part shared by all heads (angle ``p * base^(-2i/rot_dim)`` without ``scaling``).
Per head the plain key is ``uk c`` and the value ``uv c``; the score is
``(q_plain . k_plain + q_rot . k_rot) * scale``, causal.  The gated outputs go through ``o``.

Only ``[c | k_rot]`` is cached (one row of kv_rank + rot_dim numbers per token, one plane of pages).
The per-head products are moved to the query side: the query row of a head is ``[uk_h^T q_plain | q_rot]``
and the kernel returns ``sum_j p_j c_j`` per head, which ``uv_h`` then maps to the head's value
(``csrc/latent_attention.cu``).  Without ``q_rank`` one product with float32 output yields ``[q | dkv | head gates]``.
"""

from __future__ import annotations

import torch

from .. import ops
from ..ops import grouped as grouped_ops
from ..ops import latent as latent_ops
from ..weights.decl import TensorDecl
from .base import Mixer, PagedKVNeed, PagedView, ResidualStream, StepContext
from .linear import Linear
from .registry import register_mixer
from .rotary import check_rotary, rotary_tables

GATES = ("entry", "head")


class LatentAttention(Mixer):
    graph_safe = True
    graph_safe_portions = True

    def __init__(self, spec, prefix, dtype, device) -> None:
        super().__init__(spec, prefix, dtype, device)
        p = spec.params
        self.hidden_size = int(p["hidden_size"])
        self.heads, self.dim, self.rot, self.vdim = int(p["heads"]), int(p["dim"]), int(p["rot_dim"]), int(p["vdim"])
        self.kv_rank = int(p["kv_rank"])
        self.q_rank = None if p.get("q_rank") is None else int(p["q_rank"])
        self.scale, self.eps, self.base = float(p["scale"]), float(p["eps"]), float(p["rope_base"])
        self.has_sink = bool(p.get("sink", True))
        self.gate_kind = str(p.get("gate", "entry"))
        if self.gate_kind not in GATES:
            raise ValueError(f"gate must be one of {GATES}, got {self.gate_kind!r}")
        if self.rot % 2:
            raise ValueError(f"rot_dim {self.rot} must be even")
        self.interleaved, self.amplitude = False, 1.0
        inv_freq = torch.zeros(1)
        if self.rot:
            rotary = {"dims": self.rot, "base": self.base, "pairing": p.get("pairing", "half"), "scaling": p.get("scaling")}
            _, _, self.interleaved = check_rotary(rotary, self.rot)
            inv_freq, self.amplitude = rotary_tables(self.rot, self.base, rotary["scaling"])
        self.inv_freq = inv_freq.to(device)
        self.q_width = self.heads * (self.dim + self.rot)
        self.sink = self.gate = None

    def cache_need(self) -> PagedKVNeed:
        return PagedKVNeed(1, self.kv_rank + self.rot, None, planes=1)

    def reserve_for_steps(self, max_seqs: int, max_ctx: int) -> None:
        if self.device.type == "cuda" and self.dtype == torch.bfloat16:
            latent_ops.reserve_scratch(self.device, self.kv_rank, self.rot)

    def tensor_decls(self):
        h, heads = self.hidden_size, self.heads
        if self.q_rank is not None:
            yield TensorDecl(self.name("dq"), (self.q_rank, h), "matrix", "linear")
            yield TensorDecl(self.name("dq.norm"), (self.q_rank,), "vector", "norm")
            yield TensorDecl(self.name("uq"), (self.q_width, self.q_rank), "matrix", "linear")
        else:
            yield TensorDecl(self.name("q"), (self.q_width, h), "matrix", "linear")
        yield TensorDecl(self.name("dkv"), (self.kv_rank + self.rot, h), "matrix", "linear")
        yield TensorDecl(self.name("dkv.norm"), (self.kv_rank,), "vector", "norm")
        yield TensorDecl(self.name("uk"), (heads * self.dim, self.kv_rank), "matrix", "linear")
        yield TensorDecl(self.name("uv"), (heads * self.vdim, self.kv_rank), "matrix", "linear")
        if self.has_sink:
            yield TensorDecl(self.name("sink"), (heads,), "vector", "bias")
        yield TensorDecl(self.name("g"), (heads * self.vdim if self.gate_kind == "entry" else heads, h), "matrix", "linear")
        yield TensorDecl(self.name("o"), (h, heads * self.vdim), "matrix", "linear")

    def load_weights(self, fetch) -> None:
        dkv, g = fetch(self.name("dkv")), fetch(self.name("g"))
        if self.q_rank is not None:
            self.dq, self.uq, self.dkv = Linear(fetch(self.name("dq"))), Linear(fetch(self.name("uq"))), Linear(dkv)
            self.dq_norm = fetch(self.name("dq.norm"))
            self.gate = Linear(g)
        else:
            rows = [fetch(self.name("q")), dkv] + ([g] if self.gate_kind == "head" else [])
            odd = -sum(t.shape[0] for t in rows) % 8  # (rows of zeros, so that the product's rows are whole 16-byte pieces)
            self.joint = Linear(torch.cat(rows + [dkv.new_zeros(odd, self.hidden_size)], dim=0).contiguous())
            self.gate = Linear(g) if self.gate_kind == "entry" else None
        self.dkv_norm = fetch(self.name("dkv.norm"))
        # per head [kv_rank, dim]: the key product's transpose, applied to the query instead of the latent
        self.uk_t = fetch(self.name("uk")).view(self.heads, self.dim, self.kv_rank).transpose(1, 2).contiguous()
        self.uv = fetch(self.name("uv")).view(self.heads, self.vdim, self.kv_rank).contiguous()
        self.sink = fetch(self.name("sink")) if self.has_sink else None
        self.o = Linear(fetch(self.name("o")))

    def _attend(self, ctx: StepContext, x, view: PagedView) -> torch.Tensor:
        n, heads, rank, rot = x.shape[0], self.heads, self.kv_rank, self.rot
        q_plain = head_gate = None
        if self.q_rank is not None:
            c_q = ops.add_rmsnorm(self.dq.to_float32(x), None, self.dq_norm, self.eps, self.dtype, ctx.status)
            q = self.uq(c_q)                      # [N, heads*(dim+rot)]
            down = self.dkv.to_float32(x)         # [N, kv_rank+rot], float32: the latent is normed from it
            if self.gate_kind == "head":
                head_gate = self.gate.to_float32(x)
        else:
            q = self.joint.to_float32(x)          # [N, heads*(dim+rot) | kv_rank+rot | heads], float32: rounded once, when turned
            down = q[:, self.q_width :]
            q_plain = torch.empty((n, heads * self.dim), dtype=self.dtype, device=x.device)
            if self.gate_kind == "head":
                head_gate = down[:, rank + rot :]
        qa = torch.empty((n, heads * (rank + rot)), dtype=self.dtype, device=x.device)
        latent_ops.latent_prepare(down, q, qa, view, self.dkv_norm, self.inv_freq, ctx.positions, heads, self.dim, rot, rank,
                                  self.eps, ctx.status, self.interleaved, self.amplitude, q_plain)
        if q_plain is not None:
            grouped_ops.per_head_product(q_plain, self.dim, self.uk_t, qa, rank + rot)
        else:
            grouped_ops.per_head_product(q, self.dim + rot, self.uk_t, qa, rank + rot)
        mixed = latent_ops.latent_attention(qa, view, ctx, self.sink, heads, rank, rot, self.scale)  # [N, heads*rank]
        out = torch.empty((n, heads * self.vdim), dtype=self.dtype, device=x.device)
        grouped_ops.per_head_product(mixed, rank, self.uv, out, self.vdim,
                                     gate=self.gate(x) if self.gate_kind == "entry" else None, head_gate=head_gate)
        return out

    def mix(self, ctx: StepContext, x, view: PagedView) -> torch.Tensor:
        return self.o.to_float32(self._attend(ctx, x, view))

    def forward(self, ctx: StepContext, x, view: PagedView, stream: ResidualStream):
        return self.o.add_or_defer(self._attend(ctx, x, view), stream)


register_mixer("latent_attention", LatentAttention, replace=True)
