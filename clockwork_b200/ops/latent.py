"""Python faces of the kernels for attention over a cached latent (``csrc/latent_attention.cu``)."""

from __future__ import annotations

import torch

from . import _need, _ptr, _stream, dtype_code
from .library import check, library


def set_tensor_cores(on: bool) -> None:
    """bfloat16 attention over the latent runs on the tensor cores when its sizes allow (the default); ``False`` keeps
    it on the CUDA-core kernel that float32 runs use (for comparisons)."""
    library().cw_latent_attention_set_mma(1 if on else 0)


def latent_prepare(down: torch.Tensor, q: torch.Tensor, qa: torch.Tensor, view, norm_weight: torch.Tensor,
                   inv_freq: torch.Tensor, positions: torch.Tensor, heads: int, dim: int, rot: int, rank: int, eps: float,
                   status: torch.Tensor, interleaved: bool = False, amplitude: float = 1.0,
                   q_plain: torch.Tensor | None = None) -> None:
    """Writes each token's cache row [normed latent | rotated shared key part] at its slot and the rotated
    parts of the queries into ``qa`` [N, heads*(rank+rot)] at [.., rank:] of every head; with ``q_plain`` [N, heads*dim] the
    queries' plain parts go there.  ``down`` float32 [N, >= rank+rot] and ``q`` [N, >= heads*(dim+rot)] (float32 or ``qa``'s
    dtype) may be column slices of one product's rows.  Entry i of a rotated part pairs with entry i + rot/2, or
    (``interleaved``) entry 2i with entry 2i + 1; sines and cosines are multiplied by ``amplitude``."""
    for name, t, width in (("down", down, rank + rot), ("q", q, heads * (dim + rot))):
        if t.dim() != 2 or t.stride(1) != 1 or t.shape[1] < width:
            raise ValueError(f"{name} must be [N, >= {width}] with unit column stride")
    _need(qa, None, "qa", 2)
    cache = view.k_cache
    _need(cache, qa.dtype, "cache", 4)
    _need(inv_freq, torch.float32, "inv_freq", 1)
    n = q.shape[0]
    if down.dtype != torch.float32 or q.dtype not in (torch.float32, qa.dtype):
        raise ValueError("down must be float32, q float32 or of the run's dtype")
    if down.shape[0] != n or tuple(qa.shape) != (n, heads * (rank + rot)) or (rot and inv_freq.shape[0] * 2 != rot):
        raise ValueError("widths do not match the head count and sizes")
    if q_plain is not None:
        _need(q_plain, qa.dtype, "q_plain", 2)
        if tuple(q_plain.shape) != (n, heads * dim):
            raise ValueError(f"q_plain {tuple(q_plain.shape)} is not [{n}, {heads * dim}]")
    if cache.shape[2] * cache.shape[3] != rank + rot:
        raise ValueError("cache rows do not hold rank + rot numbers")
    write = bool(view.write)
    ld = lambda t: t.stride(0) if n > 1 else max(t.stride(0), t.shape[1])  # noqa: E731
    check(library().cw_latent_prepare(_ptr(down), ld(down), _ptr(q), ld(q), 1 if q.dtype == torch.float32 else 0, _ptr(q_plain), _ptr(qa),
                                      _ptr(cache), _ptr(norm_weight), _ptr(inv_freq), 1 if interleaved else 0, float(amplitude),
                                      _ptr(positions), _ptr(view.slots), n, heads, dim, rot, rank, cache.shape[0] * cache.shape[1],
                                      float(eps), 1 if write else 0, dtype_code(qa.dtype), _ptr(status), _stream()), "latent_prepare")


MAX_PARTS = 128  # runs that a row's keys may be cut in
TILE_ROWS = (16, 64)   # (token, head) rows per thread block: single tokens, portions
FILL_BLOCKS = 148      # keys are cut until a step has about so many thread blocks (one to an SM)
_scratch: dict[tuple, torch.Tensor] = {}  # (device index, rank) -> the partial sums of cut rows


def _partial_sums(device, rank: int) -> torch.Tensor:
    """Room for every step whose keys ``plan_parts`` cuts; made once and never replaced (captured steps point at it)."""
    key = (torch.device(device).index or 0, rank)
    have = _scratch.get(key)
    if have is None:
        have = _scratch[key] = torch.empty(FILL_BLOCKS * TILE_ROWS[1] * (rank + 2), dtype=torch.float32, device=device)
    return have


def reserve_scratch(device, rank: int, rot: int) -> None:
    if library().cw_latent_attention_on_tensor_cores(rank, rot):
        _partial_sums(device, rank)


def plan_parts(tokens: int, seqs: int, heads: int, longest_portion: int, longest_context: int) -> tuple[bool, int]:
    """(whether the step runs in tiles of few rows, in how many runs the keys of a row are cut): few rows over a long
    context would otherwise leave most of the GPU idle.  What the device sees may be smaller than these bounds; a run
    without keys costs a block that returns at once."""
    few = longest_portion * heads <= 2 * TILE_ROWS[0]
    if few and longest_portion <= 1:
        tiles = seqs * -(-heads // TILE_ROWS[0])
    else:
        tiles = -(-tokens * heads // TILE_ROWS[0 if few else 1]) + seqs
    return few, max(1, min(FILL_BLOCKS // max(1, tiles), -(-longest_context // 64), MAX_PARTS))


def latent_attention(qa: torch.Tensor, view, ctx, sink: torch.Tensor | None, heads: int, rank: int, rot: int,
                     scale: float) -> torch.Tensor:
    """[N, heads*rank]: per head the softmax-weighted sum of the cached latents (with a ``sink``, that in the denominator)."""
    _need(qa, None, "qa", 2)
    _need(ctx.q_start, torch.int32, "q_start", 1)
    cache = view.k_cache
    n = qa.shape[0]
    out = torch.empty((n, heads * rank), dtype=qa.dtype, device=qa.device)
    few, parts, partial = False, 1, None
    if qa.dtype == torch.bfloat16 and library().cw_latent_attention_on_tensor_cores(rank, rot):
        few, parts = plan_parts(n, ctx.num_seqs, heads, ctx.max_q_len, ctx.max_ctx_len)
        partial = _partial_sums(qa.device, rank) if parts > 1 else None
    check(library().cw_latent_attention(_ptr(qa), _ptr(out), _ptr(cache), _ptr(view.block_tables), _ptr(ctx.tok_seq),
                                        _ptr(ctx.positions), _ptr(ctx.q_start), ctx.q_start.shape[0] - 1, _ptr(sink), n, heads, rank, rot,
                                        cache.shape[1], view.block_tables.shape[1], cache.shape[0], float(scale), 1 if few else 0, parts,
                                        _ptr(partial), dtype_code(qa.dtype), _ptr(ctx.status), _stream()), "latent_attention")
    return out
