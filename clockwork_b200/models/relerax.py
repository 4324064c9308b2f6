"""Relerax: a decoder whose layers are listed one by one in ``config.json``; in every layer mixer and feed-forward read the
same residual, each through a norm of its own.

``config.json`` keys: ``architecture`` ("Relerax"), ``vocab``, ``width``, ``norm.eps`` and ``layers``, a list of ``{"type",
"mixer", "mlp"}``.  ``type`` names the mixer:

* ``attention`` (``heads, kv_heads, dim, vdim, scale, mask.size, rot.dims, rot.base, rot.scaling``): softmax attention over a
  sliding window of ``mask.size`` positions whose values are its keys before the rotation (``vdim`` = ``dim``, no value
  product); rotary positions on the leading ``rot.dims`` entries of every query and key head (neighbouring entries form a
  pair), stretched by ``rot.scaling`` (``factor, original, fast, slow``; absent or null: not); one added to the softmax's
  denominator; an output gate per entry.
* ``latent_attention`` (``heads, dim, rot_dim, vdim, kv_rank, scale, rot.base, rot.scaling``): causal attention over a cached
  latent and one rotated key part shared by the heads, the same rotation; an output gate per head.

``mlp`` is ``null``, ``{"kind": "dense", "ff"}`` (two products with biases, the square of relu between them) or ``{"kind":
"moe", "expert": {"ff"}, "router": {"experts", "top", "identity"}}``: routed experts of the same form without biases; the
last ``identity`` of the router's ``experts + identity`` outputs (absent or 0: none) stand for experts that hand their input
on; scores are the softmax over all outputs, experts are ranked with a correction each and weighted by the chosen ones'
scores, which are made to sum to one.  Tensor names: ``embed``, ``l<i>.norm1|norm2``, ``l<i>.mix.*``, ``l<i>.mlp.up|up.b|down|
down.b``, ``l<i>.mlp.e<j>.up|down``, ``l<i>.mlp.router|correction``, ``final.norm``, ``head``.  Nothing here fixes a size.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any

from ..config.model_spec import LayerSpec, ModelSpec, PartSpec, sequential_schedule
from ..config.registry import register_architecture
from .rapitar import _need

LAYER_TYPES = ("attention", "latent_attention")


@dataclass(frozen=True)
class ReleraxConfig:
    vocab: int
    width: int
    eps: float
    layers: tuple  # of (mixer PartSpec, feed-forward PartSpec)
    raw: dict


def _layers_2k(repeats: int) -> list:
    """Layer sizes of a model of 2,048 width: latent attention of 16 heads over a latent of 512 + 64, windowed attention of 16
    heads of 128 on 4 key/value heads over 1,024 positions, half of every head rotated; dense feed-forwards of 3.5 widths and
    64 experts of 1,408 (and 4 that hand their input on) of which 6 are chosen."""
    scaling = {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}
    dense = {"kind": "dense", "ff": 7168}
    moe = {"kind": "moe", "expert": {"ff": 1408}, "router": {"experts": 64, "top": 6, "identity": 4}}
    latent = {"heads": 16, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "scale": 192 ** -0.5,
              "rot": {"base": 10000.0, "dims": 64, "scaling": scaling}}
    window = {"heads": 16, "kv_heads": 4, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": 1024},
              "rot": {"base": 10000.0, "dims": 64, "scaling": scaling}}
    return [{"type": "latent_attention", "mixer": latent, "mlp": dense}, {"type": "attention", "mixer": window, "mlp": moe},
            {"type": "latent_attention", "mixer": latent, "mlp": moe}, {"type": "attention", "mixer": window, "mlp": dense}] * repeats


class ReleraxArchitecture:
    name = "Relerax"
    layer_count_key = None  # the layers are a list: a shape with fewer layers is another list
    named_shapes = {
        "relerax-2k": {"architecture": "Relerax", "vocab": 32768, "width": 2048, "norm": {"eps": 1e-6}, "layers": _layers_2k(2)},
        "relerax-tiny": {"architecture": "Relerax", "vocab": 256, "width": 64, "norm": {"eps": 1e-5}, "layers": [
            {"type": "attention", "mlp": {"kind": "moe", "expert": {"ff": 32}, "router": {"experts": 5, "top": 2, "identity": 1}},
             "mixer": {"heads": 4, "kv_heads": 2, "dim": 16, "vdim": 16, "scale": 0.3, "mask": {"size": 20}, "rot": {
                 "dims": 8, "base": 1000.0, "scaling": {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}}}},
            {"type": "latent_attention", "mlp": {"kind": "dense", "ff": 96},
             "mixer": {"heads": 4, "dim": 16, "rot_dim": 8, "vdim": 24, "kv_rank": 40, "scale": 0.25, "rot": {"dims": 8, "base": 500.0}}},
            {"type": "attention", "mlp": None,
             "mixer": {"heads": 2, "kv_heads": 1, "dim": 24, "vdim": 24, "scale": 0.2, "mask": {"size": 50}, "rot": {
                 "dims": 24, "base": 10000.0}}}]},
    }

    @staticmethod
    def _rotary(m: dict[str, Any], where: str) -> dict:
        rot = m.get("rot") or {}
        scaling = rot.get("scaling")
        if scaling is not None:
            scaling = {k: _need(scaling, k, where + ".rot.scaling", float) for k in ("factor", "original", "fast", "slow")}
        return {"dims": _need(rot, "dims", where + ".rot"), "base": _need(rot, "base", where + ".rot", float),
                "pairing": "interleaved", "scaling": scaling}

    @classmethod
    def _mixer(cls, kind: str, m: dict[str, Any], width: int, eps: float, where: str) -> PartSpec:
        if kind not in LAYER_TYPES:
            raise ValueError(f"config.json: {where}: unknown layer type {kind!r}; known: {list(LAYER_TYPES)}")
        rotary = cls._rotary(m, where)
        common = dict(hidden_size=width, heads=_need(m, "heads", where), dim=_need(m, "dim", where), vdim=_need(m, "vdim", where),
                      scale=_need(m, "scale", where, float))
        if kind == "attention":
            if common["vdim"] != common["dim"]:
                raise ValueError(f"config.json: {where}: the values are the keys, but vdim {common['vdim']} differs from dim {common['dim']}")
            return PartSpec("window_attention", dict(
                common, kv_heads=_need(m, "kv_heads", where), window=_need(m.get("mask") or {}, "size", where + ".mask"),
                weights="softmax", sink="zero", values="keys", gate="entry", rotary=rotary))
        rot_dim = _need(m, "rot_dim", where)
        if rotary["dims"] != rot_dim:
            raise ValueError(f"config.json: {where}: rot.dims {rotary['dims']} differs from rot_dim {rot_dim}")
        return PartSpec("latent_attention", dict(
            common, rot_dim=rot_dim, kv_rank=_need(m, "kv_rank", where), q_rank=None, sink=False, gate="head",
            rope_base=rotary["base"], pairing=rotary["pairing"], scaling=rotary["scaling"], eps=eps))

    @staticmethod
    def _ffn(f, width: int, where: str) -> PartSpec:
        if f is None:
            return PartSpec("none", {})
        kind = f.get("kind")
        if kind == "dense":
            return PartSpec("relu2_mlp", dict(hidden_size=width, intermediate_size=_need(f, "ff", where), bias=True))
        if kind == "moe":
            router = f.get("router") or {}
            identity = router.get("identity") or 0
            if isinstance(identity, bool) or not isinstance(identity, int) or identity < 0:
                raise ValueError(f"config.json: {where}.router.identity must be a non-negative integer, got {identity!r}")
            return PartSpec("moe", dict(hidden_size=width, expert_size=_need(f.get("expert") or {}, "ff", where + ".expert"),
                                        experts=_need(router, "experts", where + ".router"), top=_need(router, "top", where + ".router"),
                                        identity=identity, gated=False, scoring="all", correction=True, renormalize=True,
                                        router_bias=False))
        raise ValueError(f"config.json: {where}: unknown feed-forward kind {kind!r}")

    def parse_config(self, raw: dict[str, Any]) -> ReleraxConfig:
        width = _need(raw, "width", "the model")
        eps = _need(raw.get("norm") or {}, "eps", "norm", float)
        listed = raw.get("layers")
        if not isinstance(listed, list) or not listed:
            raise ValueError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, entry in enumerate(listed):
            where = f"layers[{i}]"
            layers.append((self._mixer(entry.get("type"), entry.get("mixer") or {}, width, eps, where + ".mixer"),
                           self._ffn(entry.get("mlp"), width, where + ".mlp")))
        return ReleraxConfig(_need(raw, "vocab", "the model"), width, eps, tuple(layers), dict(raw))

    def model_spec(self, config: ReleraxConfig) -> ModelSpec:
        norm = PartSpec("rmsnorm", {"size": config.width, "eps": config.eps, "weight_suffix": ""})
        layers = [LayerSpec(block="parallel_residual_two_norms", mixer=mixer, ffn=ffn, mixer_norm=norm, ffn_norm=norm, prefix=f"l{i}")
                  for i, (mixer, ffn) in enumerate(config.layers)]
        return ModelSpec(architecture=self.name, vocab_size=config.vocab, hidden_size=config.width, layers=layers,
                         schedule=sequential_schedule(len(layers)), final_norm=norm, embedding_name="embed",
                         final_norm_prefix="final.norm", head_name="head", tie_word_embeddings=False, raw=config.raw)


register_architecture(ReleraxArchitecture(), replace=True)
