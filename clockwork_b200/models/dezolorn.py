"""Dezolorn: a decoder whose layers are listed one by one in ``config.json``; a run of them may be looped, and every pass
but the first begins with the embedding rows added to the residual again.

``config.json`` keys: ``architecture`` ("Dezolorn"), ``vocab``, ``width``, ``norm.eps``, ``logit_scale``, ``logit_softcap``
(absent or null: none), ``loop`` (``{"start", "stop", "times"}``: layers start .. stop-1 run ``times`` times in a row with the
same weights, every pass with a cache and state of its own; absent or null: no loop) and ``layers``, a list of ``{"type",
"mixer", "mlp"}``.  ``type`` names the mixer:

* ``attention`` (``heads, kv_heads, dim, vdim, scale, mask.size, mask.keep_first, rot.dims, rot.base, rot.scaling``): softmax
  attention over a sliding window of ``mask.size`` positions that keeps the sequence's first ``mask.keep_first`` positions in
  sight; RMS norms over all queries and over all keys of a token; rotary positions on the leading ``rot.dims`` entries of
  every query and key head (neighbouring entries form a pair), stretched by ``rot.scaling`` (``factor, original, fast, slow``;
  absent or null: not).
* ``retention`` (``heads, dim, vdim, decay, rot.dims, rot.base``): linear attention with one constant decay per head (the list
  ``decay``) and rotary positions (entry i with entry i + dims/2).
* ``delta`` (``heads, kv_heads, dim, vdim, conv``): the gated delta rule with one decay per head and token, short causal
  convolutions on q, k and v.

``mlp`` is ``null`` or ``{"kind": "dense", "ff"}`` (silu(gate) * up, then down).  Every layer is a pre-norm residual block;
its norms are layer norms with a weight and no bias.  The logits are the output product times ``logit_scale``, bent by ``cap
tanh(logits / cap)``.  Tensor names: ``embed``, ``l<i>.norm1|norm2``, ``l<i>.mix.*``, ``l<i>.mlp.gate|up|down``, ``final.norm``,
``head``.  Nothing here fixes a size.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any

from ..config.model_spec import LayerSpec, ModelSpec, PartSpec, looped_schedule
from ..config.registry import register_architecture
from .gamesun import GamesunArchitecture
from .kapolorn import _loop_bounds
from .rapitar import _need

LAYER_TYPES = ("attention", "retention", "delta")


@dataclass(frozen=True)
class DezolornConfig:
    vocab: int
    width: int
    eps: float
    logit_scale: float
    logit_softcap: float | None
    loop: tuple  # (start, stop, times)
    layers: tuple  # of (mixer PartSpec, feed-forward PartSpec)
    raw: dict


def _layers_2k(repeats: int) -> list:
    """Layer sizes of a model of 2,048 width: attention of 16 heads of 128 on 4 key/value heads over windows of 1,024 and the
    first 4 positions; retention and the delta rule with 16 heads of 128 x 128; a feed-forward of 3.5 widths."""
    dense = {"kind": "dense", "ff": 7168}
    attention = {"type": "attention", "mlp": dense, "mixer": {
        "heads": 16, "kv_heads": 4, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": 1024, "keep_first": 4},
        "rot": {"dims": 128, "base": 1000000.0, "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}}
    retention = {"type": "retention", "mlp": dense, "mixer": {
        "heads": 16, "dim": 128, "vdim": 128, "decay": [1.0 - 2.0 ** (-5 - 3 * h / 15) for h in range(16)],
        "rot": {"dims": 128, "base": 10000.0}}}
    delta = {"type": "delta", "mlp": dense, "mixer": {"heads": 16, "kv_heads": 16, "dim": 128, "vdim": 128, "conv": 4}}
    return [attention, retention, attention, delta] * repeats


class DezolornArchitecture:
    name = "Dezolorn"
    layer_count_key = None  # the layers are a list: a shape with fewer layers is another list
    named_shapes = {
        "dezolorn-2k": {"architecture": "Dezolorn", "vocab": 32768, "width": 2048, "norm": {"eps": 1e-5}, "logit_scale": 1.0,
                        "logit_softcap": 30.0, "layers": _layers_2k(2)},
        "dezolorn-tiny": {"architecture": "Dezolorn", "vocab": 256, "width": 64, "norm": {"eps": 1e-5}, "logit_scale": 0.5,
                          "logit_softcap": 20.0, "loop": {"start": 1, "stop": 3, "times": 2}, "layers": [
            {"type": "delta", "mlp": {"kind": "dense", "ff": 96}, "mixer": {"heads": 4, "kv_heads": 2, "dim": 8, "vdim": 16, "conv": 3}},
            {"type": "attention", "mlp": None, "mixer": {
                "heads": 4, "kv_heads": 2, "dim": 16, "vdim": 24, "scale": 0.3, "mask": {"size": 20, "keep_first": 3},
                "rot": {"dims": 8, "base": 1000.0, "scaling": {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}}}},
            {"type": "retention", "mlp": {"kind": "dense", "ff": 80}, "mixer": {
                "heads": 2, "dim": 16, "vdim": 16, "decay": [0.9, 0.99], "rot": {"dims": 16, "base": 500.0}}}]},
    }

    @staticmethod
    def _mixer(kind: str, m: dict[str, Any], width: int, eps: float, where: str) -> PartSpec:
        if kind not in LAYER_TYPES:
            raise ValueError(f"config.json: {where}: unknown layer type {kind!r}; known: {list(LAYER_TYPES)}")
        common = dict(hidden_size=width, heads=_need(m, "heads", where), dim=_need(m, "dim", where), vdim=_need(m, "vdim", where))
        if kind == "delta":
            return PartSpec("head_delta", dict(common, kv_heads=_need(m, "kv_heads", where), conv=_need(m, "conv", where), eps=eps))
        rot = m.get("rot") or {}
        rotary = {"dims": _need(rot, "dims", where + ".rot"), "base": _need(rot, "base", where + ".rot", float)}
        if kind == "retention":
            decay = m.get("decay")
            if not isinstance(decay, list) or len(decay) != common["heads"] or any(isinstance(d, bool) or not isinstance(d, (int, float)) for d in decay):
                raise ValueError(f"config.json: {where}.decay must list one number per head ({common['heads']}), got {decay!r}")
            return PartSpec("retention", dict(common, decay=[float(d) for d in decay], rotary=dict(rotary, pairing="half"), eps=eps))
        scaling = rot.get("scaling")
        if scaling is not None:
            scaling = {k: _need(scaling, k, where + ".rot.scaling", float) for k in ("factor", "original", "fast", "slow")}
        mask = m.get("mask") or {}
        keep = mask.get("keep_first", 0)
        if isinstance(keep, bool) or not isinstance(keep, int) or keep < 0:
            raise ValueError(f"config.json: {where}.mask.keep_first must be a non-negative integer, got {keep!r}")
        return PartSpec("window_attention", dict(
            common, kv_heads=_need(m, "kv_heads", where), scale=_need(m, "scale", where, float), weights="softmax",
            window=_need(mask, "size", where + ".mask"), keep_first=keep, qk_norm=eps,
            rotary=dict(rotary, pairing="interleaved", scaling=scaling)))

    def parse_config(self, raw: dict[str, Any]) -> DezolornConfig:
        width = _need(raw, "width", "the model")
        eps = _need(raw.get("norm") or {}, "eps", "norm", float)
        cap = raw.get("logit_softcap")
        if cap is not None:
            cap = _need(raw, "logit_softcap", "the model", float)
            if not cap > 0:
                raise ValueError(f"config.json: logit_softcap must be positive, got {cap!r}")
        listed = raw.get("layers")
        if not isinstance(listed, list) or not listed:
            raise ValueError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, entry in enumerate(listed):
            where = f"layers[{i}]"
            layers.append((self._mixer(entry.get("type"), entry.get("mixer") or {}, width, eps, where + ".mixer"),
                           GamesunArchitecture._ffn(entry.get("mlp"), width, where + ".mlp")))
        return DezolornConfig(_need(raw, "vocab", "the model"), width, eps, _need(raw, "logit_scale", "the model", float), cap,
                              _loop_bounds(raw.get("loop"), len(layers)), tuple(layers), dict(raw))

    def model_spec(self, config: DezolornConfig) -> ModelSpec:
        norm = PartSpec("layernorm", {"size": config.width, "eps": config.eps, "weight_suffix": ""})
        layers = [LayerSpec(block="prenorm_residual_short", mixer=mixer, ffn=ffn, mixer_norm=norm, ffn_norm=norm, prefix=f"l{i}")
                  for i, (mixer, ffn) in enumerate(config.layers)]
        return ModelSpec(architecture=self.name, vocab_size=config.vocab, hidden_size=config.width, layers=layers,
                         schedule=looped_schedule(len(layers), *config.loop, add_input=True), final_norm=norm, embedding_name="embed",
                         final_norm_prefix="final.norm", head_name="head", tie_word_embeddings=False,
                         logit_scale=config.logit_scale, logit_softcap=config.logit_softcap, raw=config.raw)


register_architecture(DezolornArchitecture(), replace=True)
