"""Small Dezolorn configurations of the tests and random weights for them, drawn here (tensor names and shapes are
written out from the configuration by this file's own rules, not asked of the package).

The four differ in every size, in the order of layers and in the values that a model may happen to make equal or 1: one
key/value head for all query heads and as many as query heads; values narrower and wider than keys; all of a head rotated
and only its first entries, an odd number of pairs, with and without a stretched rotation; windows of 1 position, shorter
than a page, no multiple of a page, and longer than the prompts; no kept position, one, a whole page of them, and more
than the window holds; one head; heads of sizes that no vector access fits; convolutions of 1, 3, 4 and 6 taps; q and k
heads shared by several value heads and not; layers without feed-forward; no loop, a loop in the middle, one over all
layers, one that begins with each kind of mixer; a logit scale of 1; a cap that bends and one that does not; widths that
are no power of two and no multiple of 4."""

from __future__ import annotations

import json
import math
from pathlib import Path

import torch

from tests.plain import dezolorn_plain as plain


def _attention(heads, kv_heads, dim, vdim, scale, size, keep, rot, base, scaling=None):
    turned = {"dims": rot, "base": base}
    if scaling is not None:
        turned["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                                           "mask": {"size": size, "keep_first": keep}, "rot": turned}}


def _retention(dim, vdim, decay, rot, base):
    return {"type": "retention", "mixer": {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": decay,
                                           "rot": {"dims": rot, "base": base}}}


def _delta(heads, kv_heads, dim, vdim, conv):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def _model(vocab, width, eps, scale, cap, loop, layers):
    out = {"architecture": "Dezolorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": scale, "logit_softcap": cap,
           "layers": [dict(layer, mlp=None if ff is None else {"kind": "dense", "ff": ff}) for layer, ff in layers]}
    if loop is not None:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


CONFIG_A = _model(96, 64, 1e-5, 0.4, 8.0, (1, 3, 2), [
    (_delta(4, 2, 8, 16, 4), 40),
    (_attention(4, 2, 24, 12, 0.2, 21, 5, 8, 1000.0, (4.0, 60, 6.0, 1.0)), None),
    (_retention(12, 20, [0.9, 0.97, 0.995], 12, 300.0), 56),
    (_attention(3, 1, 16, 40, 0.25, 7, 2, 16, 50000.0, (2.0, 200, 16.0, 0.5)), 24),
])
CONFIG_B = _model(80, 50, 1e-6, 1.0, 50.0, None, [
    (_attention(3, 3, 10, 8, 0.3, 200, 0, 6, 100.0), 30),
    (_retention(16, 8, [0.98], 16, 10000.0), None),
    (_attention(2, 2, 12, 20, 0.3, 3, 9, 12, 500.0, (8.0, 32, 4.0, 2.0)), None),
    (_delta(3, 3, 10, 7, 1), 44),
])
CONFIG_C = _model(120, 74, 1e-5, 0.25, 4.0, (0, 4, 3), [
    (_retention(8, 24, [0.5, 0.8, 0.9, 0.95, 0.99], 4, 50.0), None),
    (_attention(6, 1, 8, 24, 0.35, 1, 1, 2, 10000.0), 28),
    (_delta(6, 1, 24, 12, 6), None),
    (_attention(2, 2, 40, 8, 0.15, 16, 16, 40, 200000.0, (16.0, 1024, 32.0, 1.0)), 12),
])
CONFIG_D = _model(1000, 384, 1e-6, 0.5, 10.0, (2, 4, 2), [  # sizes that the tensor-core kernels take
    (_attention(8, 2, 32, 64, 32 ** -0.5, 33, 4, 32, 10000.0, (4.0, 256, 24.0, 1.0)), 128),
    (_delta(4, 2, 64, 48, 3), None),
    (_retention(64, 96, [0.9, 0.99], 32, 5000.0), 96),
    (_attention(12, 3, 48, 80, 48 ** -0.5, 60, 20, 16, 500000.0), 160),
    (_attention(4, 4, 80, 200, 80 ** -0.5, 100, 7, 80, 1000.0, (2.0, 128, 8.0, 0.25)), None),
])
CONFIGS = {"A": (CONFIG_A, 4), "B": (CONFIG_B, 8), "C": (CONFIG_C, 16), "D": (CONFIG_D, 16)}  # name -> (config, page size)


def tensor_shapes(config: dict) -> dict[str, tuple]:
    w = config["width"]
    out = {"embed": (config["vocab"], w), "head": (config["vocab"], w), "final.norm": (w,)}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.mix", layer["mixer"]
        out[f"l{i}.norm1"] = (w,)
        h, dk, dv = m["heads"], m["dim"], m["vdim"]
        g = m.get("kv_heads", h)
        vh = g if layer["type"] == "attention" else h  # heads of values
        qh = h if layer["type"] == "attention" else g  # heads of queries
        out.update({f"{p}.q": (qh * dk, w), f"{p}.k": (g * dk, w), f"{p}.v": (vh * dv, w), f"{p}.o": (w, h * dv)})
        if layer["type"] == "attention":
            out.update({f"{p}.q.norm": (h * dk,), f"{p}.k.norm": (g * dk,)})
        else:
            out[f"{p}.g"] = (h * dv, w)
        if layer["type"] == "delta":
            out.update({f"{p}.{n}.conv": (out[f"{p}.{n}"][0], m["conv"]) for n in "qkv"})
            out.update({f"{p}.a": (h, w), f"{p}.b": (h, w), f"{p}.A_log": (h,), f"{p}.dt_bias": (h,), f"{p}.norm": (dv,)})
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            out.update({f"l{i}.norm2": (w,), f"l{i}.mlp.gate": (ff, w), f"l{i}.mlp.up": (ff, w), f"l{i}.mlp.down": (w, ff)})
    return out


def draw_weights(config: dict, seed: int) -> dict[str, torch.Tensor]:
    """bfloat16 tensors.  Matrices N(0, 1/in) so that activations keep their size; embedding rows with a mean, so that a
    norm that does not take it off shows; the query and key norms' weights large, so that attention is peaked and a key
    that is missed or seen wrongly moves the logits; decays near 1, so that a state remembers dozens of tokens and a lost
    or stale state shows."""
    gen = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(config).items():
        leaf = name.split(".", 1)[-1] if name.startswith("l") else name
        n = lambda scale=1.0: torch.randn(shape, generator=gen) * scale  # noqa: E731
        if leaf == "embed":
            t = 0.5 + n(0.7)
        elif leaf in ("norm1", "norm2", "final.norm", "mix.norm"):
            t = 1.0 + n(0.2)
        elif leaf in ("mix.q.norm", "mix.k.norm"):
            t = 1.6 + n(0.2)
        elif leaf.endswith(".conv"):
            t = n(0.3)
            t[:, -1] += 0.7
        elif leaf == "mix.A_log":
            t = n(0.4)
        elif leaf == "mix.dt_bias":
            t = -3.0 + n(0.7)
        elif leaf == "head":
            t = n(2.0 / math.sqrt(shape[-1]))
        else:
            t = n(1.0 / math.sqrt(shape[-1]))
        out[name] = t.to(torch.bfloat16)
    return out


def write_model(folder, name: str, seed: int = 0) -> Path:
    from clockwork_b200.weights import save_safetensors

    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(CONFIGS[name][0]))
    save_safetensors(folder / "model.safetensors", draw_weights(CONFIGS[name][0], seed))
    return folder


def tokens_for(config: dict, length: int, salt: int = 0, first: int | None = None) -> list[int]:
    """``first``: the sequence's first token (``plain.steady_first_token``: an answer at position 0 that rounding cannot flip)."""
    state = (7919 * salt + 32452843 * length + 313) & 0x7FFFFFFF
    out = []
    for _ in range(length):
        state = (1103515245 * state + 12345) & 0x7FFFFFFF
        out.append((state >> 8) % config["vocab"])
    if first is not None and out:
        out[0] = first
    return out


def first_tokens(dirs: dict) -> dict[str, int]:
    return {name: plain.steady_first_token(*plain.read_model_dir(folder, dtype=torch.float64)) for name, folder in dirs.items()}
