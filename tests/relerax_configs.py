"""Small Relerax configurations of the tests and random weights for them, drawn here (tensor names and shapes are written
out from the configuration by this file's own rules, not asked of the package).

The four differ in every size, in the order of layers and in the values that a model may happen to make equal or 1: one
key head for all query heads and as many as query heads; all of a head rotated and only its first entries, an odd number
of pairs, with and without a stretched rotation; windows of 1 position, shorter than a page, no multiple of a page, a page,
and longer than the prompts; one latent head and more than a tile of the tensor-core kernel holds; latents shorter and
longer than a block of threads; values narrower and wider than keys; head sizes that no vector access fits; no, one and as
many identity experts as others, one choice and as many as there are experts; layers without feed-forward; widths that
are no power of two and no multiple of 4."""

from __future__ import annotations

import json
import math
from pathlib import Path

import torch

from tests.plain import relerax_plain as plain


def _rot(dims, base, scaling):
    out = {"dims": dims, "base": base}
    if scaling is not None:
        out["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return out


def attention(heads, kv_heads, dim, scale, size, rot, base, scaling=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale,
                                           "mask": {"size": size}, "rot": _rot(rot, base, scaling)}}


def latent(heads, dim, rot, vdim, rank, scale, base, scaling=None):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank,
                                                  "scale": scale, "rot": _rot(rot, base, scaling)}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, identity):
    router = {"experts": experts, "top": top}
    if identity:
        router["identity"] = identity
    return {"kind": "moe", "expert": {"ff": ff}, "router": router}


def _model(vocab, width, eps, layers):
    return {"architecture": "Relerax", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "layers": [dict(layer, mlp=mlp) for layer, mlp in layers]}


CONFIG_A = _model(96, 64, 1e-5, [
    (latent(3, 24, 8, 20, 40, 0.22, 300.0, (4.0, 60, 6.0, 1.0)), dense(40)),
    (attention(4, 2, 24, 0.2, 21, 8, 1000.0, (2.0, 90, 8.0, 0.5)), moe(28, 5, 2, 1)),
    (attention(3, 1, 16, 0.25, 7, 16, 50000.0), None),
])
CONFIG_B = _model(80, 50, 1e-6, [
    (attention(3, 3, 10, 0.3, 200, 6, 100.0), moe(17, 4, 4, 0)),
    (latent(1, 16, 16, 12, 16, 0.3, 10000.0), None),
    (latent(5, 8, 4, 14, 136, 0.35, 50.0, (8.0, 32, 4.0, 2.0)), dense(30)),
    (attention(2, 2, 12, 0.3, 3, 12, 500.0, (8.0, 32, 4.0, 2.0)), moe(20, 3, 1, 3)),
])
CONFIG_C = _model(120, 74, 1e-5, [
    (attention(6, 1, 8, 0.4, 1, 2, 10000.0), moe(12, 3, 4, 3)),
    (attention(2, 2, 40, 0.15, 16, 40, 200000.0, (16.0, 1024, 32.0, 1.0)), dense(56)),
    (latent(6, 16, 2, 8, 24, 0.3, 20.0), moe(24, 7, 3, 2)),
])
CONFIG_D = _model(1000, 384, 1e-6, [  # sizes that the tensor-core kernels take
    (latent(8, 48, 16, 40, 112, 0.14, 10000.0, (4.0, 256, 24.0, 1.0)), dense(160)),
    (attention(8, 2, 64, 0.12, 33, 32, 500000.0, (4.0, 512, 24.0, 1.0)), moe(48, 11, 3, 2)),
    (latent(20, 16, 64, 24, 256, 0.12, 5000.0, (2.0, 128, 8.0, 0.25)), moe(64, 6, 2, 1)),
    (attention(4, 4, 80, 80 ** -0.5, 100, 16, 1000.0), dense(96)),
])
CONFIGS = {"A": (CONFIG_A, 4), "B": (CONFIG_B, 8), "C": (CONFIG_C, 16), "D": (CONFIG_D, 16)}  # name -> (config, page size)


def tensor_shapes(config: dict) -> dict[str, tuple]:
    w = config["width"]
    out = {"embed": (config["vocab"], w), "head": (config["vocab"], w), "final.norm": (w,)}
    for i, layer in enumerate(config["layers"]):
        p, m, f = f"l{i}.mix", layer["mixer"], layer["mlp"]
        h, d, dv = m["heads"], m["dim"], m["vdim"]
        out[f"l{i}.norm1"] = (w,)
        if layer["type"] == "attention":
            out.update({f"{p}.q": (h * d, w), f"{p}.k": (m["kv_heads"] * d, w), f"{p}.g": (h * dv, w)})
        else:
            r, rank = m["rot_dim"], m["kv_rank"]
            out.update({f"{p}.q": (h * (d + r), w), f"{p}.dkv": (rank + r, w), f"{p}.dkv.norm": (rank,), f"{p}.uk": (h * d, rank),
                        f"{p}.uv": (h * dv, rank), f"{p}.g": (h, w)})
        out[f"{p}.o"] = (w, h * dv)
        if f is not None:
            out[f"l{i}.norm2"] = (w,)
        if f is not None and f["kind"] == "dense":
            out.update({f"l{i}.mlp.up": (f["ff"], w), f"l{i}.mlp.up.b": (f["ff"],), f"l{i}.mlp.down": (w, f["ff"]), f"l{i}.mlp.down.b": (w,)})
        elif f is not None:
            ff, outputs = f["expert"]["ff"], f["router"]["experts"] + f["router"].get("identity", 0)
            out.update({f"l{i}.mlp.router": (outputs, w), f"l{i}.mlp.correction": (outputs,)})
            for e in range(f["router"]["experts"]):
                out.update({f"l{i}.mlp.e{e}.up": (ff, w), f"l{i}.mlp.e{e}.down": (w, ff)})
    return out


def draw_weights(config: dict, seed: int) -> dict[str, torch.Tensor]:
    """bfloat16 tensors.  Matrices N(0, 1/in) so that activations keep their size; queries and keys larger, so that
    attention is peaked and a key that is missed or seen wrongly moves the logits; corrections of the scores' size."""
    gen = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(config).items():
        leaf = name.split(".", 1)[-1] if name.startswith("l") else name
        n = lambda scale=1.0: torch.randn(shape, generator=gen) * scale  # noqa: E731
        if leaf == "embed":
            t = n(0.7)
        elif leaf in ("norm1", "norm2", "final.norm", "mix.dkv.norm"):
            t = 1.0 + n(0.2)
        elif leaf in ("mix.q", "mix.k", "mix.dkv"):
            t = n(2.0 / math.sqrt(shape[-1]))
        elif leaf in ("mix.uk", "mlp.router"):
            t = n(1.6 / math.sqrt(shape[-1]))
        elif leaf in ("mlp.up.b", "mlp.down.b"):
            t = n(0.3)
        elif leaf == "mlp.correction":
            t = n(0.15)
        elif leaf == "head":
            t = n(2.0 / math.sqrt(shape[-1]))
        else:
            t = n(1.0 / math.sqrt(shape[-1]))
        out[name] = t.to(torch.bfloat16)
    return out


ROUTING_CLASSES = 8
MARGIN = 0.01  # how far the last chosen expert's rank lies ahead of the next one's, at least


def steady_routing(config: dict, weights: dict[str, torch.Tensor], probes: list[list[int]], seed: int = 0) -> dict[str, torch.Tensor]:
    """Router choices that rounding cannot flip, for runs in bfloat16 that are compared with a run that rounds elsewhere.
    The first ``ROUTING_CLASSES`` coordinates of the residual become a one-hot code of token mod classes that no layer
    writes to (an identity expert makes it larger), and every router reads, for each class, a permutation of the levels 0,
    0.6, 1.2 .. from that class's coordinate, besides a small part of its drawn weights on the others; corrections are
    a permutation of evenly spaced values.  Layer by layer the first of such permutations is taken that keeps every choice
    along ``probes`` wide (corrections may bring two experts close)."""
    c = ROUTING_CLASSES
    gen = torch.Generator().manual_seed(1000 + seed)
    out = {k: v.clone() for k, v in weights.items()}
    rows = torch.arange(config["vocab"])
    out["embed"][:, :c] = 0.0
    out["embed"][rows, rows % c] = 3.0
    for name, t in out.items():
        if name.endswith((".o", ".down", ".down.b")):
            t[:c] = 0.0
        elif name.endswith(".mlp.router"):
            t.mul_(0.02)
        elif name.endswith(".norm2"):
            t[:c] = 1.0
    for i, layer in enumerate(config["layers"]):
        if layer["mlp"] is None or layer["mlp"]["kind"] != "moe":
            continue
        router, correction = out[f"l{i}.mlp.router"], out[f"l{i}.mlp.correction"]
        for attempt in range(400):
            levels = torch.stack([0.6 * torch.randperm(router.shape[0], generator=gen) for _ in range(c)], dim=1)
            router[:, :c] = levels.to(torch.bfloat16)
            correction.copy_(0.08 * (torch.randperm(correction.shape[0], generator=gen) - correction.shape[0] / 2))
            margins: list = []
            for probe in probes:
                plain.forward(dict(config, layers=config["layers"][: i + 1]), out, probe, dtype=torch.float32, margins=margins)
                if margins[-1] < 3 * MARGIN:
                    break
            else:
                break
        else:
            raise AssertionError(f"layer {i}: no permutation keeps the choices wide")
    return out


def write_model(folder, name: str, seed: int = 0, steady: bool = False) -> Path:
    from clockwork_b200.weights import save_safetensors

    config = CONFIGS[name][0]
    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(config))
    weights = draw_weights(config, seed)
    save_safetensors(folder / "model.safetensors", steady_routing(config, weights, [tokens_for(config, 90, 90 + i) for i in range(8)], seed) if steady else weights)
    return folder


def tokens_for(config: dict, length: int, salt: int = 0) -> list[int]:
    state = (7919 * salt + 32452843 * length + 313) & 0x7FFFFFFF
    out = []
    for _ in range(length):
        state = (1103515245 * state + 12345) & 0x7FFFFFFF
        out.append((state >> 8) % config["vocab"])
    return out
