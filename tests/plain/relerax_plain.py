"""A plain, slow forward pass of the Relerax design: whole sequences, no cache, one function per
mechanism, float32 or float64 torch on the CPU.  It is the yardstick of the tests and shares no
code with ``clockwork_b200``.

The design in this file's notation (x: residual row, W: a stored [out, in] matrix, t: position in the
sequence from 0, sg = logistic sigmoid, n(y) = y / sqrt(mean(y^2) + eps)):

* input:    x_t = E[token]
* layer:    x <- x + mixer(n(x) g1) + ff(n(x) g2), both norms of the same x      (a layer may have no ff)
* rotation: entry 2i turns with entry 2i+1 by the angle t f_i, sines and cosines times an amplitude; with a scaling
            {factor s, original L, fast, slow}: e_i = base^(-2i/dims), turns(m) = dims ln(L / (2 pi m)) / (2 ln base),
            lo = max(floor(turns(fast)), 0), hi = min(ceil(turns(slow)), dims - 1),
            w_i = clamp((i - lo) / max(hi - lo, 0.001), 0, 1), f_i = e_i (w_i / s + 1 - w_i), amplitude 1 + ln(s)/10
* `attention` mixer: H query heads on G key heads, no biases; the value of a key head is its key before the rotation;
            q and k turn in their first `dims` entries; position t sees 0 <= t - j < size; a_j = scale (q . k_j),
            weights exp(a_j) / (1 + sum exp(a)); W_o (concat_heads * sg(W_g h))            (W_g: a row per entry)
* `latent_attention` mixer: q = W_q h, per head [plain | turned]; W_d h = [c' | r']: c = n(c') w, r = r' turned, one for
            all heads; a_j = scale (q_plain . (W_uk c_j)_head + turned(q_turned) . r_j); ordinary softmax over j <= t;
            heads' sums of (W_uv c_j)_head times sg(W_g h)_head                            (W_g: a row per head); W_o
* ff:       dense: W_down relu(W_up h + b)^2 + b';  experts: s = softmax(W_router h), the `top` largest s + correction are
            chosen, weights s_e / (sum of the chosen s + 1e-20); expert e: W_down relu(W_up h)^2, the last `identity` of
            the outputs: h itself
* output:   logits = W_head (n(x) g_final)
"""

from __future__ import annotations

import json
import math
import struct
from pathlib import Path

import torch

WEIGHT_FLOOR = 1e-20


def exact(x):
    return x


def to_bfloat16_and_back(x):
    return x.to(torch.bfloat16).to(x.dtype)


def rms_norm(x, g, eps):
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps) * g


# ---- rotation ---------------------------------------------------------------------------------------
def frequencies(rot):
    """(the angle per position of every pair [dims/2] in float64, the amplitude of sines and cosines)."""
    dims, base = rot["dims"], rot["base"]
    i = torch.arange(dims // 2, dtype=torch.float64)
    f = torch.tensor(float(base), dtype=torch.float64) ** (-2.0 * i / dims)
    s = rot.get("scaling")
    if s is None:
        return f, 1.0

    def turns(m):
        return dims * math.log(s["original"] / (2 * math.pi * m)) / (2 * math.log(base))

    lo, hi = max(math.floor(turns(s["fast"])), 0), min(math.ceil(turns(s["slow"])), dims - 1)
    w = torch.clamp((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f * (w / s["factor"] + 1.0 - w), 1.0 + 0.1 * math.log(s["factor"])


def rotate(x, positions, rot):
    """x [T, heads, d]: the first ``dims`` entries of every head turn by their position."""
    dims = rot["dims"]
    f, amplitude = frequencies(rot)
    angle = positions.to(x.dtype)[:, None] * f.to(x.dtype)[None, :]
    cos, sin = torch.cos(angle)[:, None, :] * amplitude, torch.sin(angle)[:, None, :] * amplitude
    a, b = x[..., 0:dims:2], x[..., 1:dims:2]
    turned = torch.stack([a * cos - b * sin, b * cos + a * sin], dim=-1).flatten(-2)
    return torch.cat([turned, x[..., dims:]], dim=-1)


# ---- attention whose values are its keys ----------------------------------------------------------------
def visible(count, size):
    t = torch.arange(count)
    return (t[None, :] <= t[:, None]) & (t[:, None] - t[None, :] < size)


def weights_with_one(scores):
    """exp(a) / (1 + sum exp(a)) over the last dimension (masked entries are -inf)."""
    top = scores.amax(-1, keepdim=True).clamp(min=0.0)
    e = torch.exp(scores - top)
    return e / (torch.exp(-top) + e.sum(-1, keepdim=True))


def window_attention(h, w, m, eps, rnd=exact):
    heads, groups, d = m["heads"], m["kv_heads"], m["dim"]
    t, per = h.shape[0], m["heads"] // m["kv_heads"]
    positions = torch.arange(t)
    raw = (h @ w["k"].T).reshape(t, groups, d)
    q = rnd(rotate((h @ w["q"].T).reshape(t, heads, d), positions, m["rot"]))
    k, v = rnd(rotate(raw, positions, m["rot"])), rnd(raw)
    scores = torch.einsum("thd,shd->hts", q, k.repeat_interleave(per, dim=1)) * m["scale"]
    scores = scores.masked_fill(~visible(t, m["mask"]["size"]), float("-inf"))
    o = torch.einsum("hts,shd->thd", weights_with_one(scores), v.repeat_interleave(per, dim=1)).reshape(t, heads * d)
    return rnd(o * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


# ---- attention over a latent ------------------------------------------------------------------------------
def latent_attention(h, w, m, eps, rnd=exact):
    heads, d, r, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    t = h.shape[0]
    positions = torch.arange(t)
    q = (h @ w["q"].T).reshape(t, heads, d + r)
    down = h @ w["dkv"].T
    c = rnd(rms_norm(down[:, :rank], w["dkv.norm"], eps))
    turned_key = rnd(rotate(down[:, None, rank:], positions, m["rot"]))[:, 0]
    turned_query = rnd(rotate(q[..., d:], positions, m["rot"]))
    k = (c @ w["uk"].T).reshape(t, heads, d)
    v = (c @ w["uv"].T).reshape(t, heads, dv)
    scores = (torch.einsum("thd,shd->hts", rnd(q[..., :d]), k) + torch.einsum("thd,sd->hts", turned_query, turned_key)) * m["scale"]
    scores = scores.masked_fill(~visible(t, t), float("-inf"))
    o = torch.einsum("hts,shd->thd", torch.softmax(scores, dim=-1), v) * torch.sigmoid(h @ w["g"].T)[..., None]
    return rnd(o.reshape(t, heads * dv)) @ w["o"].T


# ---- feed-forwards ------------------------------------------------------------------------------------------
def squared_relu(z):
    return torch.relu(z) ** 2


def dense(h, w, f, rnd=exact):
    return rnd(squared_relu(h @ w["up"].T + w["up.b"])) @ w["down"].T + w["down.b"]


def route(h, w, router):
    """(chosen outputs [T, top], their weights [T, top], how far the last chosen one lies ahead of the next [T])."""
    s = torch.softmax(h @ w["router"].T, dim=-1)
    ranked = s + w["correction"]
    order = torch.argsort(ranked, dim=-1, descending=True, stable=True)
    top = router["top"]
    chosen = order[:, :top]
    weight = s.gather(1, chosen)
    sorted_rank = ranked.gather(1, order)
    margin = sorted_rank[:, top - 1] - sorted_rank[:, top] if top < s.shape[1] else torch.full((h.shape[0],), 1.0, dtype=h.dtype)
    return chosen, weight / (weight.sum(-1, keepdim=True) + WEIGHT_FLOOR), margin


def expert(h, w, e, rnd=exact):
    return rnd(squared_relu(h @ w[f"e{e}.up"].T)) @ w[f"e{e}.down"].T


def mixture(h, w, f, rnd=exact, margins=None):
    chosen, weight, margin = route(h, w, f["router"])
    if margins is not None:
        margins.append(float(margin.min()))
    out = torch.zeros_like(h)
    for e in range(w["router"].shape[0]):
        share = torch.where(chosen == e, weight, torch.zeros_like(weight)).sum(-1, keepdim=True)
        rows = share[:, 0] > 0
        if bool(rows.any()):
            y = h[rows] if e >= f["router"]["experts"] else expert(h[rows], w, e, rnd)
            out[rows] += share[rows] * y
    return out


# ---- the model -------------------------------------------------------------------------------------------
MIXERS = {"attention": window_attention, "latent_attention": latent_attention}


def sub(weights, prefix):
    return {k[len(prefix) + 1 :]: v for k, v in weights.items() if k.startswith(prefix + ".")}


def forward(config, weights, tokens, dtype=torch.float64, rnd=exact, keep_layers=False, margins=None):
    """Logits [T, vocab] of one whole sequence (and, with ``keep_layers``, the residual after every layer).
    ``rnd``: applied to what a bfloat16 run keeps in bfloat16 between kernels.  ``margins``: a list that receives, for
    every mixture of experts, how close its closest choice was."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    x, kept = w["embed"][torch.as_tensor(tokens, dtype=torch.long)], []
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}"
        y = MIXERS[layer["type"]](rnd(rms_norm(x, w[f"{p}.norm1"], eps)), sub(w, f"{p}.mix"), layer["mixer"], eps, rnd)
        f = layer.get("mlp")
        if f is not None:
            h, mlp = rnd(rms_norm(x, w[f"{p}.norm2"], eps)), sub(w, f"{p}.mlp")
            y = y + (dense(h, mlp, f, rnd) if f["kind"] == "dense" else mixture(h, mlp, f, rnd, margins))
        x = x + y
        kept.append(x)
    logits = rnd(rms_norm(x, w["final.norm"], eps)) @ w["head"].T
    return (logits, torch.stack(kept)) if keep_layers else logits


def greedy(config, weights, prompt, new_tokens, dtype=torch.float64):
    tokens = list(prompt)
    for _ in range(new_tokens):
        tokens.append(int(forward(config, weights, tokens, dtype)[-1].argmax()))
    return tokens[len(prompt):]


def read_model_dir(folder, dtype=torch.float32):
    """(config, {name: tensor}) of a folder with config.json and model.safetensors, read with nothing but the file format:
    an 8-byte little-endian header length, a JSON header, raw little-endian data."""
    folder = Path(folder)
    config = json.loads((folder / "config.json").read_text())
    blob = (folder / "model.safetensors").read_bytes()
    (n,) = struct.unpack("<Q", blob[:8])
    header, data = json.loads(blob[8 : 8 + n]), blob[8 + n :]
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32}
    out = {}
    for name, meta in header.items():
        if name != "__metadata__":
            a, b = meta["data_offsets"]
            out[name] = torch.frombuffer(bytearray(data[a:b]), dtype=kinds[meta["dtype"]]).reshape(meta["shape"]).to(dtype)
    return config, out
