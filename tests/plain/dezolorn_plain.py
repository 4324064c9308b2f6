"""A plain, slow forward pass of the Dezolorn design: whole sequences, no cache, one function per
mechanism, float32 or float64 torch on the CPU.  It is the yardstick of the tests and shares no
code with ``clockwork_b200``.

The design in this file's notation (x: residual row, W: a stored [out, in] matrix, t: position in the
sequence from 0, sg = logistic sigmoid, r(y) = y / sqrt(mean(y^2) + eps), c(y) = y - mean(y)):

* input:    x_t = E[token]
* order:    layers 0 .. a-1 once, layers a .. b-1 `times` times over (same weights, every pass a cache or
            state of its own), layers b .. once; ahead of every pass but the first the input rows E[token]
            are added to x once
* layer:    x <- x + mixer(n(x) g1);  x <- x + ff(n(x) g2)     (a layer may have no ff)
            n(y) = c(y) / sqrt(mean(c(y)^2) + eps)
* `attention` mixer: H query heads on G key/value heads, no biases; r over all of q's rows at once times a
            weight, the same for k; then the first `dims` entries of every query and key head are rotated,
            entry 2i with entry 2i+1 by the angle t f_i, sines and cosines times an amplitude; with a scaling
            {factor s, original L, fast, slow}: e_i = base^(-2i/dims), turns(m) = dims ln(L / (2 pi m)) / (2 ln base),
            lo = max(floor(turns(fast)), 0), hi = min(ceil(turns(slow)), dims - 1),
            w_i = clamp((i - lo) / max(hi - lo, 0.001), 0, 1), f_i = e_i (w_i / s + 1 - w_i), amplitude 1 + ln(s)/10;
            position t sees j <= t with t - j < size or j < keep_first; softmax of scale (q . k); W_o
* `retention` mixer: q, k rotated (entry i with entry i + dims/2), k also times dk^(-1/2);
            S <- d_h S + k v^T, o = S^T q;  out = W_o (concat_heads(r(o_head)) silu(W_g h))
* `delta` mixer: q, k, v = silu(conv(W h)), conv a causal per-channel convolution over the last `taps` inputs;
            q, k per head divided by sqrt(|.|^2 + 1e-6), q also by sqrt(dk);  beta = sg(W_b h) per head;
            g = exp(-exp(A_head) softplus(W_a h + dt)) per head;
            S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q;
            out = W_o concat_heads(r(o_head) w silu(W_g h)_head)       (w of size dv, shared by the heads)
* ff:       W_down (silu(W_gate h) * W_up h)
* output:   z = s_l (W_head (n(x) g_final));  logits = cap tanh(z / cap)
"""

from __future__ import annotations

import json
import math
import struct
from pathlib import Path

import torch
import torch.nn.functional as F

UNIT_EPS = 1e-6


def exact(x):
    return x


def to_bfloat16_and_back(x):
    return x.to(torch.bfloat16).to(x.dtype)


def unit_rms(x, eps):
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def layer_norm(x, g, eps):
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt(c.pow(2).mean(-1, keepdim=True) + eps) * g


def run_order(config):
    """(layer, whether a pass other than the loop's first begins here) for every layer run, in order."""
    count = len(config["layers"])
    loop = config.get("loop") or {"start": 0, "stop": 0, "times": 1}
    a, b, times = loop["start"], loop["stop"], loop["times"]
    order = [(i, False) for i in range(a)]
    for p in range(times):
        order += [(i, p > 0 and i == a) for i in range(a, b)]
    order += [(i, False) for i in range(b, count)]
    return order


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


def rotate(x, positions, rot, interleaved):
    """x [T, heads, d]: the first ``dims`` entries of every head turn by their position."""
    dims = rot["dims"]
    f, amplitude = frequencies(rot)
    angle = positions.to(x.dtype)[:, None] * f.to(x.dtype)[None, :]
    cos, sin = torch.cos(angle)[:, None, :] * amplitude, torch.sin(angle)[:, None, :] * amplitude
    if interleaved:
        a, b = x[..., 0:dims:2], x[..., 1:dims:2]
        turned = torch.stack([a * cos - b * sin, b * cos + a * sin], dim=-1).flatten(-2)
    else:
        a, b = x[..., : dims // 2], x[..., dims // 2 : dims]
        turned = torch.cat([a * cos - b * sin, b * cos + a * sin], dim=-1)
    return torch.cat([turned, x[..., dims:]], dim=-1)


# ---- attention over a sliding window that keeps the first tokens ---------------------------------------
def visible(count, size, keep_first):
    t = torch.arange(count)
    return (t[None, :] <= t[:, None]) & ((t[:, None] - t[None, :] < size) | (t[None, :] < keep_first))


def window_attention(h, w, m, eps, rnd=exact):
    heads, groups, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    t = h.shape[0]
    positions = torch.arange(t)
    q = (unit_rms(h @ w["q"].T, eps) * w["q.norm"]).reshape(t, heads, dk)
    k = (unit_rms(h @ w["k"].T, eps) * w["k.norm"]).reshape(t, groups, dk)
    v = rnd(h @ w["v"].T).reshape(t, groups, dv)
    q, k = (rnd(rotate(x, positions, m["rot"], True)) for x in (q, k))
    per = heads // groups
    scores = torch.einsum("thd,shd->hts", q, k.repeat_interleave(per, dim=1)) * m["scale"]
    scores = scores.masked_fill(~visible(t, m["mask"]["size"], m["mask"]["keep_first"]), float("-inf"))
    o = torch.einsum("hts,shd->thd", torch.softmax(scores, dim=-1), v.repeat_interleave(per, dim=1))
    return rnd(o.reshape(t, heads * dv)) @ w["o"].T


# ---- retention -------------------------------------------------------------------------------------------
def retention(h, w, m, eps, rnd=exact):
    heads, dk, dv = m["heads"], m["dim"], m["vdim"]
    t = h.shape[0]
    positions = torch.arange(t)
    q, k = ((h @ w[n].T).reshape(t, heads, dk) for n in "qk")
    v = (h @ w["v"].T).reshape(t, heads, dv)
    q, k = (rotate(x, positions, m["rot"], False) for x in (q, k))
    k = k * dk ** -0.5
    decay = torch.tensor(m["decay"], dtype=torch.float64).to(h.dtype)[:, None, None]
    state = torch.zeros(heads, dk, dv, dtype=h.dtype)
    out = []
    for i in range(t):
        state = decay * state + k[i][:, :, None] * v[i][:, None, :]
        out.append(torch.einsum("hkv,hk->hv", state, q[i]))
    o = unit_rms(torch.stack(out), eps).reshape(t, heads * dv)
    return rnd(o * F.silu(h @ w["g"].T)) @ w["o"].T


# ---- the gated delta rule with one decay per head --------------------------------------------------------
def short_convolution(x, taps_weight):
    """x [T, C], taps_weight [C, taps] (the last column is the current token's): zeros before the first row."""
    taps = taps_weight.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x])
    return sum(padded[j : j + x.shape[0]] * taps_weight[:, j] for j in range(taps))


def unit_length(x):
    return x / torch.sqrt(x.pow(2).sum(-1, keepdim=True) + UNIT_EPS)


def head_decays(z, a_log, dt_bias):
    """z [T, H] -> the decay of every head: exp(-exp(A) softplus(z + dt))."""
    return torch.exp(-torch.exp(a_log) * F.softplus(z + dt_bias, threshold=1e9))


def delta_scan(q, k, v, decay, beta):
    """q, k [T, H, dk], v [T, H, dv], decay, beta [T, H] -> [T, H, dv]; the read-out sees the token's own write."""
    t, heads, dk = q.shape
    state = torch.zeros(heads, dk, v.shape[-1], dtype=q.dtype)
    out = []
    for i in range(t):
        state = decay[i][:, None, None] * state
        u = beta[i][:, None] * (v[i] - torch.einsum("hkv,hk->hv", state, k[i]))
        state = state + k[i][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hkv,hk->hv", state, q[i]))
    return torch.stack(out)


def gated_delta(h, w, m, eps, rnd=exact):
    heads, groups, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    t, per = h.shape[0], heads // groups
    q, k, v = (F.silu(short_convolution(h @ w[n].T, w[f"{n}.conv"])) for n in "qkv")
    q, k, v = q.reshape(t, groups, dk), k.reshape(t, groups, dk), v.reshape(t, heads, dv)
    q = (unit_length(q) * dk ** -0.5).repeat_interleave(per, dim=1)
    k = unit_length(k).repeat_interleave(per, dim=1)
    o = delta_scan(q, k, v, head_decays(h @ w["a"].T, w["A_log"], w["dt_bias"]), torch.sigmoid(h @ w["b"].T))
    o = unit_rms(o, eps) * w["norm"] * F.silu(h @ w["g"].T).reshape(t, heads, dv)
    return rnd(o.reshape(t, heads * dv)) @ w["o"].T


# ---- the model -------------------------------------------------------------------------------------------
def feed_forward(h, w, rnd=exact):
    return rnd(F.silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


MIXERS = {"attention": window_attention, "retention": retention, "delta": gated_delta}


def sub(weights, prefix):
    return {k[len(prefix) + 1 :]: v for k, v in weights.items() if k.startswith(prefix + ".")}


def forward(config, weights, tokens, dtype=torch.float64, rnd=exact, keep_layers=False):
    """Logits [T, vocab] of one whole sequence (and, with ``keep_layers``, the residual after every layer run).
    ``rnd``: applied to what a bfloat16 run keeps in bfloat16 between kernels."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    rows = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    x, kept = rows, []
    for i, again in run_order(config):
        layer, p = config["layers"][i], f"l{i}"
        if again:
            x = x + rows
        x = x + MIXERS[layer["type"]](rnd(layer_norm(x, w[f"{p}.norm1"], eps)), sub(w, f"{p}.mix"), layer["mixer"], eps, rnd)
        if layer.get("mlp") is not None:
            x = x + feed_forward(rnd(layer_norm(x, w[f"{p}.norm2"], eps)), sub(w, f"{p}.mlp"), rnd)
        kept.append(x)
    z = config["logit_scale"] * (rnd(layer_norm(x, w["final.norm"], eps)) @ w["head"].T)
    cap = config["logit_softcap"]
    logits = cap * torch.tanh(z / cap)
    return (logits, torch.stack(kept)) if keep_layers else logits


def first_position_margin(config, weights, token, dtype=torch.float64):
    """At position 0 a head of the retention and of the delta mixer puts out (k . q) times a positive number times v,
    and the norm behind it makes sign(k . q) r(v) of that: the smallest |cos(q, k)| over those heads, in every layer
    run, says how far the first token is from a sign that rounding could flip."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    rows = w["embed"][torch.as_tensor([token], dtype=torch.long)]
    x, margin = rows, 1.0
    for i, again in run_order(config):
        layer, p, m = config["layers"][i], f"l{i}", config["layers"][i]["mixer"]
        if again:
            x = x + rows
        h, mix = layer_norm(x, w[f"{p}.norm1"], eps), sub(w, f"{p}.mix")
        if layer["type"] == "retention":
            q, k = ((h @ mix[n].T).reshape(m["heads"], m["dim"]) for n in "qk")
        elif layer["type"] == "delta":
            q, k = (F.silu((h @ mix[n].T) * mix[f"{n}.conv"][:, -1]).reshape(m["kv_heads"], m["dim"]) for n in "qk")
        if layer["type"] != "attention":
            margin = min(margin, float(((q * k).sum(-1) / (q.norm(dim=-1) * k.norm(dim=-1))).abs().min()))
        x = x + MIXERS[layer["type"]](h, mix, m, eps)
        if layer.get("mlp") is not None:
            x = x + feed_forward(layer_norm(x, w[f"{p}.norm2"], eps), sub(w, f"{p}.mlp"))
    return margin


def steady_first_token(config, weights, candidates=range(40)):
    """The candidate whose answer at position 0 is farthest from such a flip."""
    return max(candidates, key=lambda token: first_position_margin(config, weights, token))


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
