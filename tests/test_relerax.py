"""Relerax without a GPU: its configuration, the description the framework makes of it, the tensors it declares, what every
layer asks of the cache manager, the order in which an overlapping cache row hands out values, and properties of the plain
implementation that the GPU tests lean on (it does not look ahead; a window that is one off, the one left out of the
denominator, another pairing, values that turn with their keys, a correction in the weights or weights that do not sum to
one are other functions by far more than the tests allow)."""

import copy

import pytest
import torch

from clockwork_b200.cache import CacheManager
from clockwork_b200.config import PartSpec
from clockwork_b200.config.registry import architecture_name, shape_config, spec_from_raw
from clockwork_b200.parts import PagedKVNeed, build_model, build_part
from clockwork_b200.parts.model import tensor_decls_for_spec
from clockwork_b200.weights.loader import WeightMismatchError, check_declarations
from tests.plain import relerax_plain as plain
from tests.relerax_configs import CONFIGS, draw_weights, steady_routing, tensor_shapes, tokens_for


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_declared_tensors_are_the_checkpoints(name):
    config, _ = CONFIGS[name]
    spec = spec_from_raw(config)
    assert architecture_name(config) == "Relerax" and spec.architecture == "Relerax"
    assert not spec.tie_word_embeddings and spec.embedding_scale == 1.0 and spec.logit_softcap is None
    decls = tensor_decls_for_spec(spec)
    shapes = tensor_shapes(config)
    check_declarations(decls, shapes, "test")
    assert {d.name for d in decls if not d.optional} == set(shapes)
    for layer, listed in zip(spec.layers, config["layers"]):
        assert layer.block == "parallel_residual_two_norms" and layer.mixer_norm.kind == layer.ffn_norm.kind == "rmsnorm"
        m, mixer, mlp, ffn = listed["mixer"], layer.mixer, listed["mlp"], layer.ffn
        assert (mixer["heads"], mixer["dim"], mixer["vdim"], mixer["scale"]) == (m["heads"], m["dim"], m["vdim"], m["scale"])
        if listed["type"] == "attention":
            assert mixer.kind == "window_attention" and mixer["window"] == m["mask"]["size"] and mixer["sink"] == "zero"
            assert mixer["values"] == "keys" and mixer["gate"] == "entry" and mixer["rotary"]["scaling"] == m["rot"].get("scaling")
        else:
            assert mixer.kind == "latent_attention" and mixer["q_rank"] is None and not mixer["sink"] and mixer["gate"] == "head"
            assert (mixer["kv_rank"], mixer["rot_dim"], mixer["pairing"]) == (m["kv_rank"], m["rot_dim"], "interleaved")
        assert ffn.kind == ("none" if mlp is None else {"dense": "relu2_mlp", "moe": "moe"}[mlp["kind"]])
        if ffn.kind == "moe":
            assert (ffn["experts"], ffn["top"], ffn["identity"]) == (mlp["router"]["experts"], mlp["router"]["top"], mlp["router"].get("identity", 0))


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_what_every_layer_keeps(name):
    """A windowed layer keeps the rotated entries of a key twice and the others once; a latent layer one row for all heads."""
    config, page = CONFIGS[name]
    needs = build_model(spec_from_raw(config), torch.float32, "cpu").cache_needs()
    assert sorted(needs) == list(range(len(config["layers"])))
    for i, layer in enumerate(config["layers"]):
        m = layer["mixer"]
        if layer["type"] == "attention":
            assert needs[i] == PagedKVNeed(m["kv_heads"], m["dim"] + m["rot"]["dims"], m["mask"]["size"], planes=1)
        else:
            assert needs[i] == PagedKVNeed(1, m["kv_rank"] + m["rot_dim"], None, planes=1)
    cache = CacheManager(needs, num_pages=64, page_size=page, num_state_slots=4)
    req = cache.open("a")
    cache.reserve(req, 100)
    cache.check_invariants()
    cache.close("a")
    assert all(g.allocator.num_free == g.allocator.num_pages for g in cache.groups)


@pytest.mark.parametrize("heads, kv_heads, dim, rot", [(4, 2, 12, 4), (3, 1, 8, 8), (2, 2, 10, 6)])
def test_gate_and_output_weights_follow_the_order_of_a_value_in_its_row(heads, kv_heads, dim, rot):
    """A row holds [turned leading entries | rest | leading entries unturned]; read from where the rest begins, the value is
    the key with its leading entries last.  Gate rows and output columns are put in that order at load, so that gate and
    output product of the reordered value are those of the value."""
    gen = torch.Generator().manual_seed(dim)
    w = 16
    part = build_part("mixer", PartSpec("window_attention", dict(
        hidden_size=w, heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=1.0, window=5, sink="zero", values="keys", gate="entry",
        rotary={"dims": rot, "base": 100.0, "pairing": "interleaved"})), "m", torch.float32, "cpu")
    tensors = {d.name: torch.randn(d.shape, generator=gen) for d in part.tensor_decls()}
    assert set(tensors) == {"m.q", "m.k", "m.g", "m.o"}
    part.load_weights(tensors.__getitem__)
    raw, h = torch.randn(heads, dim, generator=gen), torch.randn(w, generator=gen)
    row = torch.cat([torch.randn(heads, rot, generator=gen), raw[:, rot:], raw[:, :rot]], dim=1)
    value = row[:, part.value_offset : part.value_offset + part.vdim]
    assert part.row == row.shape[1] == dim + rot
    assert torch.equal(value, torch.cat([raw[:, rot:], raw[:, :rot]], dim=1))
    gates = part.qkv.weight[(heads + kv_heads) * dim :] @ h
    got = part.o.weight @ (value.reshape(-1) * torch.sigmoid(gates))
    want = tensors["m.o"] @ (raw.reshape(-1) * torch.sigmoid(tensors["m.g"] @ h))
    assert torch.allclose(got, want, atol=1e-5)
    assert torch.equal(part.qkv.weight[: (heads + kv_heads) * dim], torch.cat([tensors["m.q"], tensors["m.k"]]))


def test_parts_refuse_what_does_not_go_together():
    window = dict(hidden_size=8, heads=2, kv_heads=1, dim=4, vdim=4, scale=1.0, window=5, values="keys", rotary={"dims": 2, "base": 10.0})
    for change in (dict(vdim=6), dict(pool=2), dict(values="queries")):
        with pytest.raises(ValueError):
            build_part("mixer", PartSpec("window_attention", dict(window, **change)), "m", torch.float32, "cpu")
    moe = dict(hidden_size=8, expert_size=4, experts=3, top=4, identity=1, scoring="all")
    build_part("ffn", PartSpec("moe", moe), "f", torch.float32, "cpu")
    for change in (dict(top=5), dict(scoring="chosen", renormalize=True), dict(scoring="chosen", correction=True), dict(gated=False, limit=1.0),
                   dict(identity=-1)):
        with pytest.raises(ValueError):
            build_part("ffn", PartSpec("moe", dict(moe, **change)), "f", torch.float32, "cpu")
    with pytest.raises(ValueError):
        build_part("mixer", PartSpec("latent_attention", dict(hidden_size=8, heads=2, dim=4, rot_dim=2, vdim=4, kv_rank=4, scale=1.0,
                                                              rope_base=10.0, eps=1e-5, gate="row")), "m", torch.float32, "cpu")


def test_the_named_shapes_describe_themselves():
    for name in ("relerax-tiny", "relerax-2k"):
        assert len(tensor_decls_for_spec(spec_from_raw(shape_config(name)))) > 10
    kinds = [layer.mixer.kind for layer in spec_from_raw(shape_config("relerax-2k")).layers]
    assert kinds.count("window_attention") == kinds.count("latent_attention") == 4


def test_a_wrong_shape_and_a_missing_tensor_are_reported_and_an_unused_norm_is_not():
    config, _ = CONFIGS["A"]
    shapes = tensor_shapes(config)
    shapes["l2.norm2"] = (config["width"],)  # (the last layer has no feed-forward)
    check_declarations(tensor_decls_for_spec(spec_from_raw(config)), shapes, "test")
    shapes["l1.mlp.correction"] = (5,)  # (the identity expert has one too)
    del shapes["l0.mlp.up.b"]
    shapes["l1.mix.v"] = (48, 64)
    with pytest.raises(WeightMismatchError) as e:
        check_declarations(tensor_decls_for_spec(spec_from_raw(config)), shapes, "test")
    assert all(name in str(e.value) for name in ("l1.mlp.correction", "l0.mlp.up.b", "l1.mix.v"))


@pytest.mark.parametrize("path, value, word", [
    (("layers", 0, "type"), "mamba2", "layer type"), (("layers", 1, "mixer", "mask"), {}, "size"), (("layers", 1, "mixer", "vdim"), 12, "vdim"),
    (("layers", 0, "mixer", "rot", "scaling"), {"factor": 2.0, "original": 8, "fast": 4.0}, "slow"),
    (("layers", 0, "mixer", "rot_dim"), 6, "rot_dim"), (("layers", 0, "mixer", "kv_rank"), None, "kv_rank"),
    (("layers", 1, "mlp", "router", "identity"), -1, "identity"), (("layers", 1, "mlp", "router", "top"), None, "top"),
    (("layers", 0, "mlp", "kind"), "gated", "feed-forward"), (("norm",), {}, "eps"), (("layers",), [], "layers")])
def test_configuration_errors_name_the_place(path, value, word):
    config = copy.deepcopy(CONFIGS["A"][0])
    at = config
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    with pytest.raises(ValueError) as e:
        spec_from_raw(config)
    assert word in str(e.value)


def _model(name, seed=3):
    config = CONFIGS[name][0]
    return config, {k: v.double() for k, v in draw_weights(config, seed).items()}


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_the_plain_implementation_does_not_look_ahead(name):
    config, w = _model(name)
    tokens = tokens_for(config, 50, salt=1)
    whole = plain.forward(config, w, tokens)
    for cut_at in (1, 7, 33):
        assert torch.allclose(plain.forward(config, w, tokens[:cut_at]), whole[:cut_at], atol=1e-9, rtol=0)
    other = list(tokens)
    other[20] = (other[20] + 1) % config["vocab"]
    changed = plain.forward(config, w, other)
    assert torch.equal(changed[:20], whole[:20])
    assert float((changed[21] - whole[21]).abs().max()) > 1e-3


def test_what_the_plain_implementation_is_sensitive_to():
    config, w = _model("A")
    tokens = tokens_for(config, 60, salt=2)
    want = plain.forward(config, w, tokens)

    def moved(change):
        other = copy.deepcopy(config)
        change(other["layers"])
        return float((plain.forward(other, w, tokens) - want).abs().max())

    for change in (lambda c: c[1]["mixer"]["mask"].update(size=22), lambda c: c[1]["mixer"]["mask"].update(size=20),
                   lambda c: c[2]["mixer"]["mask"].update(size=6), lambda c: c[1]["mixer"]["rot"].pop("scaling"),
                   lambda c: c[0]["mixer"]["rot"]["scaling"].update(factor=5.0), lambda c: c[0]["mixer"]["rot"].pop("scaling"),
                   lambda c: c[0]["mixer"].update(scale=0.2), lambda c: c[1]["mlp"]["router"].update(top=1)):
        assert moved(change) > 0.01
    for name, change in (("l0.mix.g", lambda t: t.zero_()), ("l1.mix.g", lambda t: t.zero_()), ("l0.mix.dkv.norm", lambda t: t.fill_(1.0)),
                         ("l0.mlp.up.b", lambda t: t.zero_()), ("l0.mlp.down.b", lambda t: t.zero_()), ("l1.mlp.correction", lambda t: t.zero_()),
                         ("l0.norm2", lambda t: t.copy_(w["l0.norm1"])), ("l1.norm2", lambda t: t.copy_(w["l1.norm1"]))):
        t = w[name].clone()
        change(t)
        assert float((plain.forward(config, dict(w, **{name: t}), tokens) - want).abs().max()) > 0.01, name


def test_weights_with_one_in_the_denominator():
    scores = torch.tensor([[-3.0, 0.5, float("-inf")], [40.0, 41.0, -50.0], [-900.0, -950.0, float("-inf")]], dtype=torch.float64)
    got = plain.weights_with_one(scores)
    want = torch.exp(scores[:2]) / (1 + torch.exp(scores[:2]).sum(-1, keepdim=True))
    assert torch.allclose(got[:2], want, atol=1e-12) and float(got[2].abs().max()) == 0.0


def test_choices_weights_and_identity_experts():
    """Two experts and one that hands its input on; the correction decides who is chosen and is in no weight."""
    h = torch.tensor([[1.0, 0.0], [0.0, 1.0]], dtype=torch.float64)
    w = {"router": torch.tensor([[2.0, 0.0], [1.0, 0.0], [0.0, 0.5]], dtype=torch.float64), "correction": torch.tensor([0.0, 0.0, 0.6])}
    s = torch.softmax(h @ w["router"].T, -1)
    chosen, weight, margin = plain.route(h, w, {"top": 2})
    assert chosen[0].tolist() == [2, 0] and margin[0] > 0  # the correction brings output 2 to the front
    assert torch.allclose(weight[0], s[0, [2, 0]] / s[0, [2, 0]].sum())
    w.update({f"e{e}.up": torch.full((3, 2), 1.0 + e, dtype=torch.float64) for e in range(2)})
    w.update({f"e{e}.down": torch.full((2, 3), 0.1 - e, dtype=torch.float64) for e in range(2)})
    out = plain.mixture(h, w, {"router": {"experts": 2, "top": 2, "identity": 1}})
    want = weight[0, 0] * h[0] + weight[0, 1] * plain.expert(h[:1], w, 0)[0]
    assert torch.allclose(out[0], want)


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_steady_routing_keeps_choices_wide_and_uses_several_experts(name):
    config = CONFIGS[name][0]
    probes = [tokens_for(config, 40, 50 + i) for i in range(2)]
    w = steady_routing(config, draw_weights(config, 4), probes)
    margins: list = []
    plain.forward(config, w, probes[0], margins=margins)
    assert len(margins) == sum(layer["mlp"] is not None and layer["mlp"]["kind"] == "moe" for layer in config["layers"])
    assert min(margins) > 0.02


def test_the_visible_positions():
    assert plain.visible(6, 3)[5].tolist() == [False, False, False, True, True, True]
    assert plain.visible(5, 1).tolist() == torch.eye(5, dtype=torch.bool).tolist()
    assert plain.visible(5, 9).tolist() == torch.ones(5, 5).tril().bool().tolist()
