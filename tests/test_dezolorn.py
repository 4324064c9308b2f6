"""Dezolorn without a GPU: its configuration, the description the framework makes of it, the tensors it declares, what
every layer run asks of the cache manager (pages of kept first positions among them), the tables of a stretched rotation,
and properties of the plain implementation that the GPU tests lean on (it does not look ahead; a window or a number of
kept positions that is one off, norms left out, another pairing, a state that starts late, input rows that are not added
again are other functions by far more than the tests allow)."""

import copy

import pytest
import torch

from clockwork_b200.cache import CacheManager
from clockwork_b200.config.model_spec import looped_schedule
from clockwork_b200.config.registry import architecture_name, shape_config, spec_from_raw
from clockwork_b200.parts import PagedKVNeed, SlotStateNeed, build_model
from clockwork_b200.parts.model import tensor_decls_for_spec
from clockwork_b200.parts.rotary import check_rotary, rotary_tables
from clockwork_b200.weights.loader import WeightMismatchError, check_declarations
from tests.dezolorn_configs import CONFIGS, draw_weights, tensor_shapes, tokens_for
from tests.plain import dezolorn_plain as plain


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_declared_tensors_are_the_checkpoints(name):
    config, _ = CONFIGS[name]
    spec = spec_from_raw(config)
    assert architecture_name(config) == "Dezolorn" and spec.architecture == "Dezolorn"
    assert not spec.tie_word_embeddings and spec.embedding_scale == 1.0
    assert (spec.logit_scale, spec.logit_softcap) == (config["logit_scale"], config["logit_softcap"])
    decls = tensor_decls_for_spec(spec)
    shapes = tensor_shapes(config)
    check_declarations(decls, shapes, "test")
    assert {d.name for d in decls if not d.optional} == set(shapes)
    for layer, listed in zip(spec.layers, config["layers"]):
        assert layer.block == "prenorm_residual_short" and layer.mixer_norm.kind == layer.ffn_norm.kind == "layernorm"
        m, mixer = listed["mixer"], layer.mixer
        assert mixer.kind == {"attention": "window_attention", "retention": "retention", "delta": "head_delta"}[listed["type"]]
        assert (mixer["heads"], mixer["dim"], mixer["vdim"]) == (m["heads"], m["dim"], m["vdim"])
        if listed["type"] == "attention":
            assert mixer["window"] == m["mask"]["size"] and mixer["keep_first"] == m["mask"]["keep_first"]
            assert mixer["scale"] == m["scale"] and mixer["qk_norm"] == config["norm"]["eps"]
            assert mixer["rotary"]["pairing"] == "interleaved" and mixer["rotary"]["scaling"] == m["rot"].get("scaling")
        elif listed["type"] == "retention":
            assert mixer["decay"] == m["decay"] and mixer["rotary"]["pairing"] == "half"
        else:
            assert mixer["conv"] == m["conv"] and mixer["kv_heads"] == m["kv_heads"]
        assert layer.ffn.kind == ("none" if listed["mlp"] is None else "swiglu")


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_the_order_of_runs_and_what_every_run_keeps(name):
    config, page = CONFIGS[name]
    spec = spec_from_raw(config)
    order = plain.run_order(config)
    assert [(s.layer, s.add_input) for s in spec.schedule] == order
    layers = [s.resolved_cache_layer() for s in spec.schedule]
    assert len(set(layers)) == len(layers)  # every run keeps a cache or state of its own
    needs = build_model(spec, torch.float32, "cpu").cache_needs()
    assert sorted(needs) == sorted(layers)
    for step, (i, _) in zip(spec.schedule, order):
        m, kind = config["layers"][i]["mixer"], config["layers"][i]["type"]
        need = needs[step.resolved_cache_layer()]
        if kind == "attention":
            assert need == PagedKVNeed(m["kv_heads"], m["dim"] + m["vdim"], m["mask"]["size"], planes=1, keep_first=m["mask"]["keep_first"])
        elif kind == "retention":
            assert need == SlotStateNeed((m["heads"] * m["dim"] * m["vdim"],))
        else:
            channels = 2 * m["kv_heads"] * m["dim"] + m["heads"] * m["vdim"]
            assert need == SlotStateNeed((m["heads"] * m["dim"] * m["vdim"] + (m["conv"] - 1) * channels,))
    cache = CacheManager(needs, num_pages=64, page_size=page, num_state_slots=4)
    req = cache.open("a")
    cache.reserve(req, 100)
    cache.check_invariants()
    cache.close("a")
    assert all(g.allocator.num_free == g.allocator.num_pages for g in cache.groups)


def test_a_loop_may_add_the_input_rows_ahead_of_every_further_pass():
    steps = looped_schedule(5, 1, 3, 3, add_input=True)
    assert [s.layer for s in steps] == [0, 1, 2, 1, 2, 1, 2, 3, 4]
    assert [s.add_input for s in steps] == [False, False, False, True, False, True, False, False, False]
    assert not any(s.add_input for s in looped_schedule(5, 1, 3, 3))
    assert not any(s.add_input for s in looped_schedule(5, 1, 3, 1, add_input=True) + looped_schedule(5, 2, 2, 4, add_input=True))


@pytest.mark.parametrize("keep, window, page", [(5, 12, 4), (4, 12, 4), (1, 3, 4), (0, 12, 4), (9, 3, 8), (20, 6, 16), (16, 6, 16)])
def test_pages_of_kept_first_positions_are_never_given_back(keep, window, page):
    need = PagedKVNeed(2, 8, window, planes=1, keep_first=keep)
    cache = CacheManager({0: need}, num_pages=40, page_size=page, num_state_slots=2)
    req = cache.open("a")
    for n in range(1, 120):
        cache.reserve(req, n)
        req.num_computed = n
        cache.release_behind_window(req, n)
        table = req.tables[0]
        for p in range(n + 1):  # what position n reads next (its own page comes with its reservation)
            if p < n and (n - p < window or p < keep):
                assert table[p // page] >= 0, (n, p)
        held = sum(t >= 0 for t in table)
        assert held <= -(-keep // page) + window // page + 2
        cache.check_invariants()
    assert cache.slots(req, 0, 0, min(keep, 1)) == [table[0] * page][: min(keep, 1)]
    cache.close("a")
    assert cache.groups[0].allocator.num_free == 40


@pytest.mark.parametrize("rot", [
    {"dims": 16, "base": 10000.0}, {"dims": 6, "base": 50.0}, {"dims": 2, "base": 3.0},
    {"dims": 32, "base": 10000.0, "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}},
    {"dims": 24, "base": 500.0, "scaling": {"factor": 8.0, "original": 64, "fast": 6.0, "slow": 0.5}},
    {"dims": 8, "base": 1e6, "scaling": {"factor": 1.0, "original": 128, "fast": 2.0, "slow": 2.0}},
    {"dims": 12, "base": 20.0, "scaling": {"factor": 2.0, "original": 16, "fast": 64.0, "slow": 16.0}}])
def test_the_tables_of_a_rotation(rot):
    got, amplitude = rotary_tables(rot["dims"], rot["base"], rot.get("scaling"))
    want, expected = plain.frequencies(rot)
    assert got.dtype == torch.float32 and torch.allclose(got.double(), want, rtol=1e-7, atol=0)
    assert abs(amplitude - expected) < 1e-12
    if rot.get("scaling") is None:
        assert amplitude == 1.0
    elif rot["scaling"]["factor"] > 1:
        plain_freq, _ = rotary_tables(rot["dims"], rot["base"])
        ratio = got / plain_freq  # between 1 / factor and 1, falling with the pair's index
        assert float(ratio.min()) >= 1 / rot["scaling"]["factor"] - 1e-6 and bool((ratio[1:] <= ratio[:-1] + 1e-6).all())


def test_a_long_stretched_rotation_ramps_between_its_ends():
    got, _ = rotary_tables(128, 10000.0, {"factor": 40.0, "original": 4096, "fast": 32.0, "slow": 1.0})
    plain_freq, _ = rotary_tables(128, 10000.0)
    ratio = got / plain_freq
    assert float(ratio[0]) == 1.0 and abs(float(ratio[-1]) - 1 / 40) < 1e-6
    between = (ratio < 0.999) & (ratio > 1 / 40 + 1e-3)
    assert 10 < int(between.sum()) < 40


@pytest.mark.parametrize("rotary", [{"dims": 3, "base": 10.0}, {"dims": 20, "base": 10.0}, {"dims": 4, "base": 0.0},
                                    {"dims": 4, "base": 10.0, "pairing": "pairs"},
                                    {"dims": 4, "base": 10.0, "scaling": {"factor": 0.0, "original": 4, "fast": 2.0, "slow": 1.0}}])
def test_rotations_that_do_not_fit_are_refused(rotary):
    with pytest.raises(ValueError):
        check_rotary(rotary, 16)


def test_the_named_shapes_describe_themselves():
    for name in ("dezolorn-tiny", "dezolorn-2k"):
        assert len(tensor_decls_for_spec(spec_from_raw(shape_config(name)))) > 10
    kinds = [layer.mixer.kind for layer in spec_from_raw(shape_config("dezolorn-2k")).layers]
    assert kinds.count("window_attention") == 4 and kinds.count("retention") == kinds.count("head_delta") == 2


def test_a_wrong_shape_and_a_missing_tensor_are_reported():
    config, _ = CONFIGS["A"]
    shapes = tensor_shapes(config)
    shapes["l1.mix.q.norm"] = (5, 4)
    del shapes["l0.mix.dt_bias"]
    shapes["head"] = (3, config["width"])
    with pytest.raises(WeightMismatchError) as e:
        check_declarations(tensor_decls_for_spec(spec_from_raw(config)), shapes, "test")
    assert all(name in str(e.value) for name in ("l1.mix.q.norm", "l0.mix.dt_bias", "head"))


@pytest.mark.parametrize("path, value, word", [
    (("layers", 0, "type"), "attention_2", "layer type"), (("layers", 1, "mixer", "mask"), {"keep_first": 4}, "size"),
    (("layers", 1, "mixer", "mask", "keep_first"), -1, "keep_first"), (("layers", 2, "mixer", "decay"), [0.5], "decay"),
    (("layers", 1, "mixer", "rot", "scaling"), {"factor": 2.0, "original": 8, "fast": 4.0}, "slow"),
    (("layers", 0, "mixer", "conv"), None, "conv"), (("logit_scale",), None, "logit_scale"), (("logit_softcap",), -1.0, "logit_softcap"),
    (("layers", 0, "mlp", "kind"), "moe", "feed-forward"), (("loop",), {"start": 2, "stop": 9, "times": 2}, "loop"),
    (("loop",), {"start": 1, "stop": 3}, "times"), (("norm",), {}, "eps")])
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
        change(other)
        return float((plain.forward(other, w, tokens) - want).abs().max())

    def mixer(i):
        return lambda c: c["layers"][i]["mixer"]

    for change in (lambda c: mixer(1)(c)["mask"].update(size=22), lambda c: mixer(1)(c)["mask"].update(keep_first=4),
                   lambda c: mixer(1)(c)["mask"].update(keep_first=6), lambda c: mixer(3)(c)["mask"].update(keep_first=0),
                   lambda c: mixer(3)(c)["mask"].update(size=6), lambda c: mixer(1)(c)["rot"].pop("scaling"),
                   lambda c: mixer(1)(c)["rot"]["scaling"].update(factor=5.0), lambda c: mixer(1)(c)["rot"]["scaling"].update(slow=3.0),
                   lambda c: mixer(2)(c)["rot"].update(base=100.0), lambda c: mixer(2)(c).update(decay=[0.9, 0.97, 0.99]),
                   lambda c: c.update(loop={"start": 1, "stop": 3, "times": 1}), lambda c: c.update(logit_scale=0.5),
                   lambda c: c.update(logit_softcap=9.0)):
        assert moved(change) > 0.01
    for name, change in (("l0.mix.dt_bias", lambda t: t.add_(1.0)), ("l0.mix.A_log", lambda t: t.add_(1.0)), ("l0.mix.b", lambda t: t.zero_()),
                         ("l0.mix.q.conv", lambda t: t[:, 0].zero_()), ("l1.mix.q.norm", lambda t: t.fill_(1.0)),
                         ("l1.mix.k.norm", lambda t: t.fill_(1.0)), ("l2.mix.g", lambda t: t.zero_()), ("l0.mix.norm", lambda t: t.fill_(1.0))):
        t = w[name].clone()
        change(t)
        assert float((plain.forward(config, dict(w, **{name: t}), tokens) - want).abs().max()) > 0.01, name


def test_the_input_rows_are_added_once_a_pass_and_every_norm_takes_the_mean_off():
    config, w = _model("C")
    tokens = tokens_for(config, 30, salt=4)
    _, kept = plain.forward(config, w, tokens, keep_layers=True)
    rows = w["embed"][torch.tensor(tokens)]
    per = len(config["layers"])
    layer = config["layers"][0]
    for p in (1, 2):
        x = kept[p * per - 1] + rows
        want = x + plain.retention(plain.layer_norm(x, w["l0.norm1"], config["norm"]["eps"]), plain.sub(w, "l0.mix"), layer["mixer"],
                                   config["norm"]["eps"])
        assert torch.allclose(kept[p * per], want, atol=1e-12)
    shifted = plain.layer_norm(rows + 3.0, w["l0.norm1"], config["norm"]["eps"])
    assert torch.allclose(shifted, plain.layer_norm(rows, w["l0.norm1"], config["norm"]["eps"]), atol=1e-9)


def test_the_visible_positions():
    # size 3, first 2 kept: position 6 sees 0, 1 and 4, 5, 6
    seen = plain.visible(8, 3, 2)
    assert seen[6].tolist() == [True, True, False, False, True, True, True, False]
    assert seen[1].tolist() == [True, True] + [False] * 6
    assert plain.visible(5, 1, 0).tolist() == torch.eye(5, dtype=torch.bool).tolist()
    assert plain.visible(5, 1, 9).tolist() == torch.ones(5, 5).tril().bool().tolist()
