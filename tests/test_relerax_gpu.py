"""Relerax through the framework against the plain implementation (``tests/plain/relerax_plain.py``): each mechanism alone,
the residual behind every layer, whole prompts, token-by-token decoding through the captured steps, portions down to two
tokens, unequal requests in one batch against each alone, pages that are given back and used again, long decoding (windows
pass while tokens are decoded, latents stay), and greedy generation through the engine's own entry point and scheduler.
Four small configurations that differ in every size (``relerax_configs``); weights are drawn so that attention is peaked,
and the tests of the mechanisms alone first show, with the plain implementation, that a window one off, the one left out
of the denominator, values that turn with their keys, another pairing or a gate left open would be seen.  Router choices
are no close calls (``relerax_configs.steady_routing``; the margins are asserted).

Tolerances are derived: the float32 engine may be off by a multiple of what float32 arithmetic costs the plain
implementation itself (float32 against float64); the bfloat16 engine by 3 times what rounding the activations to bfloat16,
where a bfloat16 run stores them, costs the plain implementation."""

import functools

import pytest
import torch

from clockwork_b200 import EngineConfig, ops
from clockwork_b200.config import PartSpec
from clockwork_b200.engine import LLMEngine
from clockwork_b200.engine.trace import TraceSession
from clockwork_b200.ops import gemm as gemm_ops
from clockwork_b200.ops import grouped as grouped_ops
from clockwork_b200.ops import latent as latent_ops
from clockwork_b200.parts import build_part
from clockwork_b200.parts.base import ResidualStream
from clockwork_b200.sampling import SamplingParams
from clockwork_b200.weights.loader import make_fetch
from tests import relerax_configs
from tests.gpu_tools import DEV, PartHarness
from tests.plain import relerax_plain as plain
from tests.relerax_configs import CONFIGS, MARGIN, tokens_for, write_model
from tests.trace_tools import cut

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]


@pytest.fixture(scope="module")
def dirs(tmp_path_factory):
    return {name: write_model(tmp_path_factory.mktemp(f"relerax_{name}"), name, seed=5 + i, steady=True) for i, name in enumerate(sorted(CONFIGS))}


@pytest.fixture(scope="module")
def oracle(dirs):
    """(name, tokens) -> (float64 logits [T, V], what float32 costs, what bfloat16 storage costs)."""
    weights = {name: plain.read_model_dir(folder, dtype=torch.float64) for name, folder in dirs.items()}

    @functools.lru_cache(maxsize=None)
    def get(name, tokens):
        config, w = weights[name]
        margins: list = []
        exact = plain.forward(config, w, list(tokens), dtype=torch.float64, margins=margins)
        assert min(margins) > MARGIN
        single = plain.forward(config, w, list(tokens), dtype=torch.float32).double()
        rounded = plain.forward(config, w, list(tokens), dtype=torch.float64, rnd=plain.to_bfloat16_and_back)
        return exact, float((single - exact).abs().max()), float((rounded - exact).abs().max())

    return get


def check(got, name, tokens, dtype, oracle, first=0):
    exact, cost32, cost16 = oracle(name, tuple(tokens))
    diff = (got.double().cpu() - exact[first : first + got.shape[0]]).abs()
    allowed = 30 * cost32 + 1e-5 if dtype == "float32" else 3 * cost16
    worst = float(diff.max())
    assert worst <= allowed, f"{name} {dtype}: off by {worst:.3g} at position {first + int(diff.max(1).values.argmax())}, allowed {allowed:.3g}"


class Replay:
    """Steps through ``TraceSession`` (what ``bin/trace_run`` runs), logits wanted everywhere."""

    def __init__(self, folder, name, dtype, max_tokens, **kw):
        self.session = TraceSession(folder, dtype, max_tokens, page_size=CONFIGS[name][1], **kw)
        self.logits: dict[str, list] = {}
        self.n = 0

    def step(self, portions: dict, end=()):
        record = {"step": self.n, "end": list(end),
                  "entries": [{"id": rid, "tokens": toks, "want": list(range(len(toks)))} for rid, toks in portions.items()]}
        self.n += 1
        out, _ = self.session.run_step(record)
        row = 0
        for rid, toks in portions.items():
            self.logits.setdefault(rid, []).append(torch.from_numpy(out[row : row + len(toks)].copy()))
            row += len(toks)

    def of(self, rid):
        return torch.cat(self.logits[rid])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompt(name, dtype, dirs, oracle):
    tokens = tokens_for(CONFIGS[name][0], 75, 1)
    run = Replay(dirs[name], name, dtype, 128)
    run.step({"a": tokens}, end=["a"])
    check(run.of("a"), name, tokens, dtype, oracle)


@pytest.mark.parametrize("length", [40, 300])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_the_residual_behind_every_layer(name, length, dirs):
    """float32, layer by layer; 300 rows go through the norms' kernel of many rows."""
    config, w = plain.read_model_dir(dirs[name], dtype=torch.float64)
    tokens = tokens_for(CONFIGS[name][0], length, 11)
    _, want = plain.forward(config, w, tokens, dtype=torch.float64, keep_layers=True)
    _, single = plain.forward(config, w, tokens, dtype=torch.float32, keep_layers=True)
    run = Replay(dirs[name], name, "float32", 512, graphs=False)
    seen = []
    for block in run.session.model.blocks:
        def wrapped(ctx, stream, view, *args, _inner=block.forward, **kw):
            out = _inner(ctx, stream, view, *args, **kw)
            stream.flush()
            seen.append(stream.residual.clone())
            return out
        block.forward = wrapped
    run.step({"a": tokens}, end=["a"])
    assert len(seen) == want.shape[0] == len(config["layers"])
    for r, got in enumerate(seen):
        allowed = 30 * float((single[r].double() - want[r]).abs().max()) + 1e-5
        assert float((got.double().cpu() - want[r]).abs().max()) <= allowed, f"behind layer {r}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prefill_then_token_by_token(name, dtype, dirs, oracle):
    """The decoded tokens run through the captured single-token steps; the first tokens of a sequence too (a prompt of one
    token).  70 tokens pass every window but the longest."""
    tokens = tokens_for(CONFIGS[name][0], 70, 2)
    for start in (9, 1):
        run = Replay(dirs[name], name, dtype, 128)
        run.step({"a": tokens[:start]})
        for t in tokens[start:]:
            run.step({"a": [t]})
        assert run.session.uses_graphs
        check(run.of("a"), name, tokens, dtype, oracle)


@pytest.mark.parametrize("graphs", [True, False])
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_portions_of_many_sizes(name, dtype, graphs, dirs, oracle):
    """Cuts in the middle of pages and of windows; portions of two and three tokens, of one page, longer than a window."""
    tokens = tokens_for(CONFIGS[name][0], 90, 3)
    for sizes in ([2, 3, 1, 7, 2, 16, 5, 4], [37, 2, 2, 2, 30, 1, 1, 3]):
        run = Replay(dirs[name], name, dtype, 128, graphs=graphs)
        for portion in cut(tokens, sizes):
            run.step({"a": portion})
        check(run.of("a"), name, tokens, dtype, oracle)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_unequal_requests_in_one_batch_against_each_alone(name, dtype, dirs, oracle):
    prompts = {"p": tokens_for(CONFIGS[name][0], 61, 4), "q": tokens_for(CONFIGS[name][0], 23, 5), "r": tokens_for(CONFIGS[name][0], 40, 6), "s": tokens_for(CONFIGS[name][0], 9, 7)}
    plans = {"p": [17, 2, 1, 1, 30, 1, 1, 1, 7], "q": [1, 1, 1, 5, 1, 2, 12], "r": [40], "s": [2, 1, 1, 1, 1, 1, 1, 1]}
    cuts = {rid: cut(toks, plans[rid]) for rid, toks in prompts.items()}
    together = Replay(dirs[name], name, dtype, 4 * 64)
    for i in range(max(len(c) for c in cuts.values())):
        step = {rid: c[i] for rid, c in cuts.items() if i < len(c)}
        together.step(step, end=[rid for rid, c in cuts.items() if i == len(c) - 1])
    for rid, toks in prompts.items():
        alone = Replay(dirs[name], name, dtype, 64)
        for portion in cuts[rid]:
            alone.step({rid: portion})
        if dtype == "float32":  # a row's result does not depend on the rest of the batch at all
            assert torch.equal(together.of(rid), alone.of(rid)), rid
        check(together.of(rid), name, toks, dtype, oracle)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_slots_and_pages_given_back_and_used_again(name, dtype, dirs, oracle):
    """Ten requests, at most four at a time, through a pool of pages for 4 x 64 tokens: a request that takes a page that
    another one left sees none of the other's keys."""
    run = Replay(dirs[name], name, dtype, 4 * 64)
    prompts = {f"r{i}": tokens_for(CONFIGS[name][0], 20 + 4 * i, 20 + i) for i in range(10)}
    waiting, live, at = list(prompts), [], {}
    while waiting or live:
        while waiting and len(live) < 4:
            live.append(waiting.pop(0))
            at[live[-1]] = 0
        step, done = {}, []
        for k, rid in enumerate(live):
            n = min([13, 1, 2, 5][(k + at[rid]) % 4], len(prompts[rid]) - at[rid])
            step[rid] = prompts[rid][at[rid] : at[rid] + n]
            at[rid] += n
            if at[rid] == len(prompts[rid]):
                done.append(rid)
        run.step(step, end=done)
        live = [rid for rid in live if rid not in done]
    run.session.cache.check_invariants()
    assert not run.session.cache.requests and all(g.allocator.num_free == g.allocator.num_pages for g in run.session.cache.groups)
    for rid, toks in prompts.items():
        check(run.of(rid), name, toks, dtype, oracle)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "C"])
def test_long_decoding_while_windows_pass(name, dtype, dirs, oracle):
    """300 decoded tokens behind a short prompt: windows move over decoded tokens and the pages behind them go back to the
    pool while the request runs; the latents of all tokens stay."""
    tokens = tokens_for(CONFIGS[name][0], 320, 8)
    run = Replay(dirs[name], name, dtype, 320)
    run.step({"a": tokens[:20]})
    for t in tokens[20:]:
        run.step({"a": [t]})
    req = run.session.cache.get("a")
    page = CONFIGS[name][1]
    for group, table in zip(run.session.cache.groups, req.tables):
        held = sum(p >= 0 for p in table)
        assert held == -(-320 // page) if group.need.window is None else held <= group.need.window // page + 2
    check(run.of("a"), name, tokens, dtype, oracle)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_greedy_generation_through_the_engine(name, dtype, dirs):
    """The engine's own entry point and scheduler: prompts cut under a small token budget, several requests at once."""
    config, page = CONFIGS[name]
    cfg = EngineConfig.defaults(str(dirs[name]), dtype=dtype, block_size=page, num_blocks=256, max_model_len=256, max_num_seqs=4,
                                max_num_batched_tokens=24)
    engine = LLMEngine(cfg)
    prompts = [tokens_for(CONFIGS[name][0], n, 30 + n) for n in (5, 31, 18, 1, 44)]
    outs = engine.generate(prompts, SamplingParams(max_tokens=12, ignore_eos=True))
    _, w = plain.read_model_dir(dirs[name], dtype=torch.float64)
    for tokens, out in zip(prompts, outs):
        got = list(out.token_ids)
        logits = plain.forward(config, w, tokens + got, dtype=torch.float64)
        single = plain.forward(config, w, tokens + got, dtype=torch.float32).double()
        rounded = plain.forward(config, w, tokens + got, dtype=torch.float64, rnd=plain.to_bfloat16_and_back)
        # every token is within rounding of the best one, given the engine's own history
        yard = 60 * float((single - logits).abs().max()) + 2e-5 if dtype == "float32" else 6 * float((rounded - logits).abs().max())
        for i, token in enumerate(got):
            row = logits[len(tokens) + i - 1]
            assert float(row.max() - row[token]) <= yard
        if dtype == "float32" and all(float(r.topk(2).values.diff().abs()) > yard for r in logits[len(tokens) - 1 : -1]):
            assert got == plain.greedy(config, w, tokens, 12)


# ---- every mechanism alone ----------------------------------------------------------------------------

def part_with_weights(category, spec, prefix, dtype, tensors):
    part = build_part(category, spec, prefix, dtype, DEV)
    decls = {d.name: d for d in part.tensor_decls()}
    assert set(decls) == set(tensors), (sorted(decls), sorted(tensors))
    part.load_weights(make_fetch(lambda n: tensors[n], decls, dtype, DEV))
    return part


def run_mixer(part, x, portions, page_size=4, num_pages=128):
    """The mixer's output for every row of ``x`` [T, W], fed in portions through a cache of its own."""
    harness = PartHarness({0: part.cache_need()}, part.dtype, num_pages=num_pages, page_size=page_size, slots=2)
    out, at = [], 0
    for n in portions:
        prepared = harness.prepare({"a": n})
        got = part.mix(prepared.ctx, x[at : at + n].to(DEV, part.dtype).contiguous(), prepared.ctx.views[0])
        harness.commit(prepared)
        out.append(got.float().cpu())
        at += n
        req = harness.cache.get("a")
        harness.cache.release_behind_window(req, req.num_computed)
    assert at == x.shape[0]
    return torch.cat(out)


def draw(gen, shape, scale=1.0, shift=0.0):
    return (shift + scale * torch.randn(shape, generator=gen)).to(torch.bfloat16).float()


def assert_close(got, want, what, rel=3e-5):
    """float32 arithmetic against float64: a few units of float32 rounding of the largest value, per term summed."""
    worst, allowed = float((got.double() - want).abs().max()), 2e-4 + rel * float(want.abs().max())
    assert worst <= allowed, f"{what}: off by {worst:.3g}, allowed {allowed:.3g}"


def named(tensors, prefix="m"):
    return {f"{prefix}.{k}": v for k, v in tensors.items()}


def doubled(tensors):
    return {k: v.double() for k, v in tensors.items()}


def attention_tensors(gen, w, m, peak=0.3):
    h, g, d = m["heads"], m["kv_heads"], m["dim"]
    return {"q": draw(gen, (h * d, w), peak), "k": draw(gen, (g * d, w), peak), "g": draw(gen, (h * d, w), 0.3), "o": draw(gen, (w, h * d), 0.2)}


def attention_spec(w, m):
    return PartSpec("window_attention", dict(hidden_size=w, heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["dim"],
                                             scale=m["scale"], weights="softmax", window=m["mask"]["size"], sink="zero", values="keys",
                                             gate="entry", rotary=dict(m["rot"], pairing="interleaved")))


def attention_config(*args):
    return relerax_configs.attention(*args)["mixer"]


@pytest.mark.parametrize("heads, kv_heads, dim, size, rot, base, scaling, page", [
    (4, 2, 24, 21, 8, 1000.0, (4.0, 60, 6.0, 1.0), 4), (3, 1, 16, 7, 16, 50000.0, None, 8), (6, 6, 8, 1, 2, 10000.0, None, 4),
    (2, 2, 12, 400, 12, 100.0, (8.0, 32, 4.0, 2.0), 16), (8, 2, 32, 100, 32, 10000.0, (2.0, 300, 20.0, 1.0), 16),
    (5, 5, 17, 64, 6, 300.0, None, 16), (12, 3, 48, 60, 16, 500000.0, (4.0, 100, 8.0, 0.5), 16), (33, 11, 8, 10, 6, 20.0, None, 4)])
def test_a_window_whose_values_are_its_keys_alone(heads, kv_heads, dim, size, rot, base, scaling, page):
    """300 positions whole, token by token and in portions that cut pages and windows, the pages behind the window given back
    on the way.  First the plain implementation shows what counts: a window one off, the one in the denominator, values that
    turn with their keys, gates, an amplitude left out."""
    gen = torch.Generator().manual_seed(heads * 100 + size)
    w, eps = 48, 1e-5
    m = attention_config(heads, kv_heads, dim, 0.25, size, rot, base, scaling)
    t = attention_tensors(gen, w, m)
    wd = doubled(t)
    x = draw(gen, (300, w))
    want = plain.window_attention(x.double(), wd, m, eps)

    def moved(other, weights=wd):
        return float((plain.window_attention(x.double(), weights, other, eps) - want).abs().max())

    for other in (size - 1, size + 1):
        if 1 <= other < 300:
            assert moved(dict(m, mask={"size": other})) > 0.02
    if scaling is not None:
        assert moved(dict(m, rot={"dims": rot, "base": base})) > 0.02
    assert moved(m, dict(wd, g=wd["g"] * 0)) > 0.02
    if size > 1:  # (of a lone key, turned by its own angle, the score does not tell)
        with_softmax = plain.weights_with_one
        try:
            plain.weights_with_one = lambda s: torch.softmax(s, -1)
            assert moved(m) > 0.02
        finally:
            plain.weights_with_one = with_softmax
    part = part_with_weights("mixer", attention_spec(w, m), "m", torch.float32, named(t))
    for portions in ([131, 169], [1] * 300, [2, 3, 1, 1, 9, 2, 5, 41, 100, 1, 1, 1, 131, 2], [page - 1, 2, page, 1, 300 - 2 * page - 2]):
        assert sum(portions) == 300
        got = run_mixer(part, x, portions, page_size=page, num_pages=300 // page + 8)
        assert_close(got, want, portions)


@pytest.mark.parametrize("heads, kv_heads, dim, size, rot, page", [
    (4, 4, 256, 100, 128, 16), (8, 8, 64, 130, 64, 64), (16, 1, 64, 40, 64, 16), (8, 2, 128, 150, 64, 16), (6, 3, 96, 45, 40, 8),
    (4, 1, 240, 70, 16, 16), (4, 4, 32, 33, 24, 16), (16, 4, 128, 300, 128, 16), (12, 12, 48, 77, 8, 16), (8, 2, 64, 5000, 32, 16)])
def test_a_window_whose_values_are_its_keys_in_bfloat16_on_the_tensor_cores(heads, kv_heads, dim, size, rot, page):
    """Sizes that take each arrangement of the tensor-core kernel (windows that are cut in parts among them: few rows, windows
    over 256), whole and in portions, against the plain implementation in float64; allowed is 3 times what rounding q, k, v and
    the output to bfloat16 costs the plain implementation."""
    gen = torch.Generator().manual_seed(heads * 100 + size)
    w, eps = 64, 1e-5
    m = attention_config(heads, kv_heads, dim, dim ** -0.5, size, rot, 10000.0, (4.0, 128, 16.0, 1.0))
    t = attention_tensors(gen, w, m, peak=0.2)
    wd = doubled(t)
    x = draw(gen, (400, w))
    want = plain.window_attention(x.double(), wd, m, eps)
    rounded = plain.to_bfloat16_and_back(plain.window_attention(x.double(), wd, m, eps, rnd=plain.to_bfloat16_and_back))
    allowed = 3 * float((rounded - want).abs().max()) + 0.01 * float(want.abs().max())
    assert allowed < 0.15 * float(want.abs().max())
    part = part_with_weights("mixer", attention_spec(w, m), "m", torch.bfloat16, named(t))
    for portions in ([400], [340] + [1] * 60, [3, 64, 1, 61, 2, 249] + [1] * 20):
        got = run_mixer(part, x, portions, page_size=page, num_pages=400 // page + 8)
        worst = float((got.double() - want).abs().max())
        assert worst <= allowed, f"{portions[:6]}: off by {worst:.3g}, allowed {allowed:.3g}"


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_keys_that_stand_out_at_the_edge_of_the_window(dtype):
    """A query and two keys are made so that their scores tower over all others: the window's far edge takes the whole
    softmax, the position behind it, as strong, is not seen, in a prompt and in decoding, also where a portion ends at the
    edge and after the pages behind it have been given back."""
    heads, kv_heads, dim, size, w, rot, eps = 2, 1, 16, 37, 32, 4, 1e-5
    gen = torch.Generator().manual_seed(9)
    m = attention_config(heads, kv_heads, dim, 1.0, size, rot, 1000.0)
    t = attention_tensors(gen, w, m, peak=0.1)
    x = draw(gen, (120, w))
    for name, col, other, count in (("q", 3, 5, heads), ("k", 5, 3, kv_heads)):
        t[name].view(count, dim, w)[:, rot:, col] = 0.5   # unrotated entries of a towering row all point one way
        t[name].view(count, dim, w)[:, :rot, col] = 0.0
        t[name].view(count, dim, w)[:, :, other] = 0.0
    x[:, 3] = x[:, 5] = 0.0
    probe = 100
    inside, outside = probe - size + 1, probe - size
    x[probe, 3] = 8.0
    x[[inside, outside], 5] = 8.0
    wd = doubled(t)
    want = plain.window_attention(x.double(), wd, m, eps)
    value = (x[inside].double() @ wd["k"].T).repeat(heads) * torch.sigmoid(x[probe].double() @ wd["g"].T)
    assert float((value @ wd["o"].T - want[probe]).abs().max()) < 1e-6  # the edge's key takes it all
    rounded = plain.to_bfloat16_and_back(plain.window_attention(x.double(), wd, m, eps, rnd=plain.to_bfloat16_and_back))
    allowed = 3 * float((rounded - want)[probe].abs().max())
    for other in (size + 1, size - 1):
        assert float((plain.window_attention(x.double(), wd, dict(m, mask={"size": other}), eps) - want)[probe].abs().max()) > 2 * allowed
    part = part_with_weights("mixer", attention_spec(w, m), "m", dtype, named(t))
    for portions in ([120], [probe, 1, 19], [inside, 20, 16, 1, 19], [outside, 1, 1, 35, 1, 19], [70] + [1] * 50, [1] * 120):
        assert sum(portions) == 120
        got = run_mixer(part, x, portions, page_size=8)
        if dtype == torch.float32:
            assert_close(got, want, portions)
        else:
            assert float((got.double() - want)[probe].abs().max()) < allowed, portions


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_one_in_the_denominator_against_a_lone_key(dtype):
    """Position 0 and, with a window of one, every position see one key: its weight is a sigmoid of the score, anything
    between nought and one; with scores far below zero nothing is left, far above everything."""
    heads, kv_heads, dim, w, rot, eps = 4, 2, 16, 32, 8, 1e-5
    gen = torch.Generator().manual_seed(12)
    m = attention_config(heads, kv_heads, dim, 0.1, 1, rot, 100.0)
    t = attention_tensors(gen, w, m)
    x = draw(gen, (60, w))
    x[40:50] *= 12.0
    wd = doubled(t)
    want = plain.window_attention(x.double(), wd, m, eps)
    q, k = (x.double() @ wd["q"].T).reshape(60, heads, dim), (x.double() @ wd["k"].T).reshape(60, kv_heads, dim)
    share = torch.sigmoid(0.1 * (q * k.repeat_interleave(2, 1)).sum(-1))
    assert float(share.min()) < 1e-6 and float(share.max()) > 1 - 1e-6 and float((share - 0.5).abs().min()) < 0.05
    part = part_with_weights("mixer", attention_spec(w, m), "m", dtype, named(t))
    rounded = plain.to_bfloat16_and_back(plain.window_attention(x.double(), wd, m, eps, rnd=plain.to_bfloat16_and_back))
    for portions in ([60], [1] * 60, [2, 30, 3, 25]):
        got = run_mixer(part, x, portions)
        if dtype == torch.float32:
            assert_close(got, want, portions)
        else:
            assert float((got.double() - want).abs().max()) <= 3 * float((rounded - want).abs().max())


def latent_config(*args):
    return relerax_configs.latent(*args)["mixer"]


def latent_tensors(gen, w, m, peak=0.6):
    h, d, r, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    return {"q": draw(gen, (h * (d + r), w), peak), "dkv": draw(gen, (rank + r, w), 0.4), "dkv.norm": draw(gen, (rank,), 0.2, 1.0),
            "uk": draw(gen, (h * d, rank), 1.2 / rank ** 0.5), "uv": draw(gen, (h * dv, rank), 1.2 / rank ** 0.5), "g": draw(gen, (h, w), 0.3),
            "o": draw(gen, (w, h * dv), 0.2)}


def latent_spec(w, m, eps):
    return PartSpec("latent_attention", dict(hidden_size=w, heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"],
                                             kv_rank=m["kv_rank"], q_rank=None, scale=m["scale"], sink=False, gate="head", eps=eps,
                                             rope_base=m["rot"]["base"], pairing="interleaved", scaling=m["rot"].get("scaling")))


@pytest.mark.parametrize("heads, dim, rot, vdim, rank, base, scaling, page", [
    (3, 24, 8, 20, 40, 300.0, (4.0, 60, 6.0, 1.0), 4), (1, 16, 16, 16, 16, 10000.0, None, 16), (5, 8, 4, 12, 136, 50.0, (8.0, 32, 4.0, 2.0), 8),
    (6, 17, 2, 9, 23, 300.0, None, 4), (20, 16, 32, 24, 256, 5000.0, (2.0, 128, 8.0, 0.25), 16), (2, 8, 16, 40, 520, 1000.0, None, 16)])
def test_attention_over_a_latent_alone(heads, dim, rot, vdim, rank, base, scaling, page):
    """Peaked attention over 300 keys: most queries put most of their weight on one key far back, somewhere in another page.
    First the plain implementation shows that the rotation's amplitude, gates, keys more than a hundred tokens back and the
    norm's weights would be missed."""
    gen = torch.Generator().manual_seed(rank)
    w, eps = 48, 1e-5
    m = latent_config(heads, dim, rot, vdim, rank, 0.3, base, scaling)
    t = latent_tensors(gen, w, m)
    wd = doubled(t)
    x = draw(gen, (300, w))
    want = plain.latent_attention(x.double(), wd, m, eps)

    def moved(other, weights=wd):
        return float((plain.latent_attention(x.double(), weights, other, eps) - want).abs().max())

    if scaling is not None:
        assert moved(dict(m, rot={"dims": rot, "base": base})) > 0.02
    assert moved(m, dict(wd, g=wd["g"] * 0)) > 0.02 and moved(m, dict(wd, **{"dkv.norm": wd["dkv.norm"] * 0 + 1})) > 0.02
    fresh = plain.latent_attention(x[100:].double(), wd, m, eps)
    assert float((want[100:] - fresh).abs().max()) > 0.05
    part = part_with_weights("mixer", latent_spec(w, m, eps), "m", torch.float32, named(t))
    for portions in ([300], [129, 1, 1, 2, 127, 40], [page - 1, 2, page, 1, 300 - 2 * page - 2], [1] * 150 + [150]):
        assert_close(run_mixer(part, x, portions, page_size=page), want, portions[:6])


@pytest.mark.parametrize("q_rank, sink, gate, pairing", [(None, True, "entry", "half"), (24, False, "head", "interleaved"), (24, True, "head", "half")])
def test_the_switches_of_attention_over_a_latent_go_together(q_rank, sink, gate, pairing):
    """Combinations that no design here uses: queries through a latent of their own with gates per head, queries straight from
    the input with a sink and gates per entry."""
    gen = torch.Generator().manual_seed(5)
    w, eps = 40, 1e-5
    m = latent_config(3, 12, 8, 10, 24, 0.3, 100.0, None)
    h, d, r, dv = 3, 12, 8, 10
    t = latent_tensors(gen, w, m)
    if q_rank is not None:
        del t["q"]
        t.update({"dq": draw(gen, (q_rank, w), 0.3), "dq.norm": draw(gen, (q_rank,), 0.2, 1.0), "uq": draw(gen, (h * (d + r), q_rank), 0.8)})
    if sink:
        t["sink"] = draw(gen, (h,), 1.0, 1.0)
    if gate == "entry":
        t["g"] = draw(gen, (h * dv, w), 0.3)
    part = part_with_weights("mixer", PartSpec("latent_attention", dict(
        hidden_size=w, heads=h, dim=d, rot_dim=r, vdim=dv, kv_rank=24, q_rank=q_rank, scale=0.3, sink=sink, gate=gate, eps=eps,
        rope_base=100.0, pairing=pairing)), "m", torch.float32, named(t))
    x = draw(gen, (90, w))
    xd, wd = x.double(), doubled(t)
    q = (plain.rms_norm(xd @ wd["dq"].T, wd["dq.norm"], eps) @ wd["uq"].T if q_rank else xd @ wd["q"].T).reshape(90, h, d + r)
    down, positions = xd @ wd["dkv"].T, torch.arange(90)

    def turn(y):
        if pairing == "interleaved":
            return plain.rotate(y, positions, m["rot"])
        swapped = torch.stack([y[..., : r // 2], y[..., r // 2 :]], -1).flatten(-2)
        out = plain.rotate(swapped, positions, m["rot"])
        return torch.cat([out[..., 0::2], out[..., 1::2]], -1)

    c = plain.rms_norm(down[:, :24], wd["dkv.norm"], eps)
    scores = 0.3 * (torch.einsum("thd,shd->hts", q[..., :d], (c @ wd["uk"].T).reshape(90, h, d))
                    + torch.einsum("thd,sd->hts", turn(q[..., d:]), turn(down[:, None, 24:])[:, 0]))
    scores = scores.masked_fill(~plain.visible(90, 90), float("-inf"))
    if sink:
        scores = torch.cat([scores, wd["sink"][:, None, None].expand(h, 90, 1)], -1)
    p = torch.softmax(scores, -1)[..., :90]
    o = torch.einsum("hts,shd->thd", p, (c @ wd["uv"].T).reshape(90, h, dv))
    z = torch.sigmoid(xd @ wd["g"].T)
    o = (o * (z.reshape(90, h, dv) if gate == "entry" else z[..., None])).reshape(90, h * dv)
    want = o @ wd["o"].T
    for portions in ([90], [1] * 20 + [70]):
        assert_close(run_mixer(part, x, portions), want, portions[:3])


@pytest.mark.parametrize("heads, dim, rot, rank, page", [(16, 32, 16, 64, 16), (20, 24, 8, 136, 8), (3, 64, 64, 512, 16), (33, 16, 32, 96, 64),
                                                          (8, 128, 64, 448, 16), (1, 16, 16, 16, 16), (16, 8, 48, 208, 16)])
def test_attention_over_a_latent_in_bfloat16_on_the_tensor_cores(heads, dim, rot, rank, page):
    """Each arrangement of the tensor-core kernel: heads that do not fill a tile and that need several, latents whose columns
    do not share out evenly; whole prompts, portions that end within a tile of queries or keys, single tokens behind contexts
    that are cut in parts.  Beside the plain implementation the CUDA-core form."""
    gen = torch.Generator().manual_seed(heads + rank)
    w, eps, vdim = 64, 1e-5, 24
    m = latent_config(heads, dim, rot, vdim, rank, 0.35 * (24 / (dim + rot)) ** 0.5, 3000.0, (4.0, 128, 16.0, 1.0))
    t = latent_tensors(gen, w, m)
    wd = doubled(t)
    x = draw(gen, (700, w))
    want = plain.latent_attention(x.double(), wd, m, eps)
    yard = float((plain.latent_attention(x.double(), wd, m, eps, rnd=plain.to_bfloat16_and_back) - want).abs().max())
    assert yard < 0.1 * float(want.abs().max())
    part = part_with_weights("mixer", latent_spec(w, m, eps), "m", torch.bfloat16, named(t))
    for portions in ([700], [63, 1, 1, 2, 64, 69, 3, 97, 100, 300], [660] + [1] * 40, [5, 8, 650, 7, 30]):
        outs = []
        for on in (True, False):
            latent_ops.set_tensor_cores(on)
            try:
                outs.append(run_mixer(part, x, portions, page_size=page))
            finally:
                latent_ops.set_tensor_cores(True)
        fast, slow = outs
        for got in outs:
            assert float((got.double() - want).abs().max()) <= 3 * yard, portions[:6]
        assert float((fast - slow).abs().max()) <= 1.5 * yard, portions[:6]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_one_latent_far_back_among_hundreds(dtype):
    """One key, in the first page or at a page's edge, stands out for a late query; whole, decoded, over portions, and beside
    other requests.  Lost or shifted by one, the output is another."""
    heads, dim, rot, vdim, rank, w, eps = 4, 32, 16, 16, 48, 32, 1e-5
    gen = torch.Generator().manual_seed(10)
    m = latent_config(heads, dim, rot, vdim, rank, 1.0, 1000.0, (4.0, 256, 8.0, 1.0))
    t = latent_tensors(gen, w, m, peak=0.05)
    t["dkv"][:, 5] = 0.0
    t["dkv"][0, 5] = 1.0  # a row with a large coordinate 5 has a latent that is its first entry only
    t["q"][:, 3] = 0.0
    t["q"].view(heads, dim + rot, w)[:, 0, 3] = 1.0
    t["uk"].view(heads, dim, rank)[:, 0, 0] = 2.0
    for far in (3, 15, 16, 127):
        x = draw(gen, (900, w))
        x[:, 3] = x[:, 5] = 0.0
        x[852, 3], x[far, 5] = 12.0, 400.0
        wd = doubled(t)
        want = plain.latent_attention(x.double(), wd, m, eps)
        c = plain.rms_norm(x[far].double() @ wd["dkv"][:rank].T, wd["dkv.norm"], eps)
        value = (c @ wd["uv"].T).reshape(heads, vdim) * torch.sigmoid(x[852].double() @ wd["g"].T)[:, None]
        assert float((value.reshape(-1) @ wd["o"].T - want[852]).abs().max()) < 1e-3 * float(want[852].abs().max())
        part = part_with_weights("mixer", latent_spec(w, m, eps), "m", dtype, named(t))
        yard = float((plain.latent_attention(x.double(), wd, m, eps, rnd=plain.to_bfloat16_and_back) - want)[852].abs().max())
        assert float(want[852].abs().max()) > 30 * yard
        for portions in ([900], [840] + [1] * 60, [1, 4, 300, 545, 3, 1, 46]):
            got = run_mixer(part, x, portions, page_size=16)
            if dtype == torch.float32:
                assert_close(got, want, portions[:3])
            else:
                assert float((got.double() - want)[852].abs().max()) <= 3 * yard, portions[:3]


def run_ffn(part, x, rows, dtype):
    harness = PartHarness({}, dtype)
    prepared = harness.prepare({f"r{rows}": rows})
    stream = ResidualStream(torch.ones((rows, x.shape[1]), dtype=torch.float32, device=DEV))
    stream.push(part.forward(prepared.ctx, x[:rows].to(DEV, dtype).contiguous(), stream))
    stream.flush()
    ops.raise_on_status(harness.status)
    return stream.residual.cpu().double() - 1.0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("experts, top, identity, ff, w", [(5, 2, 1, 28, 40), (4, 4, 0, 17, 40), (3, 4, 3, 24, 36), (2, 1, 6, 20, 40), (33, 5, 7, 40, 64),
                                                           (11, 3, 2, 136, 256)])
def test_experts_some_of_which_hand_their_input_on_alone(experts, top, identity, ff, w, dtype):
    """Corrected softmax scores, weights that sum to one, identity experts; where few are chosen some tokens choose nothing
    but identity experts.  Rows whose margins are thin are left out of the comparison."""
    gen = torch.Generator().manual_seed(experts * 10 + identity)
    outputs = experts + identity
    t = {"router": draw(gen, (outputs, w), 0.35), "correction": draw(gen, (outputs,), 0.1)}
    for e in range(experts):
        t.update({f"e{e}.up": draw(gen, (ff, w), 0.3), f"e{e}.down": draw(gen, (w, ff), 0.2)})
    part = part_with_weights("ffn", PartSpec("moe", dict(hidden_size=w, expert_size=ff, experts=experts, top=top, identity=identity, gated=False,
                                                         scoring="all", correction=True, renormalize=True, router_bias=False)),
                             "f", dtype, named(t, "f"))
    x, wd = draw(gen, (300, w)), doubled(t)
    cfg = {"router": {"experts": experts, "top": top, "identity": identity}}
    want = plain.mixture(x.double(), wd, cfg)
    chosen, _, margin = plain.route(x.double(), wd, cfg["router"])
    wide = margin > (1e-4 if dtype == torch.float32 else 2e-3)
    assert int(wide.sum()) > 200
    if identity:
        kept = (chosen >= experts).sum(-1)
        assert int((kept > 0).sum()) > 10 and (top > min(identity, 2) or int((kept == top).sum()) > 0)
    uncorrected = plain.mixture(x.double(), dict(wd, correction=wd["correction"] * 0), cfg)
    assert top == outputs or float((uncorrected - want).abs().max()) > 0.1
    allowed = 1e-4 + 1e-5 * float(want.abs().max())
    if dtype == torch.bfloat16:
        rounded = plain.mixture(x.double(), wd, cfg, rnd=plain.to_bfloat16_and_back)
        allowed = 3 * float((rounded - want).abs().max()) + 1e-3
    for rows in (300, 1, 33):
        got = run_ffn(part, x, rows, dtype)
        assert float((got - want[:rows])[wide[:rows]].abs().max()) <= allowed, rows


@pytest.mark.parametrize("w, ff", [(40, 100), (50, 33), (384, 1000), (1024, 512), (2048, 640)])
@pytest.mark.parametrize("bias", [True, False])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_squared_relu_in_the_products_epilogue(w, ff, bias, dtype):
    """Every kernel that a product of these sizes may run on: few tokens (split inner dimension), more, many (persistent
    kernels, pairs of blocks); against float64 arithmetic on the same numbers."""
    gen = torch.Generator().manual_seed(w + ff)
    t = {"up": draw(gen, (ff, w), 1.5 / w ** 0.5), "down": draw(gen, (w, ff), 1.0 / ff ** 0.5)}
    if bias:
        t.update({"up.b": draw(gen, (ff,), 0.5), "down.b": draw(gen, (w,), 0.5)})
    part = part_with_weights("ffn", PartSpec("relu2_mlp", dict(hidden_size=w, intermediate_size=ff, bias=bias)), "f", dtype, named(t, "f"))
    x = draw(gen, (700, w))
    wd = doubled(dict({"up.b": torch.zeros(ff), "down.b": torch.zeros(w)}, **t))
    act = plain.squared_relu(x.double() @ wd["up"].T + wd["up.b"])
    want = plain.dense(x.double(), wd, None)
    for rows in (1, 3, 9, 33, 130, 257, 700):
        got = part.up.squared_relu(x[:rows].to(DEV, dtype).contiguous()).cpu().double()
        step = 2 ** -8 if dtype == torch.bfloat16 else 2e-6
        assert bool(((got - act[:rows]).abs() <= step * act[:rows] + 1e-4).all()), rows
        out = run_ffn(part, x, rows, dtype)
        assert float((out - want[:rows]).abs().max()) <= (1e-4 if dtype == torch.float32 else 0.01 * float(want.abs().max())), rows


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n, w", [(3, 50), (1, 64), (300, 128), (300, 74), (257, 1000), (5, 2048), (270, 4096), (40, 5000)])
def test_two_norms_in_one_pass_with_what_is_pending(n, w, dtype):
    """Few and many rows, with nothing, a tensor and the slabs of a split product pending; the sums land in the residual, and
    the first of the two is what the norm alone makes of it."""
    gen = torch.Generator().manual_seed(n + w)
    x = torch.randn((n, w), generator=gen)
    weights = [1 + 0.2 * torch.randn(w, generator=gen) for _ in range(2)]
    delta = torch.randn((n, w), generator=gen).to(dtype)
    slabs = torch.randn((3, n + 2, w), generator=gen)
    eps = 1e-3
    norms = [part_with_weights("norm", PartSpec("rmsnorm", {"size": w, "eps": eps, "weight_suffix": ""}), f"n{i}", dtype, {f"n{i}": weights[i]})
             for i in range(2)]
    status = ops.new_status(DEV)
    cases = [(None, x), (delta.to(DEV), x + delta.float())]
    if w % 4 == 0 and w <= 4096:
        cases.append((ops.PartialSums(slabs.to(DEV), n), ((x + slabs[0, :n]) + slabs[1, :n]) + slabs[2, :n]))
    for pending, y in cases:
        stream = ResidualStream(x.to(DEV))
        stream.push(pending)
        got = norms[0].forward_with(norms[1], stream, status)
        assert torch.equal(stream.residual.cpu(), y) and stream.pending is None
        for out, weight in zip(got, weights):
            want = plain.rms_norm(y.double(), weight.double(), eps)
            assert float((out.double().cpu() - want).abs().max()) <= (3e-5 if dtype == torch.float32 else 2 ** -7 * float(want.abs().max()))
        alone = norms[0].forward(ResidualStream(y.to(DEV)), status)
        assert torch.equal(alone, got[0])
    ops.raise_on_status(status)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads, n, k", [(3, 20, 24), (8, 40, 112), (16, 128, 512)])
def test_a_gate_per_head_in_the_per_head_product(heads, n, k, dtype):
    gen = torch.Generator().manual_seed(n)
    rows = 77
    a, w = draw(gen, (rows, heads * k)), draw(gen, (heads, n, k), k ** -0.5)
    gate = torch.randn((rows, heads + 5), generator=gen)
    out = torch.empty((rows, heads * n), dtype=dtype, device=DEV)
    grouped_ops.per_head_product(a.to(DEV, dtype), k, w.to(DEV, dtype), out, n, head_gate=gate.to(DEV)[:, 2 : 2 + heads])
    want = torch.einsum("rhk,hnk->rhn", a.double().reshape(rows, heads, k), w.double()) * torch.sigmoid(gate[:, 2 : 2 + heads].double())[..., None]
    diff = (out.cpu().double().reshape(rows, heads, n) - want).abs()
    assert bool((diff <= (2 ** -8 if dtype == torch.bfloat16 else 1e-6) * want.abs() + 1e-5 + (1e-4 if dtype == torch.bfloat16 else 0)).all())
    with pytest.raises(ValueError):
        grouped_ops.per_head_product(a.to(DEV, dtype), k, w.to(DEV, dtype), out, n, head_gate=gate.to(DEV)[:, : heads - 1])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "C", "D"])
def test_the_feed_forward_on_a_second_stream_changes_nothing(name, dtype, dirs):
    """The feed-forward's kernels run on a second stream beside the mixer's: the same bits as one after the other, in
    prompts, portions and captured single-token steps."""
    from clockwork_b200.parts.parallel_block import TwoNormParallelBlock

    tokens = tokens_for(CONFIGS[name][0], 120, salt=15)
    results = []
    for concurrent in (True, False):
        TwoNormParallelBlock.concurrent = concurrent
        try:
            run = Replay(dirs[name], name, dtype, 256)
            for portion in cut(tokens, [70, 3, 17, 1, 1, 1, 1, 1, 25]):
                run.step({"a": portion})
            results.append(run.of("a"))
        finally:
            TwoNormParallelBlock.concurrent = True
    assert torch.equal(results[0], results[1])


def test_how_the_keys_of_a_latent_are_cut():
    """Few rows over a long context are cut until the blocks fill the GPU, short contexts and long portions are not; the
    scratch holds every plan."""
    for tokens, seqs, heads, portion, context, want in (
            (1, 1, 16, 1, 4096, (True, 64)), (8, 8, 16, 1, 4096, (True, 18)), (8, 8, 16, 1, 60, (True, 1)), (64, 64, 20, 1, 9000, (True, 1)),
            (2048, 1, 16, 2048, 2048, (False, 1)), (64, 1, 16, 64, 16384, (False, 8)), (3, 1, 8, 2, 5000, (True, 49))):
        few, parts = latent_ops.plan_parts(tokens, seqs, heads, portion, context)
        assert (few, parts) == want, (tokens, seqs, heads, portion, context)
        assert parts == 1 or tokens * heads * parts <= latent_ops.FILL_BLOCKS * latent_ops.TILE_ROWS[1]


def test_products_take_the_new_epilogue_only_where_it_belongs():
    x, w = torch.zeros((4, 16), device=DEV), torch.zeros((8, 16), device=DEV)
    assert gemm_ops.linear_relu2(x, w, None).shape == (4, 8)
    with pytest.raises(ValueError):
        ops.gemm_ref(x, w, None, epilogue=3)


def test_a_step_at_layer_sizes_of_a_real_model():
    """Three layers of the 2,048-wide shape in bfloat16 through the engine's step function: a prompt of 300 tokens whole against
    the same prompt in portions and decoded, which must agree within rounding."""
    import tempfile

    from clockwork_b200.config.registry import get_architecture
    from clockwork_b200.weights import write_random_model

    raw = dict(get_architecture("Relerax").named_shapes["relerax-2k"])
    raw["layers"] = [dict(raw["layers"][0]), dict(raw["layers"][3], mlp=None), dict(raw["layers"][2], mlp=raw["layers"][0]["mlp"])]
    raw["vocab"] = 4096
    with tempfile.TemporaryDirectory() as folder:
        write_random_model(folder, raw, seed=3)
        tokens = tokens_for(raw, 300, salt=9)
        outs = []
        for sizes in ([300], [200, 90] + [1] * 10, [64, 2, 130, 3, 101]):
            session = TraceSession(folder, "bfloat16", 512, page_size=16)
            got, n = [], 0
            for portion in cut(tokens, sizes):
                out, _ = session.run_step({"step": n, "entries": [{"id": "a", "tokens": portion, "want": [len(portion) - 1]}], "end": []})
                got.append(torch.from_numpy(out.copy()))
                n += 1
            outs.append(torch.cat(got)[-1])
        scale = float(outs[0].std())
        for other in outs[1:]:
            assert float((other - outs[0]).abs().max()) < 0.08 * scale
