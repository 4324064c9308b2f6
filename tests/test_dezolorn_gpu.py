"""Dezolorn through the framework against the plain implementation (``tests/plain/dezolorn_plain.py``): each mechanism
alone, the residual behind every layer run, whole prompts, token-by-token decoding through the captured steps, portions
down to two tokens, unequal requests in one batch against each alone, state slots and pages that are given back and used
again, long decoding (windows pass while tokens are decoded, the kept first positions stay), and greedy generation through
the engine's own entry point and scheduler.  Four small configurations that differ in every size (``dezolorn_configs``);
weights are drawn so that attention is peaked and states remember dozens of tokens, and the tests of the mechanisms alone
first show, with the plain implementation, that a window or a number of kept positions one off, a norm left out, another
pairing or a state that forgot its past would be seen.

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
from clockwork_b200.ops import recurrence as rec_ops
from clockwork_b200.parts import build_part
from clockwork_b200.parts.rotary import rotary_tables
from clockwork_b200.sampling import SamplingParams
from clockwork_b200.weights.loader import make_fetch
from tests.dezolorn_configs import CONFIGS, first_tokens, tokens_for, write_model
from tests.gpu_tools import DEV, PartHarness
from tests.plain import dezolorn_plain as plain
from tests.trace_tools import cut

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]


@pytest.fixture(scope="module")
def dirs(tmp_path_factory):
    return {name: write_model(tmp_path_factory.mktemp(f"dezolorn_{name}"), name, seed=5 + i) for i, name in enumerate(sorted(CONFIGS))}


@pytest.fixture(scope="module")
def prompt(dirs):
    """(name, length, salt) -> tokens whose first one's answer rounding cannot flip."""
    first = first_tokens(dirs)
    return lambda name, length, salt: tokens_for(CONFIGS[name][0], length, salt, first[name])


@pytest.fixture(scope="module")
def oracle(dirs):
    """(name, tokens) -> (float64 logits [T, V], what float32 costs, what bfloat16 storage costs)."""
    weights = {name: plain.read_model_dir(folder, dtype=torch.float64) for name, folder in dirs.items()}

    @functools.lru_cache(maxsize=None)
    def get(name, tokens):
        config, w = weights[name]
        exact = plain.forward(config, w, list(tokens), dtype=torch.float64)
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
def test_whole_prompt(name, dtype, dirs, oracle, prompt):
    tokens = prompt(name, 75, 1)
    run = Replay(dirs[name], name, dtype, 128)
    run.step({"a": tokens}, end=["a"])
    check(run.of("a"), name, tokens, dtype, oracle)


@pytest.mark.parametrize("length", [40, 300])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_the_residual_behind_every_layer_run(name, length, dirs, prompt):
    """float32, run by run (a looped layer counts each time); 300 rows go through the norm kernel of many rows."""
    config, w = plain.read_model_dir(dirs[name], dtype=torch.float64)
    tokens = prompt(name, length, 11)
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
    assert len(seen) == want.shape[0] == len(plain.run_order(config))
    for r, got in enumerate(seen):
        allowed = 30 * float((single[r].double() - want[r]).abs().max()) + 1e-5
        assert float((got.double().cpu() - want[r]).abs().max()) <= allowed, f"behind layer run {r}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prefill_then_token_by_token(name, dtype, dirs, oracle, prompt):
    """The decoded tokens run through the captured single-token steps; the first tokens of a sequence too (a prompt of one
    token).  70 tokens pass every window but the longest."""
    tokens = prompt(name, 70, 2)
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
def test_portions_of_many_sizes(name, dtype, graphs, dirs, oracle, prompt):
    """Cuts in the middle of pages, of windows, of the kept positions and of a convolution's reach; portions of two and three
    tokens, of one page, longer than a window."""
    tokens = prompt(name, 90, 3)
    for sizes in ([2, 3, 1, 7, 2, 16, 5, 4], [37, 2, 2, 2, 30, 1, 1, 3]):
        run = Replay(dirs[name], name, dtype, 128, graphs=graphs)
        for portion in cut(tokens, sizes):
            run.step({"a": portion})
        check(run.of("a"), name, tokens, dtype, oracle)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_unequal_requests_in_one_batch_against_each_alone(name, dtype, dirs, oracle, prompt):
    prompts = {"p": prompt(name, 61, 4), "q": prompt(name, 23, 5), "r": prompt(name, 40, 6), "s": prompt(name, 9, 7)}
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
def test_slots_and_pages_given_back_and_used_again(name, dtype, dirs, oracle, prompt):
    """Ten requests through four state slots and a pool of pages for 4 x 64 tokens: a request that takes a slot or a page
    that another one left starts from zero state and zero inputs before the first, and sees none of the other's keys."""
    run = Replay(dirs[name], name, dtype, 4 * 64)
    prompts = {f"r{i}": prompt(name, 20 + 4 * i, 20 + i) for i in range(10)}
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
    assert not run.session.cache.requests and run.session.cache.state.num_free == 4
    for rid, toks in prompts.items():
        check(run.of(rid), name, toks, dtype, oracle)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "C"])
def test_long_decoding_while_windows_pass(name, dtype, dirs, oracle, prompt):
    """300 decoded tokens behind a short prompt, in looped layers whose every pass keeps its own cache: windows move over
    decoded tokens, states are carried 300 times, the pages behind the windows go back to the pool while the request runs
    and the pages of the kept first positions stay."""
    tokens = prompt(name, 320, 8)
    run = Replay(dirs[name], name, dtype, 320)
    run.step({"a": tokens[:20]})
    for t in tokens[20:]:
        run.step({"a": [t]})
    req = run.session.cache.get("a")
    page = CONFIGS[name][1]
    for group, table in zip(run.session.cache.groups, req.tables):
        kept = -(-group.need.keep_first // page)
        assert all(p >= 0 for p in table[:kept])
        assert sum(p >= 0 for p in table) <= kept + group.need.window // page + 2
    check(run.of("a"), name, tokens, dtype, oracle)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_greedy_generation_through_the_engine(name, dtype, dirs, prompt):
    """The engine's own entry point and scheduler: prompts cut under a small token budget, several requests at once."""
    config, page = CONFIGS[name]
    cfg = EngineConfig.defaults(str(dirs[name]), dtype=dtype, block_size=page, num_blocks=256, max_model_len=256, max_num_seqs=4,
                                max_num_batched_tokens=24)
    engine = LLMEngine(cfg)
    prompts = [prompt(name, n, 30 + n) for n in (5, 31, 18, 1, 44)]
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


def attention_tensors(gen, w, m, peak=1.5):
    h, g, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    return {"q": draw(gen, (h * dk, w), 0.5), "k": draw(gen, (g * dk, w), 0.5), "v": draw(gen, (g * dv, w), 0.3),
            "q.norm": draw(gen, (h * dk,), 0.3, peak), "k.norm": draw(gen, (g * dk,), 0.3, peak), "o": draw(gen, (w, h * dv), 0.2)}


def attention_spec(w, m, eps):
    return PartSpec("window_attention", dict(hidden_size=w, heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"],
                                             scale=m["scale"], weights="softmax", window=m["mask"]["size"],
                                             keep_first=m["mask"]["keep_first"], qk_norm=eps,
                                             rotary=dict(m["rot"], pairing="interleaved")))


def attention_config(heads, kv_heads, dim, vdim, size, keep, scale, rot, base, scaling=None):
    turned = {"dims": rot, "base": base}
    if scaling is not None:
        turned["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, mask={"size": size, "keep_first": keep}, rot=turned)


@pytest.mark.parametrize("heads, kv_heads, dim, vdim, size, keep, rot, base, scaling, page", [
    (4, 2, 24, 12, 21, 5, 8, 1000.0, (4.0, 60, 6.0, 1.0), 4), (3, 1, 16, 40, 7, 9, 16, 50000.0, None, 8),
    (6, 6, 8, 8, 1, 1, 2, 10000.0, None, 4), (2, 2, 12, 20, 400, 6, 12, 100.0, (8.0, 32, 4.0, 2.0), 16),
    (8, 2, 32, 64, 100, 12, 32, 10000.0, (2.0, 300, 20.0, 1.0), 16), (5, 5, 17, 23, 64, 16, 6, 300.0, None, 16),
    (12, 3, 48, 80, 60, 0, 16, 500000.0, (4.0, 100, 8.0, 0.5), 16), (33, 11, 8, 4, 10, 37, 6, 20.0, None, 4)])
def test_a_window_that_keeps_the_first_positions_alone(heads, kv_heads, dim, vdim, size, keep, rot, base, scaling, page):
    """300 positions whole, token by token and in portions that cut pages, windows and the kept positions, the pages behind
    the window given back on the way.  First the plain implementation shows what counts: a window or a number of kept
    positions one off, norms over each head instead of all, the other pairing, an amplitude left out."""
    gen = torch.Generator().manual_seed(heads * 100 + size)
    w, eps = 48, 1e-5
    m = attention_config(heads, kv_heads, dim, vdim, size, keep, 0.25, rot, base, scaling)
    t = attention_tensors(gen, w, m)
    wd = doubled(t)
    x = draw(gen, (300, w))
    want = plain.window_attention(x.double(), wd, m, eps)

    def moved(other):
        return float((plain.window_attention(x.double(), wd, other, eps) - want).abs().max())

    for other in (size - 1, size + 1):
        if 1 <= other < 300:
            assert moved(dict(m, mask={"size": other, "keep_first": keep})) > 0.02
    for other in (keep - 1, keep + 1):
        if other >= 0 and size < 300:
            assert moved(dict(m, mask={"size": size, "keep_first": other})) > 0.02
    if scaling is not None:
        assert moved(dict(m, rot={"dims": rot, "base": base})) > 0.02
    part = part_with_weights("mixer", attention_spec(w, m, eps), "m", torch.float32, named(t))
    for portions in ([131, 169], [1] * 300, [2, 3, 1, 1, 9, 2, 5, 41, 100, 1, 1, 1, 131, 2], [page - 1, 2, page, 1, 300 - 2 * page - 2]):
        assert sum(portions) == 300
        got = run_mixer(part, x, portions, page_size=page, num_pages=300 // page + 8)
        assert_close(got, want, portions)


@pytest.mark.parametrize("heads, kv_heads, dim, vdim, size, keep, rot, page", [
    (4, 4, 256, 256, 100, 12, 128, 16), (8, 8, 64, 64, 130, 33, 64, 64), (16, 1, 64, 64, 40, 3, 64, 16), (8, 2, 128, 128, 150, 40, 64, 16),
    (6, 3, 96, 48, 45, 4, 32, 8), (4, 1, 240, 200, 70, 5, 16, 16), (4, 4, 32, 256, 33, 64, 32, 16), (16, 4, 128, 128, 300, 70, 128, 16)])
def test_a_window_that_keeps_the_first_positions_in_bfloat16_on_the_tensor_cores(heads, kv_heads, dim, vdim, size, keep, rot, page):
    """Sizes that take each arrangement of the tensor-core kernel (windows that are cut in parts among them: few rows, windows
    over 256), whole and in portions, against the plain implementation in float64; allowed is 3 times what rounding q, k, v and
    the output to bfloat16 costs the plain implementation."""
    gen = torch.Generator().manual_seed(heads * 100 + size)
    w, eps = 64, 1e-5
    m = attention_config(heads, kv_heads, dim, vdim, size, keep, dim ** -0.5, rot, 10000.0, (4.0, 128, 16.0, 1.0))
    t = attention_tensors(gen, w, m)
    wd = doubled(t)
    x = draw(gen, (400, w))
    want = plain.window_attention(x.double(), wd, m, eps)
    rounded = plain.to_bfloat16_and_back(plain.window_attention(x.double(), wd, m, eps, rnd=plain.to_bfloat16_and_back))
    allowed = 3 * float((rounded - want).abs().max()) + 0.01 * float(want.abs().max())
    assert allowed < 0.15 * float(want.abs().max())
    part = part_with_weights("mixer", attention_spec(w, m, eps), "m", torch.bfloat16, named(t))
    for portions in ([400], [340] + [1] * 60, [3, 64, 1, 61, 2, 249] + [1] * 20):
        got = run_mixer(part, x, portions, page_size=page, num_pages=400 // page + 8)
        worst = float((got.double() - want).abs().max())
        assert worst <= allowed, f"{portions[:6]}: off by {worst:.3g}, allowed {allowed:.3g}"


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_keys_that_stand_out_at_the_edges_of_the_window_and_of_the_kept_positions(dtype):
    """A query and a few keys are made so that their scores tower over all others.  Of four equal ones, the last kept
    position and the window's far edge share the softmax; the position behind the kept ones and the one behind the window
    are not seen, in a prompt and in decoding, also where a portion ends at an edge and after the pages between have been
    given back.  Norms over all queries and over all keys keep a row's size from mattering: it is directions that stand out."""
    heads, kv_heads, dim, vdim, size, keep, w, rot, eps = 2, 1, 16, 8, 37, 6, 32, 4, 1e-5
    gen = torch.Generator().manual_seed(9)
    m = attention_config(heads, kv_heads, dim, vdim, size, keep, 1.0, rot, 1000.0)
    t = attention_tensors(gen, w, m)
    x = draw(gen, (120, w))
    for name, col, other, count in (("q", 3, 5, heads), ("k", 5, 3, kv_heads)):
        t[name].view(count, dim, w)[:, rot:, col] = 0.5   # unrotated entries of a towering row all point one way
        t[name].view(count, dim, w)[:, :rot, col] = 0.0
        t[name].view(count, dim, w)[:, :, other] = 0.0
        t[name + ".norm"] = torch.full_like(t[name + ".norm"], 2.5)
    x[:, 3] = x[:, 5] = 0.0
    t["v"][:, [3, 5]] = 0.0  # (towering rows have values of their own)
    probe = 100
    inside, outside, last_kept, first_not = probe - size + 1, probe - size, keep - 1, keep
    x[probe, 3] = 60.0
    for p in (inside, outside, last_kept, first_not):
        x[p, 5] = 60.0
    wd = doubled(t)
    want = plain.window_attention(x.double(), wd, m, eps)
    # the two in sight share every head's softmax (unequally: the rows' other coordinates) and nothing else counts
    values = x[[inside, last_kept]].double() @ wd["v"].T  # [2, vdim]: one key/value head
    parts = torch.stack([values[key] @ wd["o"][:, h * vdim : (h + 1) * vdim].T for h in range(heads) for key in range(2)])
    share = torch.linalg.lstsq(parts.T, want[probe, :, None]).solution.reshape(heads, 2)
    assert float(share.min()) > 0.02 and float((share.sum(1) - 1.0).abs().max()) < 1e-6
    assert float((share.reshape(-1) @ parts - want[probe]).abs().max()) < 1e-6
    rounded = plain.to_bfloat16_and_back(plain.window_attention(x.double(), wd, m, eps, rnd=plain.to_bfloat16_and_back))
    allowed = 3 * float((rounded - want)[probe].abs().max())
    for other in ({"size": size + 1, "keep_first": keep}, {"size": size - 1, "keep_first": keep}, {"size": size, "keep_first": keep + 1},
                  {"size": size, "keep_first": keep - 1}):
        assert float((plain.window_attention(x.double(), wd, dict(m, mask=other), eps) - want)[probe].abs().max()) > 2 * allowed
    part = part_with_weights("mixer", attention_spec(w, m, eps), "m", dtype, named(t))
    for portions in ([120], [probe, 1, 19], [inside, 20, 16, 1, 19], [outside, 1, 1, 35, 1, 19], [70] + [1] * 50, [last_kept, 1, 1, 93, 1, 19],
                     [1] * 120):
        assert sum(portions) == 120
        got = run_mixer(part, x, portions, page_size=8)
        if dtype == torch.float32:
            assert_close(got, want, portions)
        else:
            assert float((got.double() - want)[probe].abs().max()) < allowed, portions


def test_a_kept_key_far_back_among_hundreds():
    """The key at position 2 stands out for a query 850 positions on while the window holds hundreds of others; a key at
    position 300, as strong, is long out of sight.  Whole, decoded, and over portions."""
    heads, kv_heads, dim, vdim, size, keep, w, rot, eps = 4, 2, 32, 16, 400, 3, 32, 8, 1e-5
    gen = torch.Generator().manual_seed(10)
    m = attention_config(heads, kv_heads, dim, vdim, size, keep, 1.0, rot, 1000.0, (4.0, 256, 8.0, 1.0))
    t = attention_tensors(gen, w, m)
    x = draw(gen, (900, w))
    for name, col, other, count in (("q", 3, 5, heads), ("k", 5, 3, kv_heads)):
        t[name].view(count, dim, w)[:, rot:, col] = 0.5
        t[name].view(count, dim, w)[:, :rot, col] = 0.0
        t[name].view(count, dim, w)[:, :, other] = 0.0
        t[name + ".norm"] = torch.full_like(t[name + ".norm"], 4.0)
    x[:, 3] = x[:, 5] = 0.0
    x[852, 3] = 60.0
    x[[2, 300], 5] = 60.0
    wd = doubled(t)
    want = plain.window_attention(x.double(), wd, m, eps)
    far = (x[2].double() @ wd["v"].T).reshape(kv_heads, vdim).repeat_interleave(heads // kv_heads, 0).reshape(-1) @ wd["o"].T
    assert float((want[852] - far).abs().max()) < 1e-6
    part = part_with_weights("mixer", attention_spec(w, m, eps), "m", torch.float32, named(t))
    for portions in ([900], [840] + [1] * 60, [1, 4, 300, 545, 3, 1, 46]):
        got = run_mixer(part, x, portions, page_size=16)
        assert_close(got, want, portions)


@pytest.mark.parametrize("heads, dim, vdim, rot, dtype", [(3, 12, 20, 12, torch.float32), (1, 16, 8, 6, torch.float32), (5, 8, 24, 4, torch.float32),
                                                          (2, 11, 5, 2, torch.float32), (4, 64, 48, 32, torch.float32), (2, 256, 16, 256, torch.float32),
                                                          (2, 200, 40, 8, torch.float32), (3, 96, 96, 96, torch.bfloat16), (16, 128, 128, 128, torch.bfloat16)])
def test_retention_alone(heads, dim, vdim, rot, dtype):
    """200 positions whole, token by token and in portions: the state is carried from portion to portion.  First the plain
    implementation shows that a state that starts from zero in the middle, neighbouring pairs or other decays would be seen.
    (A first row whose output is all but zero is not compared: the norm behind it blows up what is left.)"""
    gen = torch.Generator().manual_seed(heads * 100 + dim)
    w, eps = 48, 1e-5
    t = {"q": draw(gen, (heads * dim, w), 0.3), "k": draw(gen, (heads * dim, w), 0.3), "v": draw(gen, (heads * vdim, w), 0.3),
         "g": draw(gen, (heads * vdim, w), 0.3), "o": draw(gen, (w, heads * vdim), 0.2)}
    m = dict(heads=heads, dim=dim, vdim=vdim, decay=[1 - 0.3 * 0.4 ** h for h in range(heads)], rot={"dims": rot, "base": 500.0})
    wd = doubled(t)
    x = draw(gen, (200, w))
    want = plain.retention(x.double(), wd, m, eps)
    fresh = plain.retention(x[100:].double(), wd, m, eps)
    assert float((fresh - want[100:]).abs().max()) > 0.05
    assert float((plain.retention(x.double(), wd, dict(m, decay=[d - 0.02 for d in m["decay"]]), eps) - want).abs().max()) > 0.02
    assert float((plain.retention(x.double(), wd, dict(m, rot={"dims": rot, "base": 400.0}), eps) - want).abs().max()) > (0.02 if rot > 2 else -1)
    spec = PartSpec("retention", dict(hidden_size=w, heads=heads, dim=dim, vdim=vdim, eps=eps, decay=m["decay"], rotary=dict(m["rot"])))
    part = part_with_weights("mixer", spec, "m", dtype, named(t))
    if dtype == torch.bfloat16:
        rounded = plain.to_bfloat16_and_back(plain.retention(x.double(), wd, m, eps, rnd=plain.to_bfloat16_and_back))
        allowed = 3 * float((rounded - want).abs().max()) + 0.01 * float(want.abs().max())
    for portions in ([200], [1] * 200, [2, 3, 1, 1, 9, 2, 5, 41, 100, 1, 1, 1, 31, 2], [17, 150, 33]):
        got = run_mixer(part, x, portions)
        if dtype == torch.float32:
            assert_close(got, want, portions, rel=1e-4)
        else:
            assert float((got.double() - want).abs().max()) <= allowed, portions


@pytest.mark.parametrize("heads, kv_heads, dim, vdim, conv, dtype", [
    (4, 2, 12, 20, 4, torch.float32), (3, 3, 10, 7, 1, torch.float32), (6, 1, 24, 12, 6, torch.float32), (1, 1, 8, 8, 2, torch.float32),
    (2, 2, 256, 16, 4, torch.float32), (2, 1, 104, 40, 3, torch.float32), (4, 4, 64, 48, 4, torch.float32), (5, 5, 16, 33, 4, torch.float32),
    (8, 4, 32, 64, 4, torch.bfloat16), (16, 16, 128, 128, 4, torch.bfloat16)])
def test_the_delta_rule_with_one_decay_per_head_alone(heads, kv_heads, dim, vdim, conv, dtype):
    """200 positions whole, token by token and in portions shorter than the convolutions' reach.  First the plain
    implementation shows that a state or convolution inputs that start from zero in the middle, write strengths of one half
    or decays that do not depend on the input would be seen."""
    gen = torch.Generator().manual_seed(heads * 100 + dim)
    w, eps = 48, 1e-5
    qk, inner = kv_heads * dim, heads * vdim
    t = {"q": draw(gen, (qk, w), 0.3), "k": draw(gen, (qk, w), 0.3), "v": draw(gen, (inner, w), 0.3), "g": draw(gen, (inner, w), 0.3),
         "a": draw(gen, (heads, w), 0.2), "b": draw(gen, (heads, w), 0.3), "A_log": draw(gen, (heads,), 0.5), "dt_bias": draw(gen, (heads,), 0.7, -3.0),
         "norm": draw(gen, (vdim,), 0.2, 1.0), "o": draw(gen, (w, inner), 0.2)}
    t.update({f"{n}.conv": draw(gen, (qk if n != "v" else inner, conv), 0.5) for n in "qkv"})
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv)
    wd = doubled(t)
    x = draw(gen, (200, w))
    want = plain.gated_delta(x.double(), wd, m, eps)
    fresh = plain.gated_delta(x[100:].double(), wd, m, eps)
    assert float((fresh - want[100:]).abs().max()) > 0.05
    for name in ("a", "b"):
        assert float((plain.gated_delta(x.double(), dict(wd, **{name: wd[name] * 0}), m, eps) - want).abs().max()) > 0.02
    spec = PartSpec("head_delta", dict(hidden_size=w, heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv, eps=eps))
    part = part_with_weights("mixer", spec, "m", dtype, named(t))
    if dtype == torch.bfloat16:
        rounded = plain.to_bfloat16_and_back(plain.gated_delta(x.double(), wd, m, eps, rnd=plain.to_bfloat16_and_back))
        allowed = 3 * float((rounded - want).abs().max()) + 0.01 * float(want.abs().max())
    for portions in ([200], [1] * 200, [2, 3, 1, 1, 9, 2, 5, 41, 100, 1, 1, 1, 31, 2], [17, 150, 33]):
        got = run_mixer(part, x, portions)
        if dtype == torch.float32:
            assert_close(got, want, portions, rel=1e-4)
        else:
            assert float((got.double() - want).abs().max()) <= allowed, portions


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n, w", [(3, 50), (1, 64), (300, 128), (300, 74), (257, 1000), (5, 2048), (270, 4096), (40, 5000)])
def test_layer_norm_with_what_is_pending_alone(n, w, dtype):
    """Rows with a mean three times their spread, few and many of them, with nothing, a tensor and the slabs of a split product
    pending, and selected rows; the sums land in the residual."""
    gen = torch.Generator().manual_seed(n + w)
    x = 3.0 + torch.randn((n, w), generator=gen)
    weight = 1 + 0.2 * torch.randn(w, generator=gen)
    delta = torch.randn((n, w), generator=gen).to(dtype)
    slabs = torch.randn((3, n + 2, w), generator=gen)
    status = ops.new_status(DEV)
    eps = 1e-3

    def close(got, y):
        want = plain.layer_norm(y.double(), weight.double(), eps)
        assert float((got.double().cpu() - want).abs().max()) <= (3e-5 if dtype == torch.float32 else 2 ** -7 * float(want.abs().max()))

    close(ops.add_rmsnorm(x.to(DEV), None, weight.to(DEV), eps, dtype, status, center=True), x)
    resid = x.to(DEV)
    close(ops.add_rmsnorm(resid, delta.to(DEV), weight.to(DEV), eps, dtype, status, center=True), x + delta.float())
    assert torch.equal(resid.cpu(), x + delta.float())
    if w % 4 == 0 and w <= 4096:
        resid = x.to(DEV)
        summed = ((x + slabs[0, :n]) + slabs[1, :n]) + slabs[2, :n]
        close(ops.add_rmsnorm(resid, ops.PartialSums(slabs.to(DEV), n), weight.to(DEV), eps, dtype, status, center=True), summed)
        assert torch.equal(resid.cpu(), summed)
    rows = torch.tensor([n - 1, 0, n // 2], dtype=torch.int32)
    close(ops.rmsnorm_rows(x.to(DEV), rows.to(DEV), weight.to(DEV), eps, dtype, status, center=True), x[rows.long()])
    ops.raise_on_status(status)


@pytest.mark.parametrize("interleaved", [False, True])
@pytest.mark.parametrize("heads, dim, rot, scaling", [(3, 16, 16, None), (5, 10, 6, None), (2, 64, 32, (4.0, 512, 32.0, 1.0)), (7, 128, 128, None)])
def test_rotation_in_place_alone(heads, dim, rot, scaling, interleaved):
    """The leading columns of wider rows; entries beyond the rotated ones and columns beyond the heads stay."""
    gen = torch.Generator().manual_seed(dim)
    n, ld = 19, heads * dim + 9
    x = torch.randn((n, ld), generator=gen)
    turned = {"dims": rot, "base": 700.0}
    if scaling is not None:
        turned["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    positions = torch.tensor([0, 1, 2, 3, 5, 8, 13, 21, 34, 55, 89, 144, 233, 377, 610, 987, 1597, 2584, 4181])
    inv_freq, amplitude = rotary_tables(rot, 700.0, turned.get("scaling"))
    got = x.to(DEV)
    rec_ops.rotate_heads_(got, positions.to(torch.int32).to(DEV), inv_freq.to(DEV), heads, dim, rot, interleaved, amplitude)
    want = plain.rotate(x[:, : heads * dim].double().reshape(n, heads, dim), positions, turned, interleaved).reshape(n, -1)
    # (an angle of thousands is good to float32's spacing there)
    assert float((got[:, : heads * dim].cpu().double() - want).abs().max()) < 2e-3
    assert float((got[:10, : heads * dim].cpu().double() - want[:10]).abs().max()) < 5e-5
    assert torch.equal(got[:, heads * dim :].cpu(), x[:, heads * dim :])
    other = plain.rotate(x[:, : heads * dim].double().reshape(n, heads, dim), positions, turned, not interleaved).reshape(n, -1)
    assert float((other - want).abs().max()) > 0.5


def test_scaled_and_bent_logits_and_a_norm_in_parts_without_a_weight():
    gen = torch.Generator().manual_seed(6)
    z = 10 * torch.randn((5, 77), generator=gen)
    for cap, scale in ((4.0, 0.3), (4.0, 1.0), (None, 0.3)):
        want = scale * z.double() if cap is None else cap * torch.tanh(scale * z.double() / cap)
        assert float((ops.softcap_(z.to(DEV), cap, scale).cpu().double() - want).abs().max()) < 1e-5
    y, g = torch.randn((9, 60), generator=gen), torch.randn((9, 60), generator=gen)
    got = rec_ops.gated_group_norm(y.to(DEV), g.to(DEV), None, 5, 1e-5, False, torch.float32, gate=rec_ops.GATE_SILU)
    want = plain.unit_rms(y.double().reshape(9, 5, 12), 1e-5).reshape(9, 60) * torch.nn.functional.silu(g.double())
    assert_close(got.cpu(), want, "norm in parts")


def test_a_step_at_layer_sizes_of_a_real_model():
    """Three layers of the 2,048-wide shape in bfloat16 through the engine's step function: a prompt of 300 tokens whole against
    the same prompt in portions and decoded, which must agree within rounding."""
    import tempfile

    from clockwork_b200.config.registry import get_architecture
    from clockwork_b200.weights import write_random_model

    raw = dict(get_architecture("Dezolorn").named_shapes["dezolorn-2k"])
    raw["layers"] = [raw["layers"][3], raw["layers"][0], raw["layers"][1]]
    raw["loop"] = {"start": 1, "stop": 2, "times": 2}
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
