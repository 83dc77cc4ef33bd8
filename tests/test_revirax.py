"""The Revirax decoder through the engine's step function, cache manager, scheduler and entry point, against the plain
implementation of tests/plain/revirax_plain.py, for every way of cutting the work.

Each test runs on the GPU with the real kernel library in float32 (captured steps) and bfloat16 (marked gpu), and on the CPU with the
stand-in kernels of tests/fake_kernels.py, which checks the host side: the batch tables, the pages a window gives back, the slots, which
cache and state each branch of a parallel mixer gets, the norm that travels with the residual from one sublayer's output to the next.
"""
import copy
import math
import random

import pytest
import torch

from roost_b200 import GenerationOptions, RoostEngine
from roost_b200.config.reader import ConfigError
from roost_b200.config.revirax import ReviraxConfig
from roost_b200.config.spec import MinGruSpec, NormSpec, ParallelMixerSpec, PositionSpec, RetentionSpec, RotationScaling, SinkAttentionSpec, TalkingAttentionSpec
from roost_b200.engine.executor import StepEntry, StepExecutor
from roost_b200.parts import Runtime
from roost_b200.parts.parallel import ParallelMixer
from roost_b200.parts.positions import RopeNeox, scaled_frequencies
from roost_b200.parts.retention import Retention
from roost_b200.weights.loader import WeightError
from tests import helpers as H
from tests import revirax_models as RM
from tests.plain import revirax_plain as P

BACKENDS = [
    pytest.param(("gpu", torch.float32), id="gpu-f32", marks=pytest.mark.gpu),
    pytest.param(("gpu", torch.bfloat16), id="gpu-bf16", marks=pytest.mark.gpu),
    pytest.param(("fake", torch.float32), id="cpu-fake"),
]
# Two bounds: the root-mean-square error of all logits of a request, and the largest root-mean-square error of one position's logits (both
# relative to the logits' own root mean square). A fault that strikes one position (a key lost at a page's or a tile's edge, a wrong page or
# slot in one step, a state taken from another request) moves that position's logits by tens of percent and barely shows among hundreds
# of positions; rounding alone stays far below both bounds.
F32_TOKEN, F32_RMS = 1e-3, 3e-5
BF16_TOKEN, BF16_RMS = 0.2, 0.05


@pytest.fixture(params=BACKENDS)
def backend(request):
    return request.param


_MODELS: dict = {}


def model_dir(tmp_path_factory, name, cfg, seed, change=None):
    """A model folder written once a session; ``change(cfg, tensors)`` edits the drawn weights first."""
    if name not in _MODELS:
        tensors = RM.draw_tensors(cfg, seed)
        if change is not None:
            change(cfg, tensors)
        _MODELS[name] = (RM.write_model(tmp_path_factory.mktemp(f"revirax_{name}"), cfg, tensors), cfg, RM.plain_weights(tensors))
    return _MODELS[name]


def position_errors(got, want):
    """Every position's error: root mean square of its logits' differences over that of its logits."""
    got, want = got.double().cpu(), want.double().cpu()
    return (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt()


_PLAIN: dict = {}


def plain_logits(cfg, weights, ids):
    """The plain logits, kept: the backends of one test ask for the same ones."""
    key = (id(weights), tuple(ids))
    if key not in _PLAIN:
        _PLAIN[key] = P.forward(cfg, weights, list(ids))
    return _PLAIN[key]


class Run:
    """Drives a StepExecutor and keeps, per request, the logits of every position."""

    def __init__(self, model_dir, cfg, backend, page_size=4, num_pages=64, slots=4, graphs=True):
        kind, self.dtype = backend
        self.cfg = cfg
        self.model = H.make_model(model_dir, self.dtype, kind)
        self.ex = StepExecutor(self.model, page_size=page_size, num_pages=num_pages, max_requests=slots, use_graphs=graphs)
        self.logits: dict = {}

    def step(self, entries):
        """entries: [(request id, tokens)]; every position's logits are asked for."""
        out = self.ex.step([StepEntry(rid, list(toks), list(range(len(toks)))) for rid, toks in entries])
        at = 0
        for rid, toks in entries:
            self.logits.setdefault(rid, []).append(out[at : at + len(toks)].float().cpu())
            at += len(toks)
        self.ex.cache.check_invariants()

    def finish(self, rid):
        self.ex.finish(rid)

    def check(self, rid, ids, weights, what):
        got = torch.cat(self.logits.pop(rid))
        ids = list(ids[: got.shape[0]])
        want = plain_logits(self.cfg, weights, ids)
        worst, bound = (F32_TOKEN, F32_RMS) if self.dtype == torch.float32 else (BF16_TOKEN, BF16_RMS)
        keep = torch.ones(got.shape[0], dtype=torch.bool)
        if self.dtype != torch.float32 and bool((position_errors(got, want) >= worst).any()):
            # A norm keeps only the direction of what it is given: where a sublayer's output is next to zero (a lightning state of one token
            # that meets a query across it, say) the direction hangs on the last bits. A position over the bound is ill-conditioned, not
            # faulty, when rounding the plain implementation's norms and projections to 16 bits (as they are, and after a relative change of
            # up to 2^-8) moves its logits far by itself. Such positions are left out in 16 bits; the 32-bit run of the same kernels checks them.
            moved = position_errors(P.forward(self.cfg, weights, ids, rounding=lambda z: z.to(torch.bfloat16).double()), want)
            for draw in range(4):
                g = torch.Generator().manual_seed(draw)
                noisy = lambda z: (z * (1.0 + 2.0 ** -8 * (2.0 * torch.rand(z.shape, generator=g, dtype=torch.float64) - 1.0))).to(torch.bfloat16).double()
                moved = torch.maximum(moved, position_errors(P.forward(self.cfg, weights, ids, rounding=noisy), want))
            keep = moved < worst / 3
            assert int((~keep).sum()) <= max(2, got.shape[0] // 20), f"{what}: the test's model is ill-conditioned at {int((~keep).sum())} positions"
        err, rms = float(position_errors(got, want)[keep].max()), H.rms_error(got[keep], want[keep])
        print(f"MEASURED {what} {self.dtype}: worst position's error {err:.3e}, rms error {rms:.3e}, {int((~keep).sum())} positions left out")
        assert err < worst and rms < bound, f"{what}: worst position's error {err}, rms error {rms}"
        return got, want

    def all_free(self):
        return all(p.used_count == 0 for p in self.ex.cache.pools)


def ids_for(cfg, n, seed):
    return H.random_ids(n, cfg["vocab"], seed)


# One mechanism a model, so that a fault names its mechanism.
SINGLE = {
    "attention_only": RM.config([(RM.attention(heads=2, kv_heads=1, dim=6, vdim=5), None)], width=24, vocab=50),
    "lightning_only": RM.config([(RM.lightning(heads=2, dim=6, vdim=5, decay=(0.8, 0.97)), None)], width=20, vocab=45),
    "parallel_only": RM.config([(RM.parallel(heads=2, kv_heads=1, dim=6, vdim=5, window=7, width=9), None)], width=16, vocab=30),
    "dense_after_attention": RM.config([(RM.attention(heads=1, kv_heads=1, dim=8, vdim=8, rot=2), RM.dense(ff=17))], width=28, vocab=33),
}
ALL = dict(RM.CONFIGS, **SINGLE)


@pytest.fixture(params=sorted(ALL))
def any_model(request, tmp_path_factory):
    return (request.param,) + model_dir(tmp_path_factory, request.param, ALL[request.param], seed=len(request.param))


@pytest.fixture(params=sorted(RM.CONFIGS))
def model(request, tmp_path_factory):
    return (request.param,) + model_dir(tmp_path_factory, request.param, RM.CONFIGS[request.param], seed=len(request.param))


# ------------------------------------------------------------------------------------------------ whole prompts
@pytest.mark.parametrize("length", [1, 2, 3, 37, 150])
def test_each_mechanism_and_each_model_on_whole_prompts(any_model, backend, length):
    """Models of one mechanism each and the mixed models; the shortest prompts are the first tokens of a sequence (an empty state, one key
    beside the sink); the longest reach far beyond every window."""
    name, folder, cfg, weights = any_model
    run = Run(folder, cfg, backend)
    ids = ids_for(cfg, length, seed=length)
    run.step([("r", ids)])
    run.finish("r")
    run.check("r", ids, weights, f"{name} whole {length}")
    assert run.all_free()


def test_the_residual_after_every_layer(model, backend):
    """The engine's stream after every layer (the 32-bit residual plus the normed branch output still to be added) against the plain one."""
    name, folder, cfg, weights = model
    kind, dtype = backend
    m = H.make_model(folder, dtype, kind)
    ex = StepExecutor(m, page_size=4, num_pages=32, max_requests=2, use_graphs=False)
    ids = ids_for(cfg, 21, seed=9)
    seen = []

    class Watched:
        def __init__(self, block):
            self.block = block

        def __getattr__(self, name):
            return getattr(self.block, name)

        def __call__(self, *args, **kwargs):
            a, residual = self.block(*args, **kwargs)
            y = a.float()
            seen.append((residual.stream.float() + y * torch.rsqrt((y * y).mean(-1, keepdim=True) + residual.post.spec.eps) * residual.post.weight).cpu())
            return a, residual

    m.blocks = [Watched(b) for b in m.blocks]
    ex.step([StepEntry("r", ids, [20])])
    want = []
    P.forward(cfg, weights, ids, layer_outputs=want)
    assert len(seen) == len(want) == len(cfg["layers"])
    for i, (g, w) in enumerate(zip(seen, want)):
        err = H.rms_error(g, w)
        assert err < (2e-5 if dtype == torch.float32 else 0.03), f"{name}: the stream after layer {i} differs by {err}"


# ------------------------------------------------------------------------------------------------ cutting the work
def test_prefill_against_token_by_token_decoding(model, backend):
    name, folder, cfg, weights = model
    run = Run(folder, cfg, backend)
    ids = ids_for(cfg, 70, seed=5)
    for head in (0, 1, 38):     # from the very first token on; after one token; after a prompt that ends inside a page
        rid = f"r{head}"
        if head:
            run.step([(rid, ids[:head])])
        for t in ids[head:]:
            run.step([(rid, [t])])
        run.finish(rid)
        run.check(rid, ids, weights, f"{name} decoded from {head}")
    assert run.all_free()


@pytest.mark.parametrize("sizes", [[2, 3, 2, 5, 7, 16, 33], [33, 2, 2, 1, 9], [1, 2]])
def test_portions_of_several_sizes_down_to_two_tokens(model, backend, sizes):
    """A portion's first token takes its states from the slots and its keys from the pages of earlier portions."""
    name, folder, cfg, weights = model
    run = Run(folder, cfg, backend)
    ids = ids_for(cfg, 90 if len(sizes) > 2 else 25, seed=sum(sizes))
    at, i = 0, 0
    while at < len(ids):
        n = min(sizes[i % len(sizes)], len(ids) - at)
        run.step([("r", ids[at : at + n])])
        at, i = at + n, i + 1
    run.finish("r")
    run.check("r", ids, weights, f"{name} portions {sizes}")


def test_batches_of_unequal_requests_with_pages_and_slots_used_again(model, backend):
    """Six requests of unequal length through three state slots and a pool of pages that holds three of them: portions of some beside single
    tokens of others; a request may sit out a step; a request that ends gives its pages and slots to the next one, whose states must
    start empty."""
    name, folder, cfg, weights = model
    run = Run(folder, cfg, backend, page_size=4, num_pages=48, slots=3)
    rng = random.Random(11)
    reqs = {f"q{i}": ids_for(cfg, n, seed=20 + i) for i, n in enumerate([41, 9, 64, 23, 2, 55])}
    waiting, live = list(reqs), {}
    slots_seen = set()
    while waiting or live:
        while waiting and len(live) < 3:
            live[waiting.pop(0)] = 0
        entries = []
        for rid in [r for r in live if rng.random() < 0.8] or [next(iter(live))]:
            left = len(reqs[rid]) - live[rid]
            n = 1 if left <= 6 else min(left - 6, rng.choice([2, 3, 5, 8, 17]))
            entries.append((rid, reqs[rid][live[rid] : live[rid] + n]))
            live[rid] += n
        run.step(entries)
        for gi, g in enumerate(run.ex.groups):
            if g.kind == "state" and g.runs:
                slots_seen.update(run.ex.cache.get(rid).slots[gi] for rid, _ in entries)
        for rid, _ in entries:
            if live[rid] == len(reqs[rid]):
                run.finish(rid)
                del live[rid]
    assert slots_seen <= {0, 1, 2}
    for rid, ids in reqs.items():
        run.check(rid, ids, weights, f"{name} mixed {rid}")
    assert run.all_free()


def test_a_batch_gives_each_request_what_it_gets_alone(model, backend):
    """The same three requests alone and side by side in one batch, cut the same way: beyond rounding nothing may differ."""
    name, folder, cfg, weights = model
    reqs = {f"s{i}": ids_for(cfg, n, seed=40 + i) for i, n in enumerate([33, 7, 50])}
    cuts = {"s0": [20, 2, 11], "s1": [1, 1, 5], "s2": [2, 40, 8]}
    alone = Run(folder, cfg, backend)
    for rid, ids in reqs.items():
        at = 0
        for n in cuts[rid]:
            alone.step([(rid, ids[at : at + n])])
            at += n
        alone.finish(rid)
    together = Run(folder, cfg, backend)
    at = {rid: 0 for rid in reqs}
    for step in range(3):
        together.step([(rid, reqs[rid][at[rid] : at[rid] + cuts[rid][step]]) for rid in reqs])
        for rid in reqs:
            at[rid] += cuts[rid][step]
    for rid in reqs:
        a, b = torch.cat(alone.logits[rid]), torch.cat(together.logits[rid])
        err = float(position_errors(b, a).max())
        assert err < (2e-5 if backend[1] == torch.float32 else 0.1), f"{name} {rid}: alone and in a batch differ by {err}"


def test_long_decoding_over_many_pages(model, backend):
    """230 tokens one by one through a pool of pages that the whole request would not leave room in twice: windows pass over decoded
    tokens and give their pages back, states are carried 227 times."""
    name, folder, cfg, weights = model
    run = Run(folder, cfg, backend, page_size=4, num_pages=62)
    ids = ids_for(cfg, 230, seed=3)
    run.step([("r", ids[:3])])
    for t in ids[3:]:
        run.step([("r", [t])])
    for gi, g in enumerate(run.ex.groups):
        if g.kind == "paged" and g.window is not None:
            assert run.ex.cache.pools[gi].used_count <= -(-(g.window + 4) // 4) + 1, "pages before the window were kept"
    run.finish("r")
    run.check("r", ids, weights, f"{name} long decoding")


LONG = RM.config([(RM.parallel(heads=4, kv_heads=2, dim=16, vdim=16, scale=0.25, window=200, rot=8, width=40), RM.dense(ff=128)),
                  (RM.lightning(heads=2, dim=20, vdim=36, decay=(0.98, 0.999)), None),
                  (RM.attention(heads=4, kv_heads=2, dim=32, vdim=32, scale=0.2, rot=16, original=200), RM.dense(ff=96)),
                  (RM.parallel(heads=2, kv_heads=2, dim=16, vdim=48, scale=0.25, window=1000, rot=16, width=24), None)], width=72, vocab=83)


def test_a_long_prompt_takes_the_forms_of_steps_of_many_rows(tmp_path_factory, backend):
    """700 tokens in one step and then 2 + 1: the kernels' forms for many tokens a row (the lightning state and the recurrence in chunks whose
    states are carried from chunk to chunk, the last chunk a partial one; the attentions on the tensor cores, a tile of queries with its
    keys dealt to several blocks)."""
    folder, cfg, weights = model_dir(tmp_path_factory, "long", LONG, seed=21)
    run = Run(folder, cfg, backend, page_size=16, num_pages=64)
    ids = ids_for(cfg, 703, seed=8)
    run.step([("r", ids[:700])])
    run.step([("r", ids[700:702])])
    run.step([("r", ids[702:])])
    run.finish("r")
    run.check("r", ids, weights, "long prompt")


def test_the_first_tokens_of_a_sequence_one_by_one(any_model, backend):
    """A request decoded from its very first token: empty states, one key beside the sink."""
    name, folder, cfg, weights = any_model
    run = Run(folder, cfg, backend)
    ids = ids_for(cfg, 6, seed=1)
    for t in ids:
        run.step([("r", [t])])
    run.finish("r")
    run.check("r", ids, weights, f"{name} first tokens")


# ------------------------------------------------------------------------------------------------ keys and states that must be seen
KEY, QUERY = 7, 11        # token ids: QUERY reads what KEY left in the first layer's mixer
SHARP = 0.2               # how far the key token must move the query's plain logits (root mean square, relative) for a test to count
# The first layer's mixer alone carries the key token to the query token here (the second layer has a mixer of another kind, so that the
# cache groups and slots of two kinds meet in one model).
FAR = {
    "attention": RM.config([(RM.attention(heads=2, kv_heads=1, dim=16, vdim=6, scale=0.3, rot=8), None),
                            (RM.lightning(heads=1, dim=4, vdim=4, decay=(0.5,)), RM.dense(ff=16))], width=32, vocab=53),
    "left": RM.config([(RM.parallel(heads=2, kv_heads=1, dim=16, vdim=16, scale=0.3, rot=8, window=400, width=6, left_scale=1.5, right_scale=0.2), None),
                       (RM.attention(heads=2, kv_heads=2, dim=4, vdim=4), RM.dense(ff=16))], width=32, vocab=53),
    "right": RM.config([(RM.parallel(heads=2, kv_heads=1, dim=8, vdim=6, window=5, width=12, left_scale=0.1, right_scale=1.5), None),
                        (RM.lightning(heads=1, dim=4, vdim=4, decay=(0.5,)), RM.dense(ff=16))], width=32, vocab=53),
    "lightning": RM.config([(RM.lightning(heads=2, dim=12, vdim=6, decay=(0.999, 0.9995)), None),
                            (RM.attention(heads=1, kv_heads=1, dim=4, vdim=4), RM.dense(ff=16))], width=32, vocab=53),
}


def sharpened(tmp_path_factory, kind, cfg=None, name=None):
    def change(c, t):
        RM.sharpen(c, t, KEY, QUERY, part=kind)
        for n in ("l1.norm1b", "l1.norm2b"):              # the second layer stays small beside what the first one carries
            t[n] = (-0.8 + 0.2 * t[n].float()).to(torch.bfloat16)
    return model_dir(tmp_path_factory, name or f"far_{kind}", cfg or FAR[kind], seed=77, change=change)


def filler(cfg, n, seed):
    rng = random.Random(seed)
    return [rng.choice([t for t in range(cfg["vocab"]) if t not in (KEY, QUERY)]) for _ in range(n)]


@pytest.mark.parametrize("decoded", [False, True], ids=["in a prompt", "decoded"])
@pytest.mark.parametrize("kind", sorted(FAR))
def test_a_key_far_away_among_hundreds_at_every_page_offset(tmp_path_factory, backend, kind, decoded):
    """The key token sits 256 to 321 places before the query token, once at every offset of a page of four and across the borders of the 32-
    and 64-key tiles; losing that one token (a wrong page, a tile's or a split's edge, a state cut short) changes the query's logits by far
    more than the bound, which the test checks on the plain logits with and without it."""
    folder, cfg, weights = sharpened(tmp_path_factory, kind)
    run = Run(folder, cfg, backend, page_size=4, num_pages=120)
    seen = {}
    places = (0, 1, 2, 3, 31, 32, 33, 63, 64, 65) if backend[0] == "gpu" else (0, 3, 32, 63)
    for at in (None,) + places:
        ids = filler(cfg, 330, seed=4)
        if at is not None:
            ids[at] = KEY
        ids[321] = QUERY
        rid = f"far{at}"
        if decoded:
            run.step([(rid, ids[:300])])
            for t in ids[300:]:
                run.step([(rid, [t])])
        else:
            run.step([(rid, ids[:130])])
            run.step([(rid, ids[130:])])
        run.finish(rid)
        got, want = run.check(rid, ids, weights, f"{kind}: far key at {at}")
        seen[at] = (got[321], want[321])
    for at in places:
        moved = H.rms_error(seen[at][1][None], seen[None][1][None])
        off = H.rms_error(seen[at][0][None], seen[at][1][None])
        print(f"MEASURED {kind}: the key at {at} moves the query's logits by {moved:.3f}; the engine is {off:.2e} from the plain logits with it")
        assert moved > SHARP                    # the test's own sharpness
        assert off < moved / 4                  # the engine saw the key


@pytest.mark.parametrize("window", [16, 31, 32, 33, 64, 100])
def test_keys_just_inside_and_just_outside_a_window(tmp_path_factory, backend, window):
    """The key token ``window`` - 1 places before the query token (the last one it sees) and ``window`` places before it (the first it does
    not), the query at several offsets of a page and a tile, in a prompt's portion and decoded. One token more or less in the window
    changes the query's logits by far more than the bound."""
    cfg = copy.deepcopy(FAR["left"])
    cfg["layers"][0]["mixer"]["left"]["mask"]["size"] = window
    folder, cfg, weights = sharpened(tmp_path_factory, "left", cfg, f"window{window}")
    run = Run(folder, cfg, backend, page_size=4, num_pages=80)
    for query_at in (127, 128, 130):
        for decoded in (False, True):
            seen = {}
            for gap in (window - 1, window):
                ids = filler(cfg, query_at + 2, seed=query_at)
                ids[query_at - gap], ids[query_at] = KEY, QUERY
                rid = f"w{query_at}_{gap}_{decoded}"
                if decoded:
                    run.step([(rid, ids[: query_at - 3])])
                    for t in ids[query_at - 3 :]:
                        run.step([(rid, [t])])
                else:
                    run.step([(rid, ids[:70])])
                    run.step([(rid, ids[70:])])
                run.finish(rid)
                got, want = run.check(rid, ids, weights, f"window {window}, key {gap} back from {query_at}, decoded {decoded}")
                seen[gap] = (got[query_at], want[query_at])
            moved = H.rms_error(seen[window - 1][1][None], seen[window][1][None])
            assert moved > SHARP
            assert all(H.rms_error(g[None], w[None]) < moved / 4 for g, w in seen.values())


@pytest.mark.parametrize("kind", ["right", "lightning"])
def test_a_state_carried_for_hundreds_of_tokens_decides_the_logits(tmp_path_factory, backend, kind):
    """Two prompts that differ in one early token only (the key token or a filler), decoded 300 tokens on through a slot that the other
    request used before, end in logits that differ by far more than the bound at the query token: a state that was lost, zeroed late, left
    over from the slot's last user or decayed once too often shows."""
    folder, cfg, weights = sharpened(tmp_path_factory, kind)
    run = Run(folder, cfg, backend, page_size=4, num_pages=100, slots=1)
    outs = {}
    for first in (KEY, 5):
        ids = [first] + filler(cfg, 305, seed=12)
        ids[301] = QUERY
        rid = f"carried{first}"
        run.step([(rid, ids[:2])])
        for t in ids[2:]:
            run.step([(rid, [t])])
        run.finish(rid)
        got, want = run.check(rid, ids, weights, f"{kind}: state carried from {first}")
        outs[first] = (got[301], want[301])
    moved = H.rms_error(outs[KEY][1][None], outs[5][1][None])
    assert moved > SHARP
    for first in (KEY, 5):
        assert H.rms_error(outs[first][0][None], outs[first][1][None]) < moved / 4


@pytest.mark.parametrize("what", ["sink", "talk", "norm1b", "norm2b", "decay", "right_scale", "o.b", "z.b"])
def test_what_is_left_out_shows(tmp_path_factory, what):
    """The plain logits of the mixed model move at most positions by more than these tests allow over all of them when one thing is left out: the tests can tell."""
    _, cfg, weights = model_dir(tmp_path_factory, "mixed", RM.MIXED, seed=len("mixed"))
    other, w = copy.deepcopy(cfg), dict(weights)
    ids = ids_for(cfg, 40, seed=2)
    if what == "decay":
        other["layers"][2]["mixer"]["decay"] = [1.0, 1.0]
    elif what == "right_scale":
        other["layers"][0]["mixer"]["right_scale"] = 1.0
    else:
        for k in w:
            if k.endswith(what):
                w[k] = torch.eye(w[k].shape[0], dtype=torch.float64) if what == "talk" else (torch.full_like(w[k], -30.0) if what == "sink" else torch.zeros_like(w[k]))
    moved = position_errors(P.forward(other, w, ids), P.forward(cfg, weights, ids))
    assert float(moved.median()) > BF16_RMS, (what, float(moved.median()))


# ------------------------------------------------------------------------------------------------ the entry point and the scheduler
def test_greedy_generation_through_the_entry_point_and_scheduler(model, backend):
    """``RoostEngine.generate`` (scheduler with a budget of 24 tokens a step, portions, decode graphs, sampler): where the plain logits have
    no near tie, the generated token is their largest."""
    name, folder, cfg, weights = model
    kind, dtype = backend
    m = H.make_model(folder, dtype, kind)
    engine = RoostEngine(m, page_size=4, attention_blocks=60, max_sequences=3, max_tokens=24, **({"device": "cpu"} if kind == "fake" else {}))
    prompts = [ids_for(cfg, n, seed=60 + n) for n in (19, 5, 31, 2)]
    outs = engine.generate(prompts, GenerationOptions(max_output_tokens=10))
    for p, out in zip(prompts, outs):
        assert out.finish_reason == "length" and len(out.token_ids) == 10
        if dtype != torch.float32:
            continue          # bfloat16 logits are checked above; a near-tie may fall the other way
        logits = P.forward(cfg, weights, list(p) + out.token_ids[:-1])
        for j, tok in enumerate(out.token_ids):
            top = logits[len(p) - 1 + j].topk(2)
            if float(top.values[0] - top.values[1]) > 1e-3:
                assert tok == int(top.indices[0]), (j, tok, int(top.indices[0]))
    assert all(pool.used_count == 0 for pool in engine.executor.cache.pools)


# ------------------------------------------------------------------------------------------------ configuration, parts and weights
def test_the_configuration_is_read_from_its_own_keys():
    cfg = ReviraxConfig.from_dict(RM.MIXED)
    assert (cfg.vocab, cfg.width, cfg.eps, len(cfg.layers), cfg.tie_word_embeddings) == (97, 40, 1e-5, 5, False)
    spec = cfg.to_spec()
    assert [b.mixer.kind for b in spec.blocks] == ["parallel", "sink_attention", "retention", "sink_attention", "parallel"]
    assert all(b.kind == "sandwich_wide" and b.input_norm.weight_offset == 1.0 and b.mixer_out_norm == b.input_norm for b in spec.blocks)
    assert spec.blocks[1].feed_forward is None and spec.blocks[1].feed_forward_out_norm is None and spec.blocks[0].feed_forward.activation == "relu_squared"
    left, right = spec.blocks[0].mixer.branches
    assert (left.window, left.bias, left.output_gate, left.out_bias, right.width) == (13, True, True, True, 11)
    assert spec.blocks[0].mixer.factors == (0.7, 1.2) and spec.blocks[4].mixer.factors == (1.3, -0.6)
    assert left.position.scaling == RotationScaling(kind="yarn", factor=4.0, original=60.0, fast=6.0, slow=1.0)
    assert spec.blocks[1].mixer.position.scaling == RotationScaling(kind="llama3", factor=3.0, original=40.0, low=1.0, high=3.0)
    assert spec.blocks[1].mixer.learned_sink and spec.blocks[1].mixer.window is None
    assert spec.blocks[2].mixer.decay == (0.9, 0.995) and spec.blocks[2].mixer.norm == "all" and spec.blocks[2].mixer.key_scale == 1.0
    assert not spec.tie_embeddings and spec.weight_names["lm_head"] == {"weight": ("head",)}
    assert ReviraxConfig.from_dict(RM.ODD).to_spec().blocks[3].mixer.position.scaling is None


@pytest.mark.parametrize("path, value, word", [
    (("layers", 0, "type"), "convolution", "type"),
    (("layers", 2, "mixer", "decay"), [0.5], "decay"),
    (("layers", 2, "mixer", "decay"), [0.5, 1.5], "decay"),
    (("layers", 1, "mixer", "rot", "dims"), 3, "dims"),
    (("layers", 1, "mixer", "rot", "dims"), 10, "dims"),
    (("layers", 1, "mixer", "rot", "scaling", "high"), 0.5, "low"),
    (("layers", 1, "mixer", "rot", "scaling", "factor"), None, "factor"),
    (("layers", 0, "mixer", "left", "rot", "scaling", "fast"), None, "fast"),
    (("layers", 0, "mixer", "left", "rot", "base"), 1.0, "base"),
    (("layers", 0, "mixer", "left", "kv_heads"), 3, "kv_heads"),
    (("layers", 0, "mixer", "left", "mask", "size"), 0, "size"),
    (("layers", 0, "mixer", "right", "width"), None, "width"),
    (("layers", 0, "mixer", "left_scale"), None, "left_scale"),
    (("layers", 1, "mixer", "scale"), 0.0, "scale"),
    (("layers", 0, "mlp", "kind"), "routed", "kind"),
    (("norm",), None, "norm"),
    (("width",), -4, "width"),
])
def test_a_faulty_configuration_is_refused_with_the_key_named(path, value, word):
    cfg = copy.deepcopy(RM.MIXED)
    node = cfg
    for k in path[:-1]:
        node = node[k]
    if value is None:
        del node[path[-1]]
    else:
        node[path[-1]] = value
    with pytest.raises(ConfigError) as e:
        ReviraxConfig.from_dict(cfg)
    assert word in str(e.value)


@pytest.mark.parametrize("dims, base, original", [(8, 300.0, 40), (64, 500000.0, 8192), (32, 10000.0, 100), (2, 7.0, 16)])
def test_scaled_frequencies_against_the_plain_ones(dims, base, original):
    for low, high in ((1.0, 4.0), (0.3, 0.9), (2.0, 40.0)):
        got, amplitude = scaled_frequencies(base, dims, RotationScaling(kind="llama3", factor=5.0, original=original, low=low, high=high))
        assert amplitude == 1.0 and got == pytest.approx(P.stepped_frequencies(dims, base, 5.0, low, high, original), rel=1e-14)
    for fast, slow in ((32.0, 1.0), (2.0, 0.5), (1.0, 1.0), (0.01, 0.001), (900.0, 800.0)):      # ramps inside, of no length, beyond either end
        got, amplitude = scaled_frequencies(base, dims, RotationScaling(kind="yarn", factor=6.0, original=original, fast=fast, slow=slow))
        want, want_amplitude = P.ramped_frequencies(dims, base, 6.0, original, fast, slow)
        assert amplitude == pytest.approx(want_amplitude) == pytest.approx(1.0 + 0.1 * math.log(6.0)) and got == pytest.approx(want, rel=1e-14)
    assert scaled_frequencies(base, dims, None) == (pytest.approx(P.plain_frequencies(dims, base), rel=1e-14), 1.0)


def _runtime():
    from tests.fake_kernels import FakeKernels
    return Runtime(torch.float32, "cpu", FakeKernels())


def test_mixers_that_do_not_scale_cosines_refuse_an_encoding_that_asks_for_it():
    yarn = PositionSpec(rotary_dim=4, theta=100.0, scaling=RotationScaling(kind="yarn", factor=4.0, original=50, fast=8.0, slow=1.0))
    assert RopeNeox(yarn, _runtime()).amplitude == pytest.approx(1.0 + 0.1 * math.log(4.0))
    with pytest.raises(ValueError, match="retention"):
        Retention(RetentionSpec(hidden=8, num_heads=1, head_dim=4, v_dim=4, decay=(0.9,), position=yarn), _runtime())


def test_a_weighted_sum_of_branches_that_do_not_split(tmp_path):
    """A retention beside a recurrence: the branches run one after another and a kernel adds their outputs; branches that split give the same
    sum from two wide products."""
    class Batch:
        def __init__(self, T):
            self.q_indptr, self.positions = torch.tensor([0, T], dtype=torch.int32), torch.arange(T, dtype=torch.int32)
            self.groups = [type("G", (), {"state_slots": torch.zeros(1, dtype=torch.int32)})() for _ in range(2)]

    view = lambda g, n: type("V", (), {"group": g, "state": torch.zeros(1, n)})()
    g = torch.Generator().manual_seed(0)
    gru, ret = MinGruSpec(hidden=12, width=7), RetentionSpec(hidden=12, num_heads=2, head_dim=3, v_dim=4, decay=(0.9, 0.8))
    x = torch.randn(9, 12, generator=g)
    for first, cls_sizes in ((ret, (2 * 3 * 4, 7)), (gru, (7, 7))):
        spec = ParallelMixerSpec(hidden=12, branches=(first, gru), combine="weighted_sum", factors=(0.5, -2.0))
        m = ParallelMixer(spec, _runtime())
        assert m.joined == (first is gru)
        params = {k: torch.randn(d.shape, generator=g) for k, d in ParallelMixer.parameters(spec).items()}
        m.load(params)
        got = m(x, Batch(9), tuple(view(i, n) for i, n in enumerate(cls_sizes)))
        want = 0
        for i, (b, f) in enumerate(zip(m.branches, spec.factors)):
            b.load({k[2:]: v for k, v in params.items() if k.startswith(f"{i}.")})
            want = want + f * b(x, Batch(9), view(i, cls_sizes[i]))
        assert torch.allclose(got, want, atol=1e-5)
    with pytest.raises(ValueError, match="factors"):
        ParallelMixer(ParallelMixerSpec(hidden=12, branches=(gru,), combine="weighted_sum"), _runtime())


def test_a_missing_or_misshapen_tensor_is_named(tmp_path):
    cfg = SINGLE["parallel_only"]
    tensors = RM.draw_tensors(cfg, 1)
    del tensors["l0.mix.left.talk"]
    tensors["l0.mix.right.z.b"] = tensors["l0.mix.right.z.b"][:-1]
    folder = RM.write_model(tmp_path / "m", cfg, tensors)
    with pytest.raises(WeightError) as e:
        H.make_model(folder, torch.float32, "fake")
    assert "l0.mix.left.talk" in e.value.missing and any(n == "l0.mix.right.z.b" for n, _, _ in e.value.wrong_shape)


# ------------------------------------------------------------------------------------------------ the programs a user runs
@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_replay_program_on_a_revirax_model(tmp_path_factory, tmp_path, dtype):
    """bin/trace_run as a subprocess: the model class found by config.json, three requests through a pool of 192 tokens (the third takes the
    pages and the slots the first gave back), portions beside single tokens, a request that sits out a step."""
    from tests.test_trace_run_gpu import TraceRun
    folder, cfg, weights = model_dir(tmp_path_factory, "mixed", RM.MIXED, seed=len("mixed"))
    a, b, c = ids_for(cfg, 70, 21), ids_for(cfg, 45, 22), ids_for(cfg, 100, 23)
    want = {k: P.forward(cfg, weights, ids) for k, ids in (("a", a), ("b", b), ("c", c))}
    run = TraceRun(folder, dtype, tmp_path, max_tokens=192)
    try:
        got_a = [run.step([("a", a[:38], list(range(38)))])]
        out = run.step([("b", b[:2], [0, 1]), ("a", a[38:40], [0, 1])])
        got_b = [out[:2]]
        got_a.append(out[2:])
        assert run.step([("b", b[2:30], [])]) is None
        out = run.step([("a", a[40:41], [0]), ("b", b[30:45], list(range(15)))], end=["b"])
        got_a.append(out[:1])
        got_b.append(out[1:])
        for i in range(41, 70):
            got_a.append(run.step([("a", a[i : i + 1], [0])], end=["a"] if i == 69 else []))
        got_c = run.step([("c", c, list(range(100)))], end=["c"])
    finally:
        run.close()
    bound = F32_TOKEN if dtype == "float32" else BF16_TOKEN
    for what, got, ref in (("a", torch.cat(got_a), want["a"]), ("b, first two", got_b[0], want["b"][:2]), ("b, last portion", got_b[1], want["b"][30:]),
                           ("c", got_c, want["c"])):
        errs = position_errors(got, ref)
        print(f"MEASURED replay {what} {dtype}: worst position's error {float(errs.max()):.3e}")
        assert float(errs.max()) < bound, (what, float(errs.max()))


@pytest.mark.gpu
def test_the_command_line_generates_from_a_revirax_model(tmp_path_factory):
    import json
    import subprocess
    import sys

    from tests.conftest import ROOT
    folder, cfg, weights = model_dir(tmp_path_factory, "odd", RM.ODD, seed=len("odd"))
    prompt = ids_for(cfg, 12, 3)
    r = subprocess.run([sys.executable, str(ROOT / "bin" / "roost"), "generate", "--model", str(folder), "--dtype", "float32", "--prompt-ids",
                        ",".join(map(str, prompt)), "--max-output-tokens", "8", "--ignore-eos", "--attention-blocks", "8", "--max-sequences", "2"],
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr
    out = json.loads(r.stdout.strip().splitlines()[-1])
    assert out["finish_reason"] == "length" and out["prompt_tokens"] == 12 and len(out["token_ids"]) == 8
    logits = P.forward(cfg, weights, list(prompt) + out["token_ids"][:-1])
    for j, tok in enumerate(out["token_ids"]):
        top = logits[len(prompt) - 1 + j].topk(2)
        if float(top.values[0] - top.values[1]) > 1e-3:
            assert tok == int(top.indices[0]), (j, tok, int(top.indices[0]))


def test_random_weights_for_a_revirax_configuration_load_and_run(tmp_path):
    """The random-weights mode writes a folder from the configuration alone (every parameter's shape and role comes from the parts'
    declarations); the loader reads it back and a step runs."""
    from roost_b200.weights.random_init import write_random_model
    write_random_model(tmp_path / "m", RM.MIXED, seed=3, std=0.05)
    model = H.make_model(tmp_path / "m", torch.float32, "fake")
    assert 0.7 < float(model.blocks[0].input_norm.weight.mean()) < 1.3, "a norm's weight stored around zero is drawn around zero"
    ex = StepExecutor(model, page_size=4, num_pages=16, max_requests=2)
    out = ex.step([StepEntry("a", [1, 2, 3], [2])])
    assert out.shape == (1, RM.MIXED["vocab"]) and bool(torch.isfinite(out).all())
