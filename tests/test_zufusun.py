"""The Zufusun decoder through the engine's step function, cache manager, scheduler and entry point, against the plain
implementation of tests/plain/zufusun_plain.py, for every way of cutting the work.

Each test runs on the GPU with the real kernel library in float32 (captured steps) and bfloat16 (marked gpu), and on the CPU with the
stand-in kernels of tests/fake_kernels.py, which checks the host side: the batch tables, the pages between the first tokens and a window that
are given back, the slots, which layer's latent a layer reads, the norm that travels with the residual from one sublayer's output to the
next.
"""
import copy
import random

import pytest
import torch

from roost_b200 import GenerationOptions, RoostEngine
from roost_b200.config.reader import ConfigError
from roost_b200.config.spec import BlockSpec, NormSpec, SinkAttentionSpec
from roost_b200.config.zufusun import ZufusunConfig
from roost_b200.engine.executor import StepEntry, StepExecutor
from roost_b200.engine.model import read_model_config
from roost_b200.parts import Runtime
from roost_b200.parts.attention_work import attention_work, kept_chunks
from roost_b200.parts.block import PostNormWideBlock
from roost_b200.parts.sink_attention import SinkAttention
from roost_b200.weights.loader import WeightError
from tests import helpers as H
from tests import zufusun_models as ZM
from tests.plain import zufusun_plain as P

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
        tensors = ZM.draw_tensors(cfg, seed)
        if change is not None:
            change(cfg, tensors)
        _MODELS[name] = (ZM.write_model(tmp_path_factory.mktemp(f"zufusun_{name}"), cfg, tensors), cfg, ZM.plain_weights(tensors))
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
            # A norm that keeps only the direction of an output next to zero moves a position's logits far for the smallest change. A position over the bound is ill-conditioned, not faulty, when rounding the plain
            # implementation's inputs and projections to 16 bits (as they are, and after a relative change of up to 2^-8) moves its logits far
            # by itself. Such positions are left out in 16 bits; the 32-bit run of the same kernels checks them.
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
    "attention_only": ZM.config([(ZM.attention(heads=2, kv_heads=1, dim=6, vdim=5, window=7, keep=3), None)], width=24, vocab=50),
    "latent_only": ZM.config([(ZM.latent(heads=2, dim=6, rot_dim=4, vdim=5, q_rank=9, kv_rank=12), None)], width=20, vocab=45),
    "latent_shared": ZM.config([(ZM.latent(heads=1, dim=6, rot_dim=4, vdim=5, q_rank=9, kv_rank=12), None),
                                (ZM.latent(heads=3, dim=5, rot_dim=4, vdim=8, q_rank=6, kv_rank=12, kv_from=0), None)], width=22, vocab=45),
    "gla_only": ZM.config([(ZM.gla(heads=2, dim=6, vdim=5, tau=4.0, decay_rank=2), None)], width=16, vocab=30),
    "moe_after_gla": ZM.config([(ZM.gla(heads=1, dim=8, vdim=8, decay_rank=4), ZM.moe(experts=4, top=2, ff=17, limit=0.5))], width=28, vocab=33),
}
ALL = dict(ZM.CONFIGS, **SINGLE)


@pytest.fixture(params=sorted(ALL))
def any_model(request, tmp_path_factory):
    return (request.param,) + model_dir(tmp_path_factory, request.param, ALL[request.param], seed=len(request.param))


@pytest.fixture(params=sorted(ZM.CONFIGS))
def model(request, tmp_path_factory):
    return (request.param,) + model_dir(tmp_path_factory, request.param, ZM.CONFIGS[request.param], seed=len(request.param))


# ------------------------------------------------------------------------------------------------ whole prompts
@pytest.mark.parametrize("length", [1, 2, 3, 37, 150])
def test_each_mechanism_and_each_model_on_whole_prompts(any_model, backend, length):
    """Models of one mechanism each and the mixed models; the shortest prompts are the first tokens of a sequence (an empty state, one key
    beside the sink); the longest reach far beyond every window and the first tokens."""
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
            kept = -(-g.keep_first // 4)
            assert run.ex.cache.pools[gi].used_count <= kept + -(-(g.window + 4) // 4) + 1, "pages between the first tokens and the window were kept"
            assert all(p >= 0 for p in run.ex.cache.get("r").tables[gi][:kept]), "a page of the first tokens was given back"
    run.finish("r")
    run.check("r", ids, weights, f"{name} long decoding")


LONG = ZM.config([(ZM.attention(heads=4, kv_heads=2, dim=16, vdim=16, scale=0.25, window=200, keep=30), ZM.moe(experts=4, top=2, ff=64)),
                  (ZM.gla(heads=2, dim=20, vdim=36, tau=16.0, decay_rank=4), None),
                  (ZM.latent(heads=4, dim=32, rot_dim=16, vdim=32, q_rank=40, kv_rank=48, scale=0.2), ZM.moe(experts=3, top=1, ff=96)),
                  (ZM.attention(heads=2, kv_heads=2, dim=16, vdim=48, scale=0.25, window=500, keep=70), None)], width=72, vocab=83)


def test_a_long_prompt_takes_the_forms_of_steps_of_many_rows(tmp_path_factory, backend):
    """700 tokens in one step and then 2 + 1: the kernels' forms for many tokens a row (the gated linear attention in chunks whose
    states are carried from chunk to chunk, the last chunk a partial one; the attentions on the tensor cores, the tiles between the first keys
    and the window left out; the experts' rows in tiles)."""
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
    "attention": ZM.config([(ZM.attention(heads=2, kv_heads=1, dim=32, vdim=32, scale=0.8, window=400, keep=2), None),
                            (ZM.gla(heads=1, dim=4, vdim=4), ZM.moe(experts=2, top=2, ff=16))], width=32, vocab=53),
    "latent_attention": ZM.config([(ZM.latent(heads=2, dim=16, rot_dim=8, vdim=6, q_rank=24, kv_rank=32, scale=0.3), None),
                                   (ZM.gla(heads=1, dim=4, vdim=4), ZM.moe(experts=2, top=2, ff=16))], width=32, vocab=53),
    "gla": ZM.config([(ZM.gla(heads=2, dim=12, vdim=6), None),
                      (ZM.attention(heads=1, kv_heads=1, dim=4, vdim=4), ZM.moe(experts=2, top=2, ff=16))], width=32, vocab=53),
}


def sharpened(tmp_path_factory, kind, cfg=None, name=None):
    def change(c, t):
        ZM.sharpen(c, t, KEY, QUERY, part=kind)
        for n in ("l1.norm1", "l1.norm2"):                # the second layer stays small beside what the first one carries
            t[n] = (0.2 * t[n].float()).to(torch.bfloat16)
        t["l0.norm1"] = (2.0 * t["l0.norm1"].float()).to(torch.bfloat16)
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
    cfg = copy.deepcopy(FAR["attention"])
    cfg["layers"][0]["mixer"]["mask"] = {"size": window, "keep_first": 5}
    folder, cfg, weights = sharpened(tmp_path_factory, "attention", cfg, f"window{window}")
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


@pytest.mark.parametrize("keep", [1, 4, 5, 31, 32, 33, 64, 70])
def test_the_first_tokens_stay_visible_and_the_next_ones_do_not(tmp_path_factory, backend, keep):
    """The key token at position ``keep`` - 1 (the last one that every later query sees) and at ``keep`` (the first one that a window of 20 has
    passed), read far on at several offsets of a page and a tile, in a prompt's portion and decoded, after the pages between the first tokens
    and the window were given back and taken by another request."""
    cfg = copy.deepcopy(FAR["attention"])
    cfg["layers"][0]["mixer"]["mask"] = {"size": 20, "keep_first": keep}
    folder, cfg, weights = sharpened(tmp_path_factory, "attention", cfg, f"keep{keep}")
    run = Run(folder, cfg, backend, page_size=4, num_pages=80)
    for query_at in (127, 128, 131):
        for decoded in (False, True):
            seen = {}
            for at in (keep - 1, keep):
                ids = filler(cfg, query_at + 2, seed=query_at)
                ids[at], ids[query_at] = KEY, QUERY
                rid, other = f"k{query_at}_{at}_{decoded}", f"o{query_at}_{at}_{decoded}"
                run.step([(rid, ids[:70])])
                if decoded:
                    run.step([(rid, ids[70 : query_at - 3]), (other, filler(cfg, 60, seed=1))])
                    for t in ids[query_at - 3 :]:
                        run.step([(rid, [t])])
                else:
                    run.step([(other, filler(cfg, 60, seed=1))])
                    run.step([(rid, ids[70:])])
                run.finish(rid)
                run.finish(other)
                run.logits.pop(other)
                got, want = run.check(rid, ids, weights, f"keep {keep}, key at {at}, query at {query_at}, decoded {decoded}")
                seen[at] = (got[query_at], want[query_at])
            moved = H.rms_error(seen[keep - 1][1][None], seen[keep][1][None])
            assert moved > SHARP
            assert all(H.rms_error(g[None], w[None]) < moved / 4 for g, w in seen.values())


@pytest.mark.parametrize("kind", ["gla"])
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


@pytest.mark.parametrize("what", ["sink", "keep_first", "q.norm", "dq.norm", "q.b", "v.b", "a2.b", "mix.g", "tau", "limit", "top", "norm1", "norm2", "kv_from", "base"])
def test_what_is_left_out_shows(tmp_path_factory, what):
    """The plain logits of the mixed model move at most positions by more than these tests allow over all of them when one thing is left out or
    changed: the tests can tell."""
    _, cfg, weights = model_dir(tmp_path_factory, "mixed", ZM.MIXED, seed=len("mixed"))
    other, w = copy.deepcopy(cfg), dict(weights)
    ids = ids_for(cfg, 40, seed=2)
    for i, layer in enumerate(other["layers"]):
        m, f = layer["mixer"], layer["mlp"]
        if what == "keep_first" and "mask" in m:
            m["mask"]["keep_first"] = 0
        elif what == "tau" and layer["type"] == "gla":
            m["tau"] = 1.0
        elif what == "limit" and f is not None:
            f["expert"]["limit"] = 1e9
        elif what == "top" and f is not None:
            f["router"]["top"] = min(f["router"]["top"] + 1, f["router"]["experts"])
        elif what == "base" and "rot" in m:
            m["rot"]["base"] = 1.0
        elif what == "kv_from" and "kv_from" in m:       # a latent of its own, made with the other layer's matrices
            del m["kv_from"]
            for n in ("dkv", "dkv.norm"):
                w[f"l{i}.mix.{n}"] = w["l0.mix." + n]
    for k in w:
        if k.endswith("." + what):
            w[k] = torch.full_like(w[k], -30.0) if what == "sink" else (torch.ones_like(w[k]) if "norm" in what else torch.zeros_like(w[k]))
    moved = position_errors(P.forward(other, w, ids), P.forward(cfg, weights, ids))
    late = moved[15:]                                     # past the windows, where what is kept counts
    assert float(late.median()) > BF16_RMS, (what, float(late.median()))


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
    cfg = ZufusunConfig.from_dict(ZM.MIXED)
    assert (cfg.vocab, cfg.width, cfg.eps, len(cfg.layers), cfg.tie_word_embeddings) == (97, 40, 1e-5, 5, True)
    cfg.take_shapes({k: tuple(s) for k, s in ZM.tensor_shapes(ZM.MIXED).items()})
    spec = cfg.to_spec()
    assert [b.mixer.kind for b in spec.blocks] == ["latent_attention", "sink_attention", "gated_linear_attention", "latent_attention", "sink_attention"]
    assert all(b.kind == "post_norm_wide" and b.input_norm is None and b.post_mixer_norm is None and b.mixer_out_norm.weight_offset == 0.0 for b in spec.blocks)
    first, att, lin, shared, last = (b.mixer for b in spec.blocks)
    assert (first.q_rank, first.kv_rank, first.rope_dim, first.learned_sink, first.output_gate, first.own_latent, first.window) == (11, 14, 6, True, True, True, None)
    assert first.position.kind == "rope_interleaved" and first.position.theta == 300.0 and first.position.rotary_dim == 6
    assert not shared.own_latent and shared.q_rank == 7 and [e.reads_cache_of for e in spec.schedule] == [None, None, None, 0, None]
    assert (att.window, att.keep_first, att.bias, att.learned_sink, att.joined_norm_eps, att.position) == (13, 5, True, True, 1e-5, None)
    assert (last.window, last.keep_first) == (5, 9) and (lin.tau, lin.decay_rank) == (8.0, 3)
    f = spec.blocks[1].feed_forward
    assert (f.score, f.weight_on, f.activation, f.limit, f.experts, f.top, f.shared_intermediate) == ("softmax_chosen", "output", "clamped_swish", 2.5, 4, 3, 0)
    assert spec.blocks[2].feed_forward is None and spec.blocks[2].feed_forward_out_norm is None
    assert spec.tie_embeddings and "lm_head" not in spec.weight_names and spec.embedding.scale == 1.0


def test_the_decays_rank_comes_from_the_checkpoint(tmp_path):
    folder = ZM.write_model(tmp_path / "m", ZM.ODD, ZM.draw_tensors(ZM.ODD, 1))
    _, cfg, _ = read_model_config(folder)
    assert [m.mixer["decay_rank"] for m in cfg.layers if m.type == "gla"] == [1, 5]
    (folder / "model.safetensors").unlink()
    assert all(m.mixer["decay_rank"] == 16 for m in read_model_config(folder)[1].layers if m.type == "gla")


@pytest.mark.parametrize("path, value, word", [
    (("layers", 0, "type"), "convolution", "type"),
    (("layers", 0, "mixer", "rot", "dims"), 3, "dims"),
    (("layers", 0, "mixer", "rot", "dims"), 8, "dims"),
    (("layers", 0, "mixer", "rot", "base"), -1.0, "base"),
    (("layers", 0, "mixer", "q_rank"), None, "q_rank"),
    (("layers", 0, "mixer", "scale"), 0.0, "scale"),
    (("layers", 3, "mixer", "kv_from"), 1, "kv_from"),
    (("layers", 3, "mixer", "kv_from"), 3, "kv_from"),
    (("layers", 3, "mixer", "kv_rank"), 15, "kv_rank"),
    (("layers", 3, "mixer", "rot", "base"), 500.0, "rot_base"),
    (("layers", 1, "mixer", "kv_heads"), 3, "kv_heads"),
    (("layers", 1, "mixer", "mask"), None, "mask"),
    (("layers", 1, "mixer", "mask", "size"), 0, "size"),
    (("layers", 1, "mixer", "mask", "keep_first"), -1, "keep_first"),
    (("layers", 2, "mixer", "tau"), None, "tau"),
    (("layers", 0, "mlp", "kind"), "dense", "kind"),
    (("layers", 0, "mlp", "router", "top"), 6, "top"),
    (("layers", 0, "mlp", "expert", "limit"), None, "limit"),
    (("norm",), None, "norm"),
    (("width",), -4, "width"),
])
def test_a_faulty_configuration_is_refused_with_the_key_named(path, value, word):
    cfg = copy.deepcopy(ZM.MIXED)
    node = cfg
    for k in path[:-1]:
        node = node[k]
    if value is None:
        del node[path[-1]]
    else:
        node[path[-1]] = value
    with pytest.raises(ConfigError) as e:
        ZufusunConfig.from_dict(cfg)
    assert word in str(e.value)


def _runtime():
    from tests.fake_kernels import FakeKernels
    return Runtime(torch.float32, "cpu", FakeKernels())


@pytest.mark.parametrize("change, word", [({"keep_first": 3, "window": None}, "kept"), ({"keep_first": -1}, "kept"), ({"keep_first": 3, "softcap": 2.0}, "cap"),
                                          ({"joined_norm_eps": 0.0}, "eps"), ({"joined_norm_eps": 1e-5, "unit_norm_eps": 1e-5}, "unit")])
def test_options_that_do_not_go_together_are_refused(change, word):
    with pytest.raises(ValueError, match=word):
        SinkAttention(SinkAttentionSpec(**dict(dict(hidden=8, num_heads=2, num_kv_heads=1, head_dim=4, v_dim=4, scale=0.5, window=9), **change)), _runtime())


def test_an_arrangement_without_norms_before_its_sublayers_refuses_them():
    norm = NormSpec(size=8, eps=1e-5, kind="rms_norm_wide")
    mixer = SinkAttentionSpec(hidden=8, num_heads=2, num_kv_heads=1, head_dim=4, v_dim=4, scale=0.5)
    with pytest.raises(ValueError, match="as it is"):
        PostNormWideBlock(BlockSpec(mixer=mixer, feed_forward=None, input_norm=norm, post_mixer_norm=None, kind="post_norm_wide", mixer_out_norm=norm), _runtime())
    with pytest.raises(ValueError, match="after it"):
        PostNormWideBlock(BlockSpec(mixer=mixer, feed_forward=None, input_norm=None, post_mixer_norm=None, kind="post_norm_wide"), _runtime())


def test_the_work_lists_cover_the_window_and_the_first_keys_once():
    """Every key that a token sees is in exactly one of its row's decode items, and no row has more items than the bound that sizes a captured
    step's tables and the kernels' clusters."""
    rng = random.Random(1)
    for _ in range(3000):
        chunk, window, keep, group = rng.choice([64, 128, 512]), rng.randint(1, 700), rng.randint(1, 300), rng.choice([1, 2, 4, 16])
        n, start = rng.randint(1, 16 // group), rng.randint(0, 3000)
        _, items, merge, slots = attention_work([start], [n], group, window, chunk, keep_first=keep)
        most = kept_chunks(start + n + rng.randint(0, 100), window, keep, chunk)
        assert len(items) // 4 <= most and len(merge) == (4 if len(items) > 4 else 0) and slots == (len(items) // 4 if len(items) > 4 else 0)
        _, fixed, no_merge, _ = attention_work([start], [n], group, window, chunk, cluster=most, keep_first=keep)
        assert len(fixed) == 4 * most and not no_merge
        for i in range(start, start + n):
            got = []
            for x in range(0, len(items), 4):
                _, first, end, _ = items[x : x + 4]
                got += [j for j in (range(-1 - first, end) if first < 0 else range(max(first, keep, i - window + 1), end)) if j <= i]
            assert sorted(got) == P.visible(i, window, keep), (start, n, window, keep, chunk)


def test_a_missing_or_misshapen_tensor_is_named(tmp_path):
    cfg = ZM.MIXED
    tensors = ZM.draw_tensors(cfg, 1)
    del tensors["l1.mix.k.norm"]
    tensors["l2.mix.a2.b"] = tensors["l2.mix.a2.b"][:-1]
    folder = ZM.write_model(tmp_path / "m", cfg, tensors)
    with pytest.raises(WeightError) as e:
        H.make_model(folder, torch.float32, "fake")
    assert "l1.mix.k.norm" in e.value.missing and any(n == "l2.mix.a2.b" for n, _, _ in e.value.wrong_shape)


# ------------------------------------------------------------------------------------------------ the programs a user runs
@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_replay_program_on_a_zufusun_model(tmp_path_factory, tmp_path, dtype):
    """bin/trace_run as a subprocess: the model class found by config.json, three requests through a pool of 192 tokens (the third takes the
    pages and the slots the first gave back), portions beside single tokens, a request that sits out a step."""
    from tests.test_trace_run_gpu import TraceRun
    folder, cfg, weights = model_dir(tmp_path_factory, "mixed", ZM.MIXED, seed=len("mixed"))
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
def test_the_command_line_generates_from_a_zufusun_model(tmp_path_factory):
    import json
    import subprocess
    import sys

    from tests.conftest import ROOT
    folder, cfg, weights = model_dir(tmp_path_factory, "odd", ZM.ODD, seed=len("odd"))
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


def test_random_weights_for_a_zufusun_configuration_load_and_run(tmp_path):
    """The random-weights mode writes a folder from the configuration alone (every parameter's shape and role comes from the parts'
    declarations); the loader reads it back and a step runs."""
    from roost_b200.weights.random_init import write_random_model
    write_random_model(tmp_path / "m", {k: v for k, v in ZM.MIXED.items() if k != "_ranks"}, seed=3, std=0.05)
    model = H.make_model(tmp_path / "m", torch.float32, "fake")
    assert model.blocks[2].mixer.spec.decay_rank == 16
    ex = StepExecutor(model, page_size=4, num_pages=16, max_requests=2)
    out = ex.step([StepEntry("a", [1, 2, 3], [2])])
    assert out.shape == (1, ZM.MIXED["vocab"]) and bool(torch.isfinite(out).all())
