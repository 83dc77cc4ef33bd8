"""The kernels of the Zufusun parts on the device against plain formulas in float64: the norm after a sublayer that hands the stream on, the
choice of experts weighted by a softmax over the chosen, queries and keys normed over the whole projection, the attention with a window
beside the first keys (the 32-bit kernel and every tensor-core kernel), the latent attention's preparation with a query latent and
neighbouring pairs, stored sinks in both of its forms, and the gated linear attention (a row at a time, with its decays made in the
walk, and in chunks that run side by side)."""
import math

import pytest
import torch

from roost_b200.parts.attention_work import kept_chunks, plan_attention
from tests import helpers as H
from tests.plain import zufusun_plain as P

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]
ROWS = [0, 1, 16, 17, 200, 3, 64]          # tokens of every row of a step; the slots are taken in another order


def i32(values):
    return torch.tensor(values, dtype=torch.int32).cuda()


def close(got, want, dtype, what, f32=3e-5, bf16=2e-2):
    err = H.scaled_error(got.float(), want)
    print(f"MEASURED {what} {dtype}: {err:.3e}", flush=True)
    assert err < (f32 if dtype == torch.float32 else bf16), (what, err)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [8, 37, 320, 2048])
def test_the_norm_after_a_sublayer_hands_the_stream_on(kernels, dtype, width):
    g = torch.Generator().manual_seed(width)
    T = 9
    stream, a = torch.randn(T, width, generator=g), (3.0 * torch.randn(T, width, generator=g)).to(dtype)
    w = 1.0 + 0.2 * torch.randn(width, generator=g)
    dev = stream.cuda()
    out = kernels.sandwich_norm(dev, a.cuda(), w.cuda(), 1e-3, None, 1e-3)
    want = stream.double() + P.rms_norm(a.double(), w.double(), 1e-3)
    close(dev.cpu(), want, torch.float32, "stream", f32=1e-6)
    assert bool((out.cpu() == dev.cpu().to(dtype)).all()) and out.data_ptr() != dev.data_ptr()
    plain = kernels.wide_rms_norm(dev, None, 1e-3, dtype)
    assert bool((plain.cpu() == dev.cpu().to(dtype)).all())


@pytest.mark.parametrize("experts,top", [(5, 1), (16, 2), (64, 6), (33, 32), (300, 8)])
def test_experts_are_weighted_by_the_softmax_over_the_chosen(kernels, experts, top):
    g = torch.Generator().manual_seed(experts)
    T = 37
    logits = 3.0 * torch.randn(T, experts, generator=g)
    logits[3] = 0.0                                        # ties go to the lower index
    logits[4] -= 200.0                                     # far below zero: only differences count
    for scale in (1.0, 2.5):
        r = kernels.moe_route(logits.cuda(), top, score="softmax_chosen", scale=scale)
        inv, weight, expert, token = r.inverse.cpu().long(), r.weight.cpu(), r.expert.cpu(), r.token.cpu()
        for t in range(T):
            best = torch.argsort(logits[t], descending=True, stable=True)[:top]
            want = torch.softmax(logits[t, best].double(), dim=0) * scale
            at = inv[t * top : (t + 1) * top]
            assert expert[at].tolist() == best.tolist() and bool((token[at] == t).all())
            assert float((weight[at].double() - want).abs().max()) < 1e-6


class Paged:
    """Two rows of unequal length whose pages lie scattered in the pool. ``given_back`` pages of each row (a range of page indices) are -1 in
    the block table, as a window leaves them."""

    def __init__(self, lens, kv_heads, dim, vdim, dtype, page, g):
        self.lens, self.page = lens, page
        self.T = sum(lens)
        need = [-(-n // page) for n in lens]
        self.need = need
        order = torch.randperm(sum(need) + 9, generator=g).tolist()
        self.pages = [order[: need[0]], order[need[0] : sum(need)]]
        self.two = dim == vdim
        # whatever an unseen entry of a page holds must not matter
        pool = torch.full((2 if self.two else 1, sum(need) + 9, kv_heads, page, dim if self.two else dim + vdim), 5.0, dtype=dtype).cuda()
        self.k_pool, self.v_pool = pool[0], (pool[1] if self.two else None)
        self.positions = torch.cat([torch.arange(n) for n in lens]).to(torch.int32)
        self.token_row = torch.cat([torch.full((n,), i) for i, n in enumerate(lens)]).to(torch.int32)
        self.slots = torch.tensor([self.pages[int(r)][int(p) // page] * page + int(p) % page for r, p in zip(self.token_row, self.positions)], dtype=torch.int32)
        self.kv_indptr = i32([0, need[0], sum(need)])

    def table(self, first, window, keep):
        """The block tables when the rows' first tokens of a step stand at ``first``: the pages between the kept keys' and the window's are gone."""
        out = []
        for row, f in zip(self.pages, first):
            for i, p in enumerate(row):
                seen = (i + 1) * self.page > f - window + 1 or i * self.page < keep
                out.append(p if seen or not window else -1)
        return i32(out)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(4, 2, 8, 6), (3, 3, 20, 33), (6, 2, 80, 80), (8, 2, 64, 64), (5, 1, 16, 16), (4, 4, 128, 128), (32, 4, 128, 128),
                                                     (2, 1, 256, 256), (1, 1, 300, 40)])
def test_the_attention_with_a_window_beside_the_first_keys(kernels, dtype, heads, kv_heads, dim, vdim):
    g = torch.Generator().manual_seed(heads * dim + vdim)
    page = 16 if dim >= 64 else 4
    lens = [45, 403]
    pg = Paged(lens, kv_heads, dim, vdim, dtype, page, g)
    T, scale = pg.T, 1.0 / math.sqrt(dim)
    Q, K, V = heads * dim, kv_heads * dim, kv_heads * vdim
    rows = (1.5 * torch.randn(T, Q + K + V, generator=g)).to(dtype)
    qw, kw = 1.0 + 0.3 * torch.randn(Q, generator=g), 1.0 + 0.3 * torch.randn(K, generator=g)
    sinks = torch.randn(heads, generator=g)
    x = rows.double()
    qn = P.rms_norm(x[:, :Q], qw.double(), 1e-5).to(dtype).double().reshape(T, heads, dim)
    kn = P.rms_norm(x[:, Q : Q + K], kw.double(), 1e-5).to(dtype).double().reshape(T, kv_heads, dim)
    v = x[:, Q + K :].reshape(T, kv_heads, vdim)
    dev = rows.cuda()
    q_out = torch.zeros(T, heads, dim, dtype=dtype).cuda()
    kernels.sink_attention_prepare_normed(dev, pg.k_pool, pg.v_pool, pg.slots.cuda(), heads, kv_heads, dim, vdim, qw.cuda(), kw.cuda(), 1e-5, page, q_out=q_out)
    close(q_out.cpu(), qn, dtype, "normed queries", f32=2e-6, bf16=1e-2)
    assert bool((dev.cpu() == rows).all())
    kernels.sink_attention_prepare_normed(dev, pg.k_pool, pg.v_pool, torch.full_like(pg.slots, -1).cuda(), heads, kv_heads, dim, vdim, qw.cuda(), kw.cuda(), 1e-5, page)
    close(dev[:, :Q].cpu(), qn.reshape(T, Q), dtype, "normed queries in place", f32=2e-6, bf16=1e-2)      # ... and no slot: nothing cached
    group = heads // kv_heads

    for window, keep in ((40, 7), (90, 24), (33, 64), (1, 1), (64, 0), (500, 30), (130, 100)):
        want = torch.zeros(T, heads, vdim, dtype=torch.float64)
        for t in range(T):
            p, base = int(pg.positions[t]), t - int(pg.positions[t])
            js = torch.tensor(P.visible(p, window, keep)) + base
            s = torch.einsum("hd,nhd->hn", qn[t], kn[js].repeat_interleave(group, 1)) * scale
            for h in range(heads):
                want[t, h] = P.softmax_with_sink(s[h], sinks[h].double()) @ v[js, h // group]
        want = want.reshape(T, -1)
        what = f"window {window} keep {keep}"
        for kv_cap in (0, 1024):
            got = kernels.sink_attention(dev, pg.k_pool, pg.v_pool, pg.positions.cuda(), pg.token_row.cuda(), pg.kv_indptr, pg.table([0, 0], window, keep), heads,
                                         kv_heads, dim, vdim, scale, True, kv_cap=kv_cap, sinks=sinks.cuda(), window=window, keep_first=keep)
            close(got.cpu(), want, dtype, f"sink attention {what}, bound {kv_cap}")
        few = torch.tensor([44, T - 1])                        # decoding: a token's keys are dealt to several blocks, pages are gone
        for kv_cap in (0, 1024):
            got = kernels.sink_attention(dev[few.cuda()].contiguous(), pg.k_pool, pg.v_pool, pg.positions[few].cuda(), pg.token_row[few].cuda(), pg.kv_indptr,
                                         pg.table([44, lens[1] - 1], window, keep), heads, kv_heads, dim, vdim, scale, True, kv_cap=kv_cap,
                                         sinks=sinks.cuda(), window=window, keep_first=keep)
            close(got.cpu(), want[few], dtype, f"sink attention of few tokens {what}, bound {kv_cap}")
        if dtype != torch.bfloat16 or not pg.two or not kernels.attention_mma_supported(dim):
            continue

        def run(first, counts, chunk, tile_rows, cluster=0):
            """The rows' tokens from ``first`` on through the tensor-core kernels."""
            at = torch.cat([torch.arange(base + f, base + f + n) for base, f, n in zip((0, lens[0]), first, counts)])
            plan = plan_attention(first, counts, group, window, chunk, "cuda", tile_rows, cluster, keep_first=keep)
            ends = [f + n for f, n in zip(first, counts)]
            table = pg.table(first, window, keep)
            got = kernels.attention_mma(q_out[at.cuda()].contiguous(), pg.k_pool, pg.v_pool, i32([0, counts[0], sum(counts)]), i32(ends), pg.kv_indptr, table, plan,
                                        scale, window, sink=True, wide_weights=True, sinks=sinks.cuda(), keep_first=keep)
            close(got.cpu(), want[at], dtype, f"on the tensor cores {what}, {counts} tokens from {first}, chunk {chunk}, cluster {cluster}")

        run([0, 0], lens, 256, 64)
        run([30, 150], [15, 253], 256, 64)
        if dim <= 128:
            run([0, 0], lens, 256, 128)
            run([30, 150], [15, 253], 256, 128)
        for first, counts in (([44, 402], [1, 1]), ([3, 65], [1, 1]), ([0, 120], [2, 2]), ([40, 128], [1, 3])):
            for chunk in (64, 256):
                run(first, counts, chunk, 64)
                if kernels._lib.roost_attention_decode_cluster_supported(dim, page, pg.k_pool.shape[0], kv_heads, pg.k_pool.data_ptr(), pg.v_pool.data_ptr()):
                    most = kept_chunks(max(f + n for f, n in zip(first, counts)), window, keep, chunk) if keep else -(-403 // chunk)
                    if most <= 8 and max(counts) * group <= 16:
                        run(first, counts, chunk, 64, 8)
    kernels.check_device_status()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,nope,rope,rot,rank,q_rank", [(5, 48, 32, 32, 80, 112), (3, 10, 6, 4, 20, 7), (16, 128, 64, 64, 512, 384), (1, 8, 2, 2, 8, 1), (20, 16, 16, 16, 64, 40)])
def test_latent_attention_with_a_query_latent_neighbouring_pairs_and_sinks(kernels, dtype, heads, nope, rope, rot, rank, q_rank):
    g = torch.Generator().manual_seed(heads * rank)
    lens, page = [45, 203], 8
    T, E = sum(lens), rank + rope
    need = [-(-n // page) for n in lens]
    order = torch.randperm(sum(need) + 5, generator=g).tolist()
    pages = [order[: need[0]], order[need[0] : sum(need)]]
    positions = torch.cat([torch.arange(n) for n in lens]).to(torch.int32)
    token_row = torch.cat([torch.full((n,), i) for i, n in enumerate(lens)]).to(torch.int32)
    slots = torch.tensor([pages[int(r)][int(p) // page] * page + int(p) % page for r, p in zip(token_row, positions)], dtype=torch.int32)
    kv_indptr, kv_indices, q_indptr = i32([0, need[0], sum(need)]), i32(pages[0] + pages[1]), i32([0, lens[0], T])
    pool = torch.full((sum(need) + 5, 1, page, E), 5.0, dtype=dtype).cuda()
    u = torch.randn(T, q_rank + E + 8, generator=g).to(dtype)
    lw, cw = 1.0 + 0.2 * torch.randn(rank, generator=g), 1.0 + 0.2 * torch.randn(q_rank, generator=g)
    inv_freq = torch.tensor([300.0 ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float64).cuda()
    dev = u.cuda()
    sizes = (heads, nope, rope, rank, 1e-5, page)
    cq = kernels.latent_prepare(None, dev[:, q_rank : q_rank + E], pool, lw.cuda(), inv_freq, rot, positions.cuda(), slots.cuda(), *sizes, interleaved=True,
                                cq=dev[:, :q_rank], cq_w=cw.cuda())
    x = u.double()
    close(cq.cpu(), P.rms_norm(x[:, :q_rank], cw.double(), 1e-5), dtype, "query latent", f32=2e-6, bf16=1e-2)
    c = P.rms_norm(x[:, q_rank : q_rank + rank], lw.double(), 1e-5)
    r = P.rotate_neighbours(x[:, None, q_rank + rank : q_rank + E], positions, rot, 300.0)[:, 0]
    entries = pool.cpu().reshape(-1, E)[slots.long()].double()
    close(entries, torch.cat([c, r], -1), dtype, "cache entries", f32=2e-6, bf16=1e-2)
    q = torch.randn(T, heads * (nope + rope), generator=g).to(dtype)
    qd = q.cuda()
    kernels.latent_prepare(qd, None, None, None, inv_freq, rot, positions.cuda(), None, *sizes, interleaved=True)
    qh = q.double().reshape(T, heads, nope + rope)
    turned = torch.cat([qh[..., :nope], P.rotate_neighbours(qh[..., nope:], positions, rot, 300.0)], -1)
    close(qd.cpu(), turned.reshape(T, -1), dtype, "rotated queries", f32=2e-6, bf16=1e-2)
    ql = (torch.randn(heads, T, rank, generator=g) * 0.5).to(dtype)
    sinks, scale = torch.randn(heads, generator=g) + 1.0, 1.0 / math.sqrt(E)
    qr = qd.cpu().double().reshape(T, heads, nope + rope)[..., nope:]
    want = torch.zeros(heads, T, rank, dtype=torch.float64)
    for t in range(T):
        lo = t - int(positions[t])
        s = (ql[:, t].double() @ entries[lo : t + 1, :rank].T + qr[t] @ entries[lo : t + 1, rank:].T) * scale
        for h in range(heads):
            want[h, t] = P.softmax_with_sink(s[h], sinks[h].double()) @ entries[lo : t + 1, :rank]
    for kv_cap in (0, 210):
        for indptr in (None, q_indptr):            # the second: on the tensor cores where the sizes allow
            got = kernels.latent_attention(ql.cuda(), qd, pool, positions.cuda(), token_row.cuda(), kv_indptr, kv_indices, heads, nope, rope, rank, scale, None,
                                           kv_cap=kv_cap, q_indptr=indptr, sinks=sinks.cuda())
            close(got.cpu(), want, dtype, f"latent attention, bound {kv_cap}")
    few = torch.tensor([44, T - 1])
    got = kernels.latent_attention(ql[:, few].contiguous().cuda(), qd[few.cuda()].contiguous(), pool, positions[few].cuda(), token_row[few].cuda(), kv_indptr, kv_indices,
                                   heads, nope, rope, rank, scale, None, kv_cap=1024, few_rows=True, q_indptr=i32([0, 1, 2]), sinks=sinks.cuda())
    close(got.cpu(), want[:, few], dtype, "latent attention of few tokens")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,col", [(8, 0), (24, 16), (37, 3), (1024, 40), (4096, 8)])
def test_a_gate_for_every_number_of_a_row(kernels, dtype, width, col):
    g = torch.Generator().manual_seed(width)
    T = 11
    x, u = torch.randn(T, width, generator=g).to(dtype), (2.0 * torch.randn(T, col + width + 8, generator=g)).to(dtype)
    got = kernels.head_gate_mul_(x.clone().cuda(), u.cuda(), col, width)
    close(got.cpu(), x.double() * P.sigmoid(u[:, col : col + width].double()), dtype, "gate", f32=1e-6, bf16=1e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,vdim,rank,tau", [(4, 32, 48, 12, 8.0), (2, 6, 7, 3, 1.0), (1, 100, 33, 5, 4.0), (3, 128, 96, 16, 16.0), (1, 160, 40, 24, 8.0), (2, 64, 1, 1, 2.0),
                                                      (8, 64, 128, 16, 16.0), (2, 128, 20, 4, 16.0), (5, 20, 200, 9, 16.0)])
@pytest.mark.parametrize("form", ["rows", "walk", "chunks"])
def test_gated_linear_attention(kernels, dtype, heads, dim, vdim, rank, tau, form):
    g = torch.Generator().manual_seed(heads * dim + vdim)
    T = sum(ROWS)
    slots = [5, 0, 3, 1, 6, 2, 4]
    indptr = [0]
    for n in ROWS:
        indptr.append(indptr[-1] + n)
    QK, V = heads * dim, heads * vdim
    a_col = 2 * QK + 2 * V
    w, bias = torch.randn(QK, rank, generator=g).to(dtype), torch.randn(QK, generator=g) + 1.0
    state = torch.zeros(8, QK * vdim + 5).cuda()                # a slot wider than the state: the stride is the slot's
    S = torch.zeros(8, heads, dim, vdim, dtype=torch.float64)
    for call in range(2):                                       # the second call starts from what the first one left
        rows = torch.randn(T, 3 + a_col + rank, generator=g).to(dtype)
        got = kernels.gla_scan(rows.cuda()[:, 3:], a_col, w.cuda(), bias.cuda(), tau, dim ** -0.5, state, i32(indptr), i32(slots), heads, dim, vdim,
                               single=form == "walk", chunked=form == "chunks")
        x = rows[:, 3:].double()
        z = x[:, a_col : a_col + rank] @ w.double().T + bias
        alpha = (P.sigmoid(z) ** (1.0 / tau)).reshape(T, heads, dim)
        q, k, v = x[:, :QK].reshape(T, heads, dim) * dim ** -0.5, x[:, QK : 2 * QK].reshape(T, heads, dim), x[:, 2 * QK : 2 * QK + V].reshape(T, heads, vdim)
        want = torch.zeros(T, heads, vdim, dtype=torch.float64)
        for r, slot in enumerate(slots):
            for t in range(indptr[r], indptr[r + 1]):
                S[slot] = alpha[t][:, :, None] * S[slot] + k[t][:, :, None] * v[t][:, None, :]
                want[t] = torch.einsum("hd,hdv->hv", q[t], S[slot])
        close(got.cpu(), want.reshape(T, V), torch.float32, f"outputs of call {call}", f32=1e-4)
        close(state[:, : QK * vdim].cpu(), S.reshape(8, -1), torch.float32, f"states after call {call}", f32=1e-4)
