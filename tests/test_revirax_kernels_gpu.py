"""The kernels of the Revirax parts on the device against plain formulas in float64: the attention that mixes its scores across the heads
(both forms, windows, splits, cache entries of one plane and of two), the attention with stored sinks (the 32-bit kernel and every
tensor-core kernel), scaled rotations, the recurrence whose gates read only the current token and the retention over activated
projections (walked a row at a time and in chunks that run side by side), the norm after a sublayer fused with the next one, the squared
relu, the weighted sum and the norm over all heads."""
import math

import pytest
import torch

from roost_b200.parts.attention_work import plan_attention
from tests import helpers as H
from tests.plain import revirax_plain as P

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]
ROWS = [0, 1, 16, 17, 200, 3, 64]          # tokens of every row of a step; the slots are taken in another order


def i32(values):
    return torch.tensor(values, dtype=torch.int32).cuda()


def close(got, want, dtype, what, f32=3e-5, bf16=2e-2):
    err = H.scaled_error(got.float(), want)
    print(f"MEASURED {what} {dtype}: {err:.3e}")
    assert err < (f32 if dtype == torch.float32 else bf16), (what, err)


class Paged:
    """Two rows of unequal length whose pages lie scattered in the pool, keys and values of given tensors [T, kv heads, .] in it."""

    def __init__(self, lens, kv_heads, dim, vdim, dtype, page, g):
        self.lens, self.page = lens, page
        self.T = sum(lens)
        need = [-(-n // page) for n in lens]
        order = torch.randperm(sum(need) + 9, generator=g).tolist()
        self.pages = [order[: need[0]], order[need[0] : sum(need)]]
        self.two = dim == vdim
        # whatever an unseen entry of a page holds must not matter
        pool = torch.full((2 if self.two else 1, sum(need) + 9, kv_heads, page, dim if self.two else dim + vdim), 5.0, dtype=dtype).cuda()
        self.k_pool, self.v_pool = pool[0], (pool[1] if self.two else None)
        self.positions = torch.cat([torch.arange(n) for n in lens]).to(torch.int32)
        self.token_row = torch.cat([torch.full((n,), i) for i, n in enumerate(lens)]).to(torch.int32)
        self.slots = torch.tensor([self.pages[int(r)][int(p) // page] * page + int(p) % page for r, p in zip(self.token_row, self.positions)], dtype=torch.int32)
        self.kv_indptr, self.kv_indices = i32([0, need[0], sum(need)]), i32(self.pages[0] + self.pages[1])
        self.q_indptr, self.kv_lens = i32([0, lens[0], self.T]), i32(lens)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,window", [(4, 2, 8, 6, 21), (3, 3, 20, 33, None), (1, 1, 48, 48, 40), (8, 2, 64, 64, 32), (12, 4, 32, 128, 33),
                                                            (16, 4, 128, 128, 100), (32, 8, 128, 128, 70), (20, 5, 64, 32, None), (32, 4, 64, 64, 96), (2, 1, 272, 16, 64),
                                                            (24, 2, 48, 112, 64)])
def test_the_attention_that_mixes_its_scores_across_the_heads(kernels, dtype, heads, kv_heads, dim, vdim, window):
    g = torch.Generator().manual_seed(heads * dim + vdim)
    pg = Paged([45, 203], kv_heads, dim, vdim, dtype, 16 if dim == 64 else 4, g)
    T, scale, out_scale = pg.T, 1.3 / math.sqrt(dim), 0.8
    width = (heads + kv_heads) * dim + kv_heads * vdim
    rows = torch.randn(T, 4 + width + heads * vdim, generator=g).to(dtype)          # other columns before, the gate's columns after
    talk = (torch.eye(heads) + 0.4 * torch.randn(heads, heads, generator=g)).to(torch.bfloat16).float()
    dev = rows.cuda()
    u, gate = dev[:, 4 : 4 + width], dev[:, 4 + width :]
    rot = min(dim, 16)
    freqs, amplitude = P.ramped_frequencies(rot, 3000.0, 4.0, 60, 8.0, 1.0)
    q = torch.zeros(T, heads, dim, dtype=dtype).cuda()
    kernels.sink_attention_prepare(u, pg.k_pool, pg.v_pool, torch.tensor(freqs, dtype=torch.float64).cuda(), rot, pg.positions.cuda(), pg.slots.cuda(), heads,
                                   kv_heads, dim, vdim, None, pg.page, q_out=q, halves=True, amplitude=amplitude)
    x = rows[:, 4 : 4 + width].double()
    Q, K = heads * dim, kv_heads * dim
    rd = lambda t: t.to(dtype).double()
    qn = rd(P.rotate(x[:, :Q].reshape(T, heads, dim), pg.positions, rot, freqs, amplitude))
    kn = rd(P.rotate(x[:, Q : Q + K].reshape(T, kv_heads, dim), pg.positions, rot, freqs, amplitude))
    v = x[:, Q + K : width].reshape(T, kv_heads, vdim)
    close(q.cpu(), qn, dtype, "prepared queries", bf16=1e-2)
    want = torch.zeros(T, heads, vdim, dtype=torch.float64)
    group = heads // kv_heads
    for t in range(T):
        p = int(pg.positions[t])
        lo = t - min(p, window - 1 if window else p)
        own = torch.einsum("hd,nhd->hn", qn[t], kn[lo : t + 1].repeat_interleave(group, 1)) * scale
        want[t] = torch.einsum("hn,nhd->hd", torch.softmax(talk.double() @ own, dim=-1), v[lo : t + 1].repeat_interleave(group, 1))
    plain = want.reshape(T, -1)
    gated = plain * P.sigmoid(rows[:, 4 + width :].double()) * out_scale

    def run(some, gate_rows, factor, kv_cap, **more):
        at = torch.arange(T) if some is None else some
        wide = torch.full((at.numel(), heads * vdim + 6), 7.0, dtype=dtype).cuda()
        kernels.talking_attention(q[at.cuda()].contiguous(), wide[:, 2 : 2 + heads * vdim], pg.k_pool, pg.v_pool, gate_rows[at.cuda()] if gate_rows is not None else None,
                                  talk.cuda(), pg.positions[at].cuda(), pg.token_row[at].cuda(), pg.kv_indptr, pg.kv_indices, kv_heads, vdim, scale,
                                  window=window, out_scale=factor, kv_cap=kv_cap, **more)
        assert bool((wide[:, :2] == 7.0).all()) and bool((wide[:, 2 + heads * vdim :] == 7.0).all()), "columns beside the output were written"
        return wide[:, 2 : 2 + heads * vdim].cpu()

    for kv_cap in (0, 210):
        close(run(None, gate, out_scale, kv_cap), gated, dtype, f"talking attention, bound {kv_cap}")
    close(run(None, None, 1.0, 210), plain, dtype, "talking attention without a gate")
    few = torch.tensor([31, 44, 45, 45 + 63, 45 + 64, T - 1])         # a step of few tokens deals every token's keys to several blocks
    for kv_cap in (210, 1024, 64):                                    # the last: a bound the second row exceeds
        close(run(few, gate, out_scale, kv_cap), gated[few], dtype, f"talking attention of few tokens, bound {kv_cap}")
    if dtype == torch.bfloat16 and kernels.talking_attention_mma_supported(heads, kv_heads, dim, vdim, pg.two):
        close(run(None, gate, out_scale, 210, q_indptr=pg.q_indptr), gated, dtype, "talking attention on the tensor cores")
        close(run(None, None, 1.0, 210, q_indptr=pg.q_indptr), plain, dtype, "talking attention on the tensor cores without a gate")
        # a tile of queries whose keys are dealt to several blocks, in chunks of one and of two tiles of 32 keys
        kept = kernels.TALKING_MMA_CHUNK_TILES
        try:
            for tiles, kv_cap in ((1, 1024), (2, 1024), (1, 64)):          # the last: a bound the second row exceeds
                kernels.TALKING_MMA_CHUNK_TILES = tiles
                close(run(None, gate, out_scale, kv_cap, q_indptr=pg.q_indptr), gated, dtype, f"talking attention on the tensor cores, chunks of {tiles}")
        finally:
            kernels.TALKING_MMA_CHUNK_TILES = kept
        # portions that start in the middle of the rows, one token beside many
        part = torch.cat([torch.arange(44, 45), torch.arange(45 + 97, T)])
        close(run(part, gate, out_scale, 210, q_indptr=i32([0, 1, part.numel()])), gated[part], dtype, "talking attention on the tensor cores, later portions")


def test_which_sizes_the_tensor_core_form_serves(kernels):
    served = [(4, 2, 64, 64), (16, 4, 128, 128), (32, 8, 64, 64), (32, 8, 128, 128), (20, 5, 16, 128), (1, 1, 16, 16), (24, 2, 48, 112)]
    for heads, kv, dim, vdim in served:
        assert kernels.talking_attention_mma_supported(heads, kv, dim, vdim, dim == vdim), (heads, kv, dim, vdim)
    for heads, kv, dim, vdim in [(4, 2, 24, 64), (4, 2, 64, 40), (4, 2, 64, 144), (64, 64, 128, 128)]:
        assert not kernels.talking_attention_mma_supported(heads, kv, dim, vdim, dim == vdim), (heads, kv, dim, vdim)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,page", [(4, 2, 8, 6, 4), (3, 3, 20, 20, 4), (6, 2, 64, 64, 16), (4, 1, 128, 128, 16), (8, 2, 32, 32, 8), (2, 2, 48, 96, 4)])
def test_the_attention_with_a_stored_sink_a_head(kernels, dtype, heads, kv_heads, dim, vdim, page):
    """Sinks from far below every score to far above: one head nearly ignores its sink, one gives it nearly everything."""
    g = torch.Generator().manual_seed(heads * dim + vdim)
    pg = Paged([45, 203], kv_heads, dim, vdim, dtype, page, g)
    T, scale = pg.T, 1.5 / math.sqrt(dim)
    width = (heads + kv_heads) * dim + kv_heads * vdim
    rows = torch.randn(T, width, generator=g).to(dtype)
    sinks = torch.linspace(-9.0, 7.0, heads)
    dev = rows.cuda()
    q = torch.zeros(T, heads, dim, dtype=dtype).cuda()
    args = (None, 0, pg.positions.cuda(), pg.slots.cuda(), heads, kv_heads, dim, vdim, None, page)
    kernels.sink_attention_prepare(dev, pg.k_pool, pg.v_pool, *args, q_out=q)
    x = rows.double()
    Q, K = heads * dim, kv_heads * dim
    qx, kx, v = x[:, :Q].reshape(T, heads, dim), x[:, Q : Q + K].reshape(T, kv_heads, dim), x[:, Q + K :].reshape(T, kv_heads, vdim)
    for window in (None, 37):
        want = torch.zeros(T, heads, vdim, dtype=torch.float64)
        for t in range(T):
            p = int(pg.positions[t])
            lo = t - min(p, window - 1 if window else p)
            for h in range(heads):
                e = torch.exp((kx[lo : t + 1, h // (heads // kv_heads)] @ qx[t, h]) * scale)
                want[t, h] = (e @ v[lo : t + 1, h // (heads // kv_heads)]) / (e.sum() + math.exp(float(sinks[h])))
        want = want.reshape(T, -1)
        more = {"window": window} if window else {}
        for kv_cap in (0, 210):
            got = kernels.sink_attention(dev, pg.k_pool, pg.v_pool, pg.positions.cuda(), pg.token_row.cuda(), pg.kv_indptr, pg.kv_indices, heads, kv_heads,
                                         dim, vdim, scale, True, kv_cap=kv_cap, sinks=sinks.cuda(), **more)
            close(got.cpu(), want, dtype, f"sink attention, window {window}, bound {kv_cap}")
        if dtype != torch.bfloat16 or not pg.two or not kernels.attention_mma_supported(dim):
            continue
        group = heads // kv_heads

        def run(first, counts, chunk, tile_rows, cluster=0):
            """The rows' last tokens from ``first`` on through the tensor-core kernels."""
            at = torch.cat([torch.arange(base + f, base + f + n) for base, f, n in zip((0, 45), first, counts)])
            plan = plan_attention(first, counts, group, window, chunk, "cuda", tile_rows, cluster)
            lens = i32([f + n for f, n in zip(first, counts)])
            got = kernels.attention_mma(q[at.cuda()].contiguous(), pg.k_pool, pg.v_pool, i32([0, counts[0], sum(counts)]), lens, pg.kv_indptr, pg.kv_indices, plan,
                                        scale, window, sink=True, wide_weights=True, sinks=sinks.cuda())
            close(got.cpu(), want[at], dtype, f"sink attention on the tensor cores, {counts} tokens, chunk {chunk}, cluster {cluster}")

        run([0, 0], [45, 203], 256, 64)
        if dim <= 128:
            run([0, 0], [45, 203], 256, 128)
        run([44, 202], [1, 1], 256, 64)              # decoding: a chunk a row
        run([44, 202], [1, 1], 64, 64)               # several chunks a row, merged by a kernel of their own
        if kernels._lib.roost_attention_decode_cluster_supported(dim, page, pg.k_pool.shape[0], kv_heads, pg.k_pool.data_ptr(), pg.v_pool.data_ptr()):
            run([44, 202], [1, 1], 64, 64, cluster=4)    # ... or by the row's cluster


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [1, 37, 288])
@pytest.mark.parametrize("chunked", [False, True])
def test_the_recurrence_whose_gates_read_only_the_current_token(kernels, dtype, width, chunked):
    g = torch.Generator().manual_seed(width)
    T = sum(ROWS)
    slots = [5, 0, 3, 1, 6, 2, 4]
    indptr = [0]
    for n in ROWS:
        indptr.append(indptr[-1] + n)
    zb, xb = torch.randn(width, generator=g) - 3.0, torch.randn(width, generator=g)
    state = torch.zeros(8, width + 3).cuda()                    # a slot wider than the state: the stride is the slot's
    S = torch.zeros(8, width, dtype=torch.float64)
    for call in range(2):                                       # the second call starts from what the first one left
        rows = (2.0 * torch.randn(T, 5 + 3 * width, generator=g)).to(dtype)
        wide = torch.full((T, width + 4), 7.0, dtype=dtype).cuda()
        kernels.min_gru_scan(rows.cuda()[:, 5:], wide[:, 3 : 3 + width], zb.cuda(), xb.cuda(), 0.75, state, i32(indptr), i32(slots), width, chunked=chunked)
        x = rows[:, 5:].double()
        z, u, gate = P.sigmoid(x[:, :width] + zb), x[:, width : 2 * width] + xb, x[:, 2 * width :]
        c = torch.where(u >= 0, u + 0.5, P.sigmoid(u))
        want = torch.zeros(T, width, dtype=torch.float64)
        for r, slot in enumerate(slots):
            for t in range(indptr[r], indptr[r + 1]):
                S[slot] = (1 - z[t]) * S[slot] + z[t] * c[t]
                want[t] = S[slot] * P.silu(gate[t]) * 0.75
        close(wide[:, 3 : 3 + width].cpu(), want, dtype, f"min_gru, chunked {chunked}, call {call}")
        assert bool((wide[:, :3] == 7.0).all()) and bool((wide[:, 3 + width :] == 7.0).all())
        close(state[:, :width].cpu(), S, torch.float32, "the states it leaves")
        assert bool((state[7] == 0).all()), "a slot of no row was written"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,vdim", [(2, 20, 36), (1, 64, 70), (3, 100, 32), (1, 160, 40)])
@pytest.mark.parametrize("chunked", [False, True])
@pytest.mark.parametrize("activation", ["none", "silu"])
def test_the_retention_over_rows_that_nothing_rotates(kernels, dtype, heads, dim, vdim, chunked, activation):
    g = torch.Generator().manual_seed(heads * dim + vdim)
    T = sum(ROWS)
    slots = [5, 0, 3, 1, 6, 2, 4]
    indptr = [0]
    for n in ROWS:
        indptr.append(indptr[-1] + n)
    decay = torch.tensor([0.0, 0.97, 1.0][:heads] if heads > 1 else [0.99], dtype=torch.float32)
    state = torch.zeros(8, heads * dim * vdim).cuda()
    S = torch.zeros(8, heads, dim, vdim, dtype=torch.float64)
    act = P.silu if activation == "silu" else (lambda t: t)
    for call in range(2):
        rows = (0.5 * torch.randn(T, heads * (2 * dim + vdim) + 3, generator=g)).to(dtype)
        got = kernels.retention_scan_raw(rows.cuda(), state, decay.cuda(), i32(indptr), i32(slots), heads, dim, vdim, activation=activation, k_scale=0.3,
                                         chunked=chunked)
        x = act(rows.double())
        q, k = x[:, : heads * dim].reshape(T, heads, dim), 0.3 * x[:, heads * dim : 2 * heads * dim].reshape(T, heads, dim)
        v = x[:, 2 * heads * dim : heads * (2 * dim + vdim)].reshape(T, heads, vdim)
        want = torch.zeros(T, heads, vdim, dtype=torch.float64)
        for r, slot in enumerate(slots):
            for t in range(indptr[r], indptr[r + 1]):
                S[slot] = decay.double()[:, None, None] * S[slot] + k[t][:, :, None] * v[t][:, None, :]
                want[t] = torch.einsum("hdv,hd->hv", S[slot], q[t])
        close(got.cpu(), want.reshape(T, -1), torch.float32, f"retention, {activation}, chunked {chunked}, call {call}")
        close(state.cpu().reshape(8, heads, dim, vdim), S, torch.float32, "the states it leaves")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden", [5, 40, 192, 2048, 9000])
def test_the_norm_after_a_sublayer_and_the_next_one_in_one_pass(kernels, dtype, hidden):
    g = torch.Generator().manual_seed(hidden)
    T = 11
    stream, y = 3.0 * torch.randn(T, hidden, generator=g), (4.0 * torch.randn(T, hidden, generator=g)).to(dtype)
    pw, w = 1.0 + 0.2 * torch.randn(hidden, generator=g), 1.0 + 0.2 * torch.randn(hidden, generator=g)
    total = stream.double() + P.rms_norm(y.double(), pw.double(), 1e-3)
    want = P.rms_norm(total, w.double(), 1e-5)
    dev = stream.cuda()
    got = kernels.sandwich_norm(dev, y.cuda(), pw.cuda(), 1e-3, w.cuda(), 1e-5)
    close(got.cpu(), want, dtype, "sandwich norm")
    close(dev.cpu(), total, torch.float32, "the stream it leaves")
    dev = stream.cuda()
    some = [7, 0, 10]
    got = kernels.sandwich_norm(dev, y.cuda(), pw.cuda(), 1e-3, w.cuda(), 1e-5, rows=i32(some))
    close(got.cpu(), want[some], dtype, "sandwich norm of some rows")
    assert bool((dev.cpu() == stream).all()), "the gathering form writes no stream"


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_squared_relu_and_the_weighted_sum(kernels, dtype):
    g = torch.Generator().manual_seed(0)
    for shape in ((3, 7), (16, 64), (1, 4096)):
        a, b, c = (torch.randn(*shape, generator=g).to(dtype) for _ in range(3))
        close(kernels.relu_squared(a.cuda()).cpu(), torch.clamp(a.double(), min=0) ** 2, dtype, "relu squared", f32=1e-6)
        got = kernels.weighted_sum([a.cuda(), b.cuda(), c.cuda()], [0.5, -1.25, 3.0])
        close(got.cpu(), 0.5 * a.double() - 1.25 * b.double() + 3.0 * c.double(), dtype, "weighted sum", f32=1e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [33, 256, 2048])
@pytest.mark.parametrize("gate", ["sigmoid", "silu"])
def test_the_norm_over_all_heads_with_a_weight_and_a_gate(kernels, dtype, width, gate):
    g = torch.Generator().manual_seed(width)
    T = 9
    o, w = 2.0 * torch.randn(T, width, generator=g), 1.0 + 0.3 * torch.randn(width, generator=g)
    u = torch.randn(T, 5 + width, generator=g).to(dtype)
    got = kernels.head_norm_gate(o.cuda(), u.cuda(), 5, w.cuda(), 1, 1e-5, dtype, gate=gate)
    gx = u[:, 5:].double()
    close(got.cpu(), P.rms_norm(o.double(), w.double(), 1e-5) * (P.sigmoid(gx) if gate == "sigmoid" else P.silu(gx)), dtype, f"row norm, {gate}")
