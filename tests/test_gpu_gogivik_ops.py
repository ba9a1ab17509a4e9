"""Kernels of the Gogivik family, each against the plain restatement: squared-ReLU products, the normed and convolved input of a sublayer,
attention in chunks with rotated values, latent attention with a sink, the state-space recurrence and its gated norm."""

import numpy as np
import pytest
import torch

import gogivik_oracle as oracle
from gpu_common import check_status, require_gpu_lib
from test_gpu_bufolorn_ops import Latent, cuts, i32, np64, tol
from test_gpu_tepetar_ops import BF16, FP32, Pages, close, padded, rnd

pytestmark = pytest.mark.gpu
BOTH = pytest.mark.parametrize("dtype", [BF16, FP32])


@pytest.fixture(scope="module", autouse=True)
def _lib():
    require_gpu_lib()
    from mfq_b200.ops.lib import dense_lib
    dense_lib()


def wide(t, n):
    """Channels of a tensor padded with zeros to a stored width."""
    return torch.nn.functional.pad(t, (0, n - t.shape[-1]))


# -- products -----------------------------------------------------------------------------------------------------------
@BOTH
@pytest.mark.parametrize("m,n,k", [(1, 16, 8), (3, 48, 72), (16, 1040, 1000), (17, 128, 64), (130, 272, 320), (700, 400, 200)])
def test_squared_relu(m, n, k, dtype):
    from mfq_b200.ops import dense
    x, w, b = rnd(m, k, dtype=dtype), rnd(n, k, dtype=dtype, scale=k ** -0.5), rnd(n, dtype=FP32)
    want = np.maximum(np64(x) @ np64(w).T + np64(b), 0) ** 2
    close(dense.DenseLinear(w, b, act="relu2")(x), want, tol(dtype))
    check_status()


# -- the input of a sublayer --------------------------------------------------------------------------------------------
@BOTH
@pytest.mark.parametrize("width,taps", [(104, 1), (104, 2), (24, 3), (1000, 4), (4096, 4), (104, 5), (3000, 8)])
def test_norm_and_convolution(width, taps, dtype):
    from mfq_b200.ops import dense
    w, lens, slots, eps = dense.up(width), [1, 1, 2, 3, 17, 64, 7, 8, 9], [5, 9, 0, 3, 1, 6, 2, 8, 10], 1e-3
    t, starts = sum(lens), cuts(lens)
    x, f, taps_w = wide(rnd(t, width, dtype=FP32) * 2, w), wide(rnd(width, dtype=FP32), w), wide(rnd(taps, width, dtype=FP32), w)
    state = wide(rnd(12, taps - 1, width, dtype=FP32), w)
    before, h = state.clone(), oracle.rms(np64(x)[:, :width], eps) * np64(f)[:width]
    kernel = np64(taps_w).T[:width]
    got = dense.norm_conv_out(x, f, taps_w, state, i32(*slots), width, eps, dtype, starts=i32(*starts), max_q=64, singles=2)
    for b, s in enumerate(slots):
        rows = h[starts[b] : starts[b + 1]]
        y, hist = oracle.causal_conv(rows, np64(before[s])[:, :width], kernel)
        close(got[starts[b] : starts[b + 1], :width], rows + y, 1e-2 if dtype == BF16 else 2e-5, f"sequence {b}")
        if taps > 1:
            close(state[s, :, :width], hist, 2e-5, f"kept rows of sequence {b}")
    assert not got[:, width:].any() and torch.equal(state[[4, 7, 11]], before[[4, 7, 11]])
    before = state.clone()
    got = dense.norm_conv_out(x[:3], f, taps_w, state, i32(4, -1, 7), width, eps, dtype)  # one row per sequence; a skipped one keeps nothing
    for row, s in ((0, 4), (2, 7)):
        y, hist = oracle.causal_conv(h[row : row + 1], np64(before[s])[:, :width], kernel)
        close(got[row : row + 1, :width], h[row : row + 1] + y, 1e-2 if dtype == BF16 else 2e-5)
        if taps > 1:
            close(state[s, :, :width], hist, 2e-5)
    rest = [s for s in range(12) if s not in (4, 7)]
    assert torch.equal(state[rest], before[rest])


@pytest.mark.parametrize("size", [1, 2, 3, 7, 8, 9, 33])
def test_norm_and_convolution_over_portions(size):
    """Any cut of a sequence gives the same rows, and leaves the same kept rows."""
    from mfq_b200.ops import dense
    x, f, k = rnd(70, 112, dtype=FP32), rnd(112, dtype=FP32), rnd(4, 112, dtype=FP32)
    outs = []
    for step in (70, size):
        state, parts = torch.zeros(1, 3, 112, device="cuda"), []
        for a in range(0, 70, step):
            n = min(step, 70 - a)
            parts.append(dense.norm_conv_out(x[a : a + n], f, k, state, i32(0), 112, 1e-5, FP32, starts=i32(0, n), max_q=n))
        outs.append((torch.cat(parts), state))
    close(outs[1][0], np64(outs[0][0]), 1e-6)
    close(outs[1][1], np64(outs[0][1]), 1e-6)


# -- attention in chunks ------------------------------------------------------------------------------------------------
@BOTH
@pytest.mark.parametrize("pairs", [False, True])
@pytest.mark.parametrize("e", [16, 28, 48, 200])
def test_normed_and_rotated_values(e, pairs, dtype):
    from mfq_b200.engine.kv_cache import PlainPagedKVCache
    from mfq_b200.ops import window_attn
    from mfq_b200.ops.dense import up
    h, g, d, rot, t, factor = 6, 2, 24, 16, 30, 2.5
    dk, dv = 32, up(e)
    cache = PlainPagedKVCache([(g, dk, dv)], dtype, num_pages=4, max_seqs=1, max_pages_per_seq=4, device="cuda")
    q, k, v = (torch.randn(t, n, x).to(dtype) for n, x in ((h, d), (g, d), (g, e)))
    rows = torch.cat([padded(q, dk).reshape(t, -1), padded(k, dk).reshape(t, -1), padded(v, dv).reshape(t, -1)], 1)
    pos = torch.randint(0, 500, (t,))
    rope = window_attn.rope_table(300.0, rot, 500, "cuda", window_attn.LinearScaling(factor))
    turn = window_attn.ValueTurn(window_attn.rope_table(300.0, e, 500, "cuda"), e)
    qw, kw = torch.randn(d), torch.randn(d)
    slots = torch.arange(16, 16 + t).int()
    slots[7] = -1
    got = window_attn.qkv_finish(rows, cache.layer(0), pos.int().cuda(), slots.cuda(), heads=h, kv_heads=g, dim=d, q_norm=wide(qw, dk).cuda(),
                                 k_norm=wide(kw, dk).cuda(), rope=rope, rot=rot, eps=1e-3, turn=turn, pairs=pairs)
    rotate, eps = oracle.rotate_pairs if pairs else oracle.rotate_halves, 1e-2 if dtype == BF16 else 1e-5
    f, vf, ok = oracle.frequencies(300.0, rot, factor), oracle.frequencies(300.0, e), (slots >= 0).numpy()
    close(got[..., :d], rotate(oracle.rms(np64(q), 1e-3) * np64(qw), pos.numpy(), f), eps, "q")
    kept = lambda pool: pool[1:].transpose(1, 2).reshape(-1, g, pool.shape[-1])[:t][ok]
    close(kept(cache.layer(0).k)[..., :d], rotate(oracle.rms(np64(k), 1e-3) * np64(kw), pos.numpy(), f)[ok], eps, "k")
    want = rotate(oracle.rms(np64(v), 1e-3), pos.numpy(), vf)
    close(kept(cache.layer(0).v)[..., :e], want[ok], eps, "v")
    assert not kept(cache.layer(0).v)[..., e:].any()
    o = padded(torch.from_numpy(want).to(dtype), dv)
    back = window_attn.turn_back(o, turn, pos.int().cuda(), pairs=pairs)
    close(back[..., :e], oracle.rms(np64(v), 1e-3), 2 * eps, "turned back")
    assert not back[..., e:].any()


class Chunked:
    def __init__(self, lens, h, g, d, e, size, dtype=BF16, turned=True):
        from mfq_b200.ops import window_attn
        self.h, self.g, self.d, self.e, self.size = h, g, d, e, size
        self.pages = Pages(lens, g, d, e, dtype)
        self.turn = window_attn.ValueTurn(window_attn.rope_table(900.0, e, max(lens), "cuda"), e) if turned else None
        self.how = dict(scale=1.5 * d ** -0.5, cap=0.0, window=1 << 30, chunk=size)

    def want(self, b, q, first):
        k, v, q = np64(self.pages.k[b]), np64(self.pages.v[b]), np64(q)
        pos = first + np.arange(len(q))
        see = oracle.in_chunk(pos, np.arange(len(k)), self.size)
        per = self.h // self.g
        o = np.stack([oracle.attend((q[:, n] @ k[:, n // per].T) * self.how["scale"], see, v[:, n // per]) for n in range(self.h)], 1)
        return oracle.rotate_halves(o, -pos, oracle.frequencies(900.0, self.e)) if self.turn else o


SHAPES = [(6, 2, 24, 28), (4, 4, 48, 16), (20, 1, 64, 64), (3, 1, 128, 128), (8, 2, 256, 256), (10, 5, 96, 200)]
SIZES = [1, 7, 16, 50, 128, 1 << 30]


@pytest.mark.parametrize("h,g,d,e", SHAPES)
@pytest.mark.parametrize("size", SIZES)
def test_decode_in_chunks(h, g, d, e, size):
    from mfq_b200.ops import window_attn
    from mfq_b200.ops.dense import up
    lens = [1, 7, 8, 16, 17, 49, 50, 51, 128, 129, 431]
    q = rnd(len(lens), h, d)
    for turned in (True, False):
        case = Chunked(lens, h, g, d, e, size, turned=turned)
        for splits in (1, 3):
            got = window_attn.decode(padded(q, up(d)), case.pages.kv, case.pages.cache.block_table, i32(*lens), splits=splits, turn=case.turn, **case.how)
            for b, n in enumerate(lens):
                close(got[b : b + 1, :, :e], case.want(b, q[b : b + 1], n - 1), 2e-2, f"length {n}")
            assert not got[..., e:].any()


@pytest.mark.parametrize("h,g,d,e", SHAPES)
@pytest.mark.parametrize("size", SIZES)
def test_prefill_and_plain_in_chunks(h, g, d, e, size):
    from mfq_b200.ops import window_attn
    from mfq_b200.ops.dense import up
    lens, counts = [70, 2, 300, 129, 400, 260], [70, 2, 40, 129, 3, 260]
    for dtype in (BF16, FP32):
        case = Chunked(lens, h, g, d, e, size, dtype)
        starts = cuts(counts)
        q = rnd(sum(counts), h, d, dtype=dtype)
        seq = torch.repeat_interleave(torch.arange(6, dtype=torch.int32), torch.tensor(counts)).cuda()
        pos = torch.cat([torch.arange(n - m, n, dtype=torch.int32) for n, m in zip(lens, counts)]).cuda()
        outs = [(window_attn.plain(padded(q, up(d)), case.pages.kv, case.pages.cache.block_table, seq, pos, **case.how), 1e-4 if dtype == FP32 else 2e-2)]
        if dtype == BF16:
            outs.append((window_attn.prefill(padded(q, up(d)), case.pages.kv, case.pages.cache.block_table, i32(*starts), i32(*lens), max(counts), **case.how), 3e-2))
        for got, t in outs:
            got = window_attn.turn_back(got, case.turn, pos)
            for b in range(6):
                close(got[starts[b] : starts[b + 1], :, :e], case.want(b, q[starts[b] : starts[b + 1]], lens[b] - counts[b]), t, f"sequence {b}")
    check_status()


@pytest.mark.parametrize("size", [5, 16, 33, 64])
def test_edges_of_the_chunks(size):
    """One key stands out and its value differs: every position shows whether it is seen."""
    from mfq_b200.ops import window_attn
    for spot in (0, size - 1, size, 2 * size + 3):
        case = Chunked([3 * size + 9], 2, 1, 16, 16, size, turned=False)
        n = case.pages.lens[0]
        case.pages.k[0].zero_()
        case.pages.k[0][spot] = 4.0
        case.pages.v[0].fill_(-1.0)
        case.pages.v[0][spot] = 1.0
        case.pages.store()
        q = torch.ones(n, 2, 16, dtype=BF16, device="cuda")
        seen = [1.0 if p >= spot and p // size == spot // size else -1.0 for p in range(n)]
        got = window_attn.prefill(q, case.pages.kv, case.pages.cache.block_table, i32(0, n), i32(n), n, **case.how)
        assert np.abs(got[:, 0, 0].float().cpu().numpy() - seen).max() < 0.05
        for p in range(n):
            one = window_attn.decode(q[:1], case.pages.kv, case.pages.cache.block_table, i32(p + 1), splits=1 + p % 3, **case.how)
            assert abs(float(one[0, 1, 3]) - seen[p]) < 0.05, p


# -- latent attention with a sink -----------------------------------------------------------------------------------------
def latent_want(case, b, qc, qr, first, window, scale, sink):
    c, r, qc, qr = np64(case.c[b]), np64(case.r[b]), np64(qc), np64(qr)
    see = oracle.in_window(first + np.arange(len(qc)), np.arange(case.lens[b]), window)
    return np.stack([oracle.attend((qc[:, n] @ c.T + qr[:, n] @ r.T) * scale, see, c, np64(sink)[n]) for n in range(qc.shape[1])], 1)


@pytest.mark.parametrize("heads,rank,rot", [(3, 40, 12), (16, 64, 16), (18, 128, 64), (40, 512, 64), (4, 24, 2)])
@pytest.mark.parametrize("window", [1, 17, 10 ** 9])
def test_sinks_in_latent_space(heads, rank, rot, window):
    from mfq_b200.ops import latent_attn
    lens, scale = [1, 16, 17, 70, 129, 333], 0.3 * rank ** -0.5
    sink = torch.linspace(-3, 6, heads).cuda()
    for dtype in (BF16, FP32):
        case = Latent(lens, rank, rot, dtype)
        qc, qr = rnd(6, heads, rank, dtype=dtype), rnd(6, heads, rot, dtype=dtype)
        how = dict(rank=case.cp, window=window, scale=scale, sink=sink)
        outs = [(latent_attn.plain(case.query(qc, qr), case.pool, case.cache.block_table, i32(*range(6)), i32(*(n - 1 for n in lens)), **how), 1e-2 if dtype == BF16 else 3e-5)]
        if dtype == BF16:
            outs += [(latent_attn.decode(case.query(qc, qr), case.pool, case.cache.block_table, i32(*lens), splits=s, **how), 2e-2) for s in (1, 3)]
        for got, t in outs:
            for b, n in enumerate(lens):
                close(got[b : b + 1, :, :rank], latent_want(case, b, qc[b : b + 1], qr[b : b + 1], n - 1, window, scale, sink), t, f"length {n}")


@pytest.mark.parametrize("heads,dim,rot,vdim,rank", [(3, 20, 12, 28, 40), (2, 128, 64, 128, 256), (5, 16, 2, 16, 24)])
@pytest.mark.parametrize("window", [1, 40, 10 ** 9])
def test_sinks_over_expanded_rows(heads, dim, rot, vdim, rank, window):
    from mfq_b200.ops import latent_attn
    from mfq_b200.ops.dense import up
    lens, counts = [150, 300, 70, 33], [150, 60, 2, 17]
    dk, dv, starts, scale = up(dim), up(vdim), cuts(counts), 1.2 * dim ** -0.5
    case = Latent(lens, rank, rot)  # for its block table
    k, v = [rnd(n, heads, dim) for n in lens], [rnd(n, heads, vdim) for n in lens]
    seq, shift = latent_attn.visible_pages([(n - m, m) for n, m in zip(lens, counts)], window)
    kv = torch.zeros(len(seq) * 16, heads, dk + dv, dtype=BF16, device="cuda")
    for b, n in enumerate(lens):
        first = max(0, n - counts[b] - window + 1) // 16 * 16
        at = torch.arange(first, n, device="cuda") + shift[b] * 16
        kv[at, :, :dim], kv[at, :, dk : dk + vdim] = k[b][first:], v[b][first:]
    q, sink = rnd(sum(counts), heads, dim), torch.linspace(-2, 5, heads).cuda()
    out = torch.zeros(sum(counts), heads, dv, dtype=BF16, device="cuda")
    for h0 in range(0, heads, 2):
        n = min(2, heads - h0)
        part = kv[:, h0 : h0 + n].reshape(kv.shape[0], -1).contiguous()
        latent_attn.prefill_rows(padded(q, dk), part, i32(*shift), i32(*starts), i32(*lens), max(counts), head0=h0, heads=n, dk=dk, dv=dv, window=window,
                                 scale=scale, sink=sink, out=out)
    for b, (n, m) in enumerate(zip(lens, counts)):
        see = oracle.in_window(n - m + np.arange(m), np.arange(n), window)
        a = np64(q[starts[b] : starts[b + 1]])
        want = np.stack([oracle.attend((a[:, h] @ np64(k[b])[:, h].T) * scale, see, np64(v[b])[:, h], np64(sink)[h]) for h in range(heads)], 1)
        close(out[starts[b] : starts[b + 1], :, :vdim], want, 3e-2, f"sequence {b}")
    assert case.cache.block_table.shape[0] == 4
    check_status()


@BOTH
@pytest.mark.parametrize("q_rank,rank,rot", [(36, 40, 12), (300, 512, 64), (16, 24, 2)])
def test_stage_behind_the_low_projections(q_rank, rank, rot, dtype):
    from mfq_b200.ops import latent_attn, window_attn
    from mfq_b200.ops.dense import up
    t, a, c, r = 21, up(q_rank), up(rank), up(rot)
    rope = window_attn.rope_table(1e4, rot, 500, "cuda")
    low, lat, kr = rnd(t, q_rank, dtype=dtype), rnd(t, rank, dtype=dtype), rnd(t, rot, dtype=dtype)
    proj, pos = torch.cat([wide(low, a), wide(lat, c), wide(kr, r)], 1).contiguous(), torch.randint(0, 500, (t,))
    qw, w = rnd(q_rank, dtype=FP32), rnd(rank, dtype=FP32)
    slots = torch.randperm(48)[:t].int() + 16
    slots[4] = -1
    pages = torch.zeros(5, 1, 16, c + r, dtype=dtype, device="cuda")
    got = latent_attn.down(proj, pages, pos.int().cuda(), slots.cuda(), q_rank=a, real_q_rank=q_rank, rank=c, rot=r, real_rank=rank, real_rot=rot,
                           q_norm=wide(qw, a), norm_w=wide(w, c), rope=rope, eps=1e-3)
    k, ok = 1e-2 if dtype == BF16 else 1e-5, (slots >= 0)
    close(got[:, :q_rank], oracle.rms(np64(low), 1e-3) * np64(qw), k, "query latent")
    assert not got[:, q_rank:].any()
    rows = pages.view(-1, c + r)[slots[ok].long().cuda()]
    close(rows[:, :rank], (oracle.rms(np64(lat), 1e-3) * np64(w))[ok.numpy()], k, "latent")
    want = oracle.rotate_pairs(np64(kr)[:, None], pos.numpy(), oracle.frequencies(1e4, rot))
    close(rows[:, c : c + rot], want[ok.numpy(), 0], k, "rotated key part")
    assert int((pages.view(-1, c + r) != 0).any(-1).sum()) == int(ok.sum())


# -- the recurrence -------------------------------------------------------------------------------------------------------
class Space:
    """Sequences of several lengths on scattered slots, behind the convolution."""

    def __init__(self, lens, h, g, n, e, dtype, a_log=0.0, dt_bias=-1.0, parts=1, slots=None):
        from mfq_b200.ops import ssd
        from mfq_b200.ops.dense import up
        self.lens, self.h, self.g, self.n, self.e = lens, h, g, n, e
        self.geo = ssd.Geometry(h, g, up(n), up(e), e, 4, parts, 1e-4)
        geo, t = self.geo, sum(lens)
        self.xs, self.bs, self.cs = rnd(t, h, e, dtype=dtype), rnd(t, g, n, dtype=dtype, scale=n ** -0.5), rnd(t, g, n, dtype=dtype)
        self.zs, self.dts = rnd(t, h, e, dtype=dtype), rnd(t, h, dtype=dtype)
        self.x = torch.cat([wide(self.xs, geo.width).reshape(t, -1), wide(self.bs, geo.state).reshape(t, -1), wide(self.cs, geo.state).reshape(t, -1)], 1).contiguous()
        self.proj = torch.cat([rnd(t, geo.channels, dtype=dtype), wide(self.zs, geo.width).reshape(t, -1), wide(self.dts, up(h))], 1).contiguous()
        self.a_log, self.dt_bias, self.skip = (torch.randn(h) * 0.3 + a_log).cuda(), (torch.randn(h) + dt_bias).cuda(), torch.randn(h).cuda()
        self.norm = wide(rnd(h, e, dtype=FP32), geo.width).reshape(-1).contiguous()
        self.w = ssd.Weights(None, None, self.dt_bias, self.a_log.exp(), self.skip, self.norm)
        self.slots = slots if slots is not None else list(range(len(lens)))[::-1]
        self.state0 = torch.zeros(len(lens) + 2, h, geo.state, geo.width)
        self.state0[:, :, :n, :e] = torch.randn(len(lens) + 2, h, n, e)
        self.state, self.starts = self.state0.cuda(), i32(*cuts(lens))

    def want(self):
        at, per, ys, states = cuts(self.lens), self.h // self.g, [], []
        for b, slot in enumerate(self.slots):
            r, s = slice(at[b], at[b + 1]), self.state0[slot, :, : self.n, : self.e].double().numpy().copy()
            dt = oracle.softplus(np64(self.dts[r]) + np64(self.dt_bias))
            ys.append(oracle.state_space(np64(self.xs[r]), np.repeat(np64(self.bs[r]), per, 1), np.repeat(np64(self.cs[r]), per, 1), dt, np64(self.a_log),
                                         np64(self.skip), s))
            states.append(s)
        return np.concatenate(ys), states

    def check(self, y, tol, state_tol):
        want, states = self.want()
        y = y.view(y.shape[0], self.h, -1)
        close(y[..., : self.e], want, tol, "y")
        assert not y[..., self.e :].any()
        for slot, s in zip(self.slots, states):
            close(self.state[slot, :, : self.n, : self.e], s, state_tol, f"state of slot {slot}")
        for other in set(range(len(self.state0))) - set(self.slots):
            assert torch.equal(self.state[other].cpu(), self.state0[other])


SPACES = [(4, 2, 24, 20), (6, 1, 16, 64), (3, 3, 128, 48), (8, 2, 64, 80), (2, 1, 256, 128), (5, 5, 20, 200)]


@BOTH
@pytest.mark.parametrize("h,g,n,e", SPACES)
def test_recurrence_token_by_token(h, g, n, e, dtype):
    from mfq_b200.ops import ssd
    case = Space([1] * 5, h, g, n, e, dtype, slots=[3, 0, 6, 2, 1])
    case.check(ssd.recurrent(case.x, case.proj, case.w, case.state, i32(*case.slots), case.geo), tol(dtype), 1e-5)
    case = Space([1, 2, 17, 40], h, g, n, e, dtype)
    case.check(ssd.recurrent(case.x, case.proj, case.w, case.state, i32(*case.slots), case.geo, starts=case.starts), tol(dtype), 1e-5)
    case = Space([1] * 3, h, g, n, e, dtype)
    y = ssd.recurrent(case.x, case.proj, case.w, case.state, i32(0, -1, 4), case.geo)  # a skipped row
    case.slots, case.lens = [0, 4], [1, 1]
    for name in ("xs", "bs", "cs", "dts"):
        setattr(case, name, getattr(case, name)[[0, 2]])
    case.check(y[[0, 2]], tol(dtype), 1e-5)


@pytest.mark.parametrize("h,g,n,e", SPACES)
@pytest.mark.parametrize("chunk", [64, 128])
def test_recurrence_in_chunks(h, g, n, e, chunk):
    from mfq_b200.ops import ssd
    if not ssd.Geometry(h, g, n, e, e, 4, 1, 1e-4).chunk_fits(chunk):
        pytest.skip("no room for such a chunk")
    for heads in sorted({1, h // g, 2 if h // g % 2 == 0 else 1}):
        if not Space([1], h, g, n, e, BF16).geo.chunk_fits(chunk, heads):
            continue
        case = Space([16, 1, 63, 64, 65, 128, 129, 300, 7], h, g, n, e, BF16)
        y = ssd.chunked(case.x, case.proj, case.w, case.state, i32(*case.slots), case.geo, case.starts, 300, chunk=chunk, heads=heads)
        case.check(y, 1.5e-2, 2e-4)


@pytest.mark.parametrize("a_log,dt_bias", [(-9.0, -3.0), (3.0, 2.0), (5.0, 4.0)])
def test_recurrence_with_extreme_decays(a_log, dt_bias):
    """States that forget nothing, and states that forget everything at once (decays that underflow)."""
    from mfq_b200.ops import ssd
    for chunk in (64, 128):
        case = Space([200, 70], 4, 2, 32, 48, BF16, a_log, dt_bias)
        y = ssd.chunked(case.x, case.proj, case.w, case.state, i32(*case.slots), case.geo, case.starts, 200, chunk=chunk)
        case.check(y, 1.5e-2, 2e-4)
    case = Space([50], 4, 2, 32, 48, FP32, a_log, dt_bias)
    case.check(ssd.recurrent(case.x, case.proj, case.w, case.state, i32(0), case.geo, starts=case.starts), 3e-5, 1e-5)


def test_recurrence_in_a_mixed_batch():
    """Single tokens in front of portions, through the convolution, against each alone."""
    from mfq_b200.ops import ssd
    for dtype in (BF16, FP32):
        case = Space([1, 1, 90, 3, 130], 4, 2, 24, 20, dtype, parts=4, slots=[5, 0, 3, 1, 6])
        case.w.conv, case.w.conv_bias = rnd(4, case.geo.channels, dtype=FP32), rnd(case.geo.channels, dtype=FP32)
        conv0 = rnd(7, 3, case.geo.channels, dtype=FP32)
        conv, slots = conv0.clone(), i32(*case.slots)
        got = ssd.ragged(case.proj, case.w, case.state, conv, slots, case.geo, case.starts, 130, 2)
        state, at = case.state.clone(), cuts(case.lens)
        case.state.copy_(case.state0)
        again = conv0.clone()
        for b, n in enumerate(case.lens):
            one = ssd.ragged(case.proj[at[b] : at[b + 1]].contiguous(), case.w, case.state, again, slots[b : b + 1], case.geo, i32(0, n), n, 0)
            close(got[at[b] : at[b + 1]], np64(one), 3e-2 if dtype == BF16 else 1e-4, f"sequence {b}")
        close(state, np64(case.state), 1e-3)
        assert torch.equal(conv, again)
    check_status()


@BOTH
@pytest.mark.parametrize("h,e,parts", [(4, 20, 1), (4, 20, 2), (6, 12, 4), (6, 12, 9), (2, 72, 8), (64, 64, 8), (16, 128, 1), (3, 16, 48)])
def test_gated_norm_in_parts(h, e, parts, dtype):
    from mfq_b200.ops import ssd
    case = Space([5], h, 1, 16, e, dtype, parts=parts)
    y = wide(rnd(5, h, e, dtype=dtype), case.geo.width).reshape(5, -1).contiguous()
    got = ssd.gate_norm(y, case.proj, case.w, case.geo).view(5, h, -1)
    real = lambda t: np64(t).reshape(-1, h, case.geo.width)[..., :e].reshape(-1, h * e)
    want = oracle.rms_parts(real(y) * oracle.silu(np64(case.zs).reshape(5, -1)), parts, 1e-4) * real(case.norm)
    close(got[..., :e].reshape(5, -1), want, 1e-2 if dtype == BF16 else 1e-5)
    assert not got[..., e:].any()


@BOTH
@pytest.mark.parametrize("taps", [1, 2, 4, 8])
def test_short_convolution_with_a_bias(taps, dtype):
    from mfq_b200.ops import ssd
    c, lens, slots = 120, [1, 2, 17, 64], [3, 0, 1, 2]
    starts = cuts(lens)
    x, w, b, state = rnd(sum(lens), c + 24, dtype=dtype), rnd(taps, c, dtype=FP32), rnd(c, dtype=FP32), rnd(4, taps - 1, c, dtype=FP32)
    before = state.clone()
    got = ssd.conv(x, w, state, i32(*slots), c, starts=i32(*starts), max_q=64, bias=b)
    for i, s in enumerate(slots):
        y, _ = oracle.causal_conv(np64(x[starts[i] : starts[i + 1], :c]), np64(before[s]), np64(w).T)
        close(got[starts[i] : starts[i + 1]], oracle.silu(y + np64(b)), tol(dtype), f"sequence {i}")
