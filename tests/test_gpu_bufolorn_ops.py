"""Kernels of the Bufolorn family, each against the plain restatement: batched and expert products with their output stages, layer norm,
token shift, short convolution, attention with a distance bias and a sink, latent attention, time mixing, the delta rule, routing."""

import numpy as np
import pytest
import torch

import bufolorn_oracle as oracle
from gpu_common import check_status, require_gpu_lib
from test_gpu_tepetar_ops import BF16, FP32, Pages, close, padded, rnd

pytestmark = pytest.mark.gpu
BOTH = pytest.mark.parametrize("dtype", [BF16, FP32])


@pytest.fixture(scope="module", autouse=True)
def _lib():
    require_gpu_lib()
    from mfq_b200.ops.lib import dense_lib
    dense_lib()


def i32(*x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


def np64(t):
    return t.double().cpu().numpy()


def tol(dtype):
    return 2e-2 if dtype == BF16 else 3e-5


# -- products -----------------------------------------------------------------------------------------------------------
@BOTH
@pytest.mark.parametrize("m,n,k", [(1, 16, 8), (3, 48, 72), (16, 1040, 1000), (17, 128, 64), (130, 272, 320), (700, 400, 200)])
def test_output_stages(m, n, k, dtype):
    from mfq_b200.ops import dense
    x, w, b = rnd(m, k, dtype=dtype), rnd(n, k, dtype=dtype, scale=k ** -0.5), rnd(n, dtype=FP32)
    y = np64(x) @ np64(w).T
    close(dense.DenseLinear(w, b)(x, fp32=True), y + np64(b), 2e-5 if dtype == FP32 else 2e-4, "fp32 result")
    stream = rnd(m, n, dtype=FP32)
    want = np64(stream) - 0.7 * (y + np64(b))
    dense.DenseLinear(w, b)(x, add_to=stream, scale=-0.7)
    close(stream, want, 2e-5 if dtype == FP32 else 2e-4, "scaled addition")
    gate, up = rnd(n // 2, k, dtype=dtype, scale=k ** -0.5), rnd(n // 2, k, dtype=dtype, scale=k ** -0.5)
    for act, f in (("relu", lambda z: np.maximum(z, 0)), ("silu", oracle.silu)):
        got = dense.DenseLinear(dense.interleave_glu(gate, up), glu=act)(x)
        close(got, f(np64(x) @ np64(gate).T) * (np64(x) @ np64(up).T), tol(dtype), act)
    check_status()


@BOTH
@pytest.mark.parametrize("m", [1, 5, 12, 40, 200])
@pytest.mark.parametrize("g,n,k,x_step,out_step", [(1, 32, 48, 64, 48), (3, 48, 32, 56, 64), (5, 16, 8, 8, 16), (4, 144, 72, 72, 144), (2, 256, 136, 200, 272)])
def test_a_matrix_per_head(m, g, n, k, x_step, out_step, dtype):
    from mfq_b200.ops import dense
    x, w, b = rnd(m, (g - 1) * x_step + k + 8, dtype=dtype), rnd(g * n, k, dtype=dtype, scale=k ** -0.5), rnd(g * n, dtype=FP32)
    out = torch.full((m, g * out_step + 16), 7.0, dtype=dtype, device="cuda")
    dense.DenseLinear(w, b, groups=g)(x, x_step=x_step, out_step=out_step, out=out)
    for i in range(g):
        want = np64(x[:, i * x_step : i * x_step + k]) @ np64(w[i * n : (i + 1) * n]).T + np64(b[i * n : (i + 1) * n])
        close(out[:, i * out_step : i * out_step + n], want, tol(dtype), f"matrix {i}")
        gap = out[:, i * out_step + n : (i + 1) * out_step]
        assert (gap == 7.0).all()
    check_status()


@BOTH
@pytest.mark.parametrize("t,e,top,tile", [(1, 5, 2, 0), (7, 4, 4, 0), (50, 7, 3, 0), (50, 7, 3, 16), (90, 3, 1, 64), (300, 9, 2, 128), (60, 40, 8, 32)])
def test_experts(t, e, top, tile, dtype):
    from mfq_b200.ops import dense, dense_moe
    w, f = 104, 40
    if dtype == FP32:
        tile = 64
    h, x = rnd(t, 112, dtype=dtype), rnd(t, 112, dtype=FP32)
    h[:, w:] = 0
    gate, up, down = (rnd(e, *s, dtype=dtype, scale=s[1] ** -0.5) for s in ((f, 112), (f, 112), (112, f)))
    bank = dense_moe.ExpertBank(e, torch.cat([dense.interleave_glu(gate[i], up[i]) for i in range(e)]).contiguous(), down.reshape(-1, f).contiguous())
    router, correction = rnd(dense.up(e), 112, dtype=dtype, scale=0.15), rnd(e, dtype=FP32)
    route = dense_moe.Router(dense.DenseLinear(router), correction, e, top, 1.7)
    ids, weight = route(h)
    z = np64(h) @ np64(router[:e]).T
    want_ids, want_w = oracle.route(np64(h), np64(router[:e]), np64(correction), top, 1.7)
    choice = np.sort(oracle.sigmoid(z) + np64(correction), -1)
    clear = np.ones(t, bool) if top == e else choice[:, e - top] - choice[:, e - top - 1] > 1e-3
    got = np.argsort(ids.cpu().numpy(), -1)
    want = np.argsort(want_ids, -1)
    take = np.take_along_axis
    assert (take(ids.cpu().numpy(), got, -1) == take(want_ids, want, -1))[clear].all()
    assert np.abs(take(weight.double().cpu().numpy(), got, -1) - take(want_w, want, -1))[clear].max() < 1e-4
    stream = np64(x)
    for i, (row, ws) in enumerate(zip(ids.tolist(), np64(weight))):
        for j, wt in zip(row, ws):
            stream[i] += 0.6 * wt * oracle.gated_unit(np64(h[i]), np64(gate[j]), np64(up[j]), np64(down[j]), oracle.silu)
    dense_moe.add_experts(h, ids, weight, bank, x, 0.6, tile=tile)
    close(x, stream, tol(dtype), "stream")
    check_status()


# -- stages of a layer --------------------------------------------------------------------------------------------------
@BOTH
@pytest.mark.parametrize("width", [24, 104, 1000, 4096, 8200])
def test_layer_norm(width, dtype):
    from mfq_b200.ops import dense
    w = dense.up(width)
    pad = lambda t: torch.nn.functional.pad(t, (0, w - width))
    x, f, b = pad(rnd(7, width, dtype=FP32) * 0.3 + 5.0), pad(rnd(width, dtype=FP32)), pad(rnd(width, dtype=FP32))
    got = dense.layer_norm_out(x, f, b, width, 1e-3, dtype)
    close(got[:, :width], oracle.layer_norm(np64(x)[:, :width], np64(f)[:width], np64(b)[:width], 1e-3), 1e-2 if dtype == BF16 else 2e-5)
    assert not got[:, width:].any()


def cuts(lens):
    return [0, *np.cumsum(lens).tolist()]


@BOTH
def test_token_shift(dtype):
    from mfq_b200.ops import gla
    w, lens, slots = 112, [1, 1, 5, 2, 40], [3, 0, 5, 2, 1]
    h, mu, last = rnd(sum(lens), w, dtype=dtype), rnd(3, w, dtype=FP32), rnd(7, w, dtype=FP32)
    if dtype == BF16:
        last = last.bfloat16().float()
    before = last.clone()
    starts = cuts(lens)
    seq = torch.repeat_interleave(torch.arange(5, dtype=torch.int32), torch.tensor(lens)).cuda()
    got = gla.token_shift(h, mu, last, i32(*slots), i32(*starts), seq).view(-1, 3, w)
    for b, s in enumerate(slots):
        rows = np64(h[starts[b] : starts[b + 1]])
        prev = oracle.shifted(rows, np64(before[s]))
        for j in range(3):
            close(got[starts[b] : starts[b + 1], j], oracle.mixed(rows, prev, np64(mu[j])), tol(dtype))
        assert torch.equal(last[s], h[starts[b + 1] - 1].float())
    assert torch.equal(last[[4, 6]], before[[4, 6]])
    again = gla.token_shift(h[:3], mu, last, i32(3, -1, 0))  # one row per sequence; a skipped one reads zeros and keeps nothing
    assert torch.equal(last[3], h[0].float()) and torch.equal(last[0], h[2].float()) and torch.equal(last[1], h[-1].float())
    close(again.view(3, 3, w)[1, 0], np64(h[1]) * (1 - np64(mu[0])), tol(dtype))


@BOTH
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5, 8])
def test_short_convolution(taps, dtype):
    from mfq_b200.ops import delta
    c, lens, slots = 120, [1, 2, 3, 17, 64, 7], [5, 0, 3, 1, 6, 2]
    t, starts = sum(lens), cuts(lens)
    x, w, state = rnd(t, c + 24, dtype=dtype), rnd(taps, c, dtype=FP32), rnd(8, taps - 1, c, dtype=FP32)
    before = state.clone()
    got = delta.conv(x, w, state, i32(*slots), c, starts=i32(*starts), max_q=64)
    for b, s in enumerate(slots):
        y, hist = oracle.short_conv(np64(x[starts[b] : starts[b + 1], :c]), np64(before[s]), np64(w).T)
        close(got[starts[b] : starts[b + 1]], oracle.silu(y), tol(dtype), f"sequence {b}")
        if taps > 1:
            close(state[s], hist, 1e-6)
    assert torch.equal(state[[4, 7]], before[[4, 7]])
    before = state.clone()
    got = delta.conv(x, w, state, i32(4, -1, 7), c)
    for row, s in ((0, 4), (2, 7)):
        y, hist = oracle.short_conv(np64(x[row : row + 1, :c]), np64(before[s]), np64(w).T)
        close(got[row : row + 1], oracle.silu(y), tol(dtype))
        if taps > 1:
            close(state[s], hist, 1e-6)
    rest = [0, 1, 2, 3, 5, 6]
    assert torch.equal(state[rest], before[rest])


@BOTH
def test_query_temperature_and_norm_without_weight(dtype):
    from mfq_b200.engine.kv_cache import PlainPagedKVCache
    from mfq_b200.ops import window_attn
    h, g, d, e, t = 6, 2, 20, 24, 30
    cache = PlainPagedKVCache([(g, 32, 32)], dtype, num_pages=4, max_seqs=1, max_pages_per_seq=4, device="cuda")
    q, k, v = (torch.randn(t, n, x).to(dtype) for n, x in ((h, d), (g, d), (g, e)))
    rows = torch.cat([padded(q, 32).reshape(t, -1), padded(k, 32).reshape(t, -1), padded(v, 32).reshape(t, -1)], 1)
    pos = torch.arange(t) + 5
    ones = torch.nn.functional.pad(torch.ones(d), (0, 12)).cuda()
    got = window_attn.qkv_finish(rows, cache.layer(0), pos.int().cuda(), torch.arange(16, 16 + t).int().cuda(), heads=h, kv_heads=g, dim=d, q_norm=ones,
                                 k_norm=ones, rope=None, rot=0, eps=1e-3, temperature=(0.6, 7))
    want = oracle.rms(np64(q), 1e-3) * oracle.temperature(pos.numpy(), 0.6, 7)[:, None, None]  # steps at positions 6, 13, 20, 27
    close(got[..., :d], want, 1e-2 if dtype == BF16 else 1e-5, "q")
    kept = cache.layer(0).k[1:].transpose(1, 2).reshape(-1, g, 32)[:t]
    close(kept[..., :d], oracle.rms(np64(k), 1e-3), 1e-2 if dtype == BF16 else 1e-5, "k")


# -- attention with a distance bias and a sink ------------------------------------------------------------------------------
class Biased:
    def __init__(self, lens, h, g, d, e, rows, most, dtype=BF16, sink=True):
        from mfq_b200.ops.window_attn import DistanceBias, log_buckets
        self.h, self.g, self.d, self.e, self.most = h, g, d, e, most
        self.pages = Pages(lens, g, d, e, dtype)
        self.rel = torch.randn(rows, h) * 2.0
        self.bias = DistanceBias.from_table(self.rel[torch.tensor(log_buckets(rows, most))].T.cuda())
        self.sink = (torch.randn(h) + 1.0).cuda() if sink else None
        self.how = dict(scale=0.4, cap=6.0, bias=self.bias, sink=self.sink, window=1 << 30)

    def want(self, b, q, first):
        k, v, q = np64(self.pages.k[b]), np64(self.pages.v[b]), np64(q)
        pos = first + np.arange(len(q))
        dist = pos[:, None] - np.arange(self.pages.lens[b])[None]
        rows = np.array([oracle.bucket(n, len(self.rel), self.most) for n in range(self.pages.lens[b])])[np.maximum(dist, 0)]
        out = []
        for n in range(self.h):
            s = oracle.softcap(q[:, n] @ k[:, n // (self.h // self.g)].T * 0.4, 6.0) + np64(self.rel)[rows, n]
            out.append(oracle.attend(s, dist >= 0, v[:, n // (self.h // self.g)], None if self.sink is None else np64(self.sink)[n]))
        return np.stack(out, 1)


SHAPES = [(6, 2, 20, 28), (4, 4, 48, 16), (20, 1, 64, 64), (3, 1, 128, 128), (8, 2, 256, 256), (10, 5, 96, 200)]


@pytest.mark.parametrize("h,g,d,e", SHAPES)
@pytest.mark.parametrize("splits", [1, 3])
@pytest.mark.parametrize("rows,most,sink", [(12, 70, True), (32, 300, True), (6, 20, False)])
def test_decode_with_bias_and_sink(h, g, d, e, splits, rows, most, sink):
    from mfq_b200.ops import window_attn
    from mfq_b200.ops.dense import up
    case = Biased([1, 5, 16, 17, 33, 90, 200, 431], h, g, d, e, rows, most, sink=sink)
    q = rnd(8, h, d)
    got = window_attn.decode(padded(q, up(d)), case.pages.kv, case.pages.cache.block_table, i32(*case.pages.lens), splits=splits, **case.how)
    for b, n in enumerate(case.pages.lens):
        close(got[b : b + 1, :, :e], case.want(b, q[b : b + 1], n - 1), 2e-2, f"length {n}")


@pytest.mark.parametrize("h,g,d,e", SHAPES)
@pytest.mark.parametrize("rows,most,sink", [(12, 70, True), (32, 300, True), (6, 20, False)])
def test_prefill_and_plain_with_bias_and_sink(h, g, d, e, rows, most, sink):
    from mfq_b200.ops import window_attn
    from mfq_b200.ops.dense import up
    lens, counts = [70, 2, 300, 129, 400], [70, 2, 40, 129, 3]
    for dtype in (BF16, FP32):
        case = Biased(lens, h, g, d, e, rows, most, dtype, sink)
        starts = cuts(counts)
        q = rnd(sum(counts), h, d, dtype=dtype)
        seq = torch.repeat_interleave(torch.arange(5, dtype=torch.int32), torch.tensor(counts)).cuda()
        pos = torch.cat([torch.arange(n - m, n, dtype=torch.int32) for n, m in zip(lens, counts)]).cuda()
        outs = [(window_attn.plain(padded(q, up(d)), case.pages.kv, case.pages.cache.block_table, seq, pos, **case.how), 1e-4 if dtype == FP32 else 2e-2)]
        if dtype == BF16:
            outs.append((window_attn.prefill(padded(q, up(d)), case.pages.kv, case.pages.cache.block_table, i32(*starts), i32(*lens), max(counts), **case.how), 2e-2))
        for got, t in outs:
            for b in range(5):
                close(got[starts[b] : starts[b + 1], :, :e], case.want(b, q[starts[b] : starts[b + 1]], lens[b] - counts[b]), t, f"sequence {b}")
    check_status()


@pytest.mark.parametrize("rows,most", [(12, 70), (8, 64)])
def test_edges_of_the_distance_buckets(rows, most):
    """Zero scores, so that the bias alone decides; one value differs: every distance shows its bucket."""
    from mfq_b200.ops import window_attn
    case = Biased([150], 2, 1, 16, 16, rows, most)
    case.rel[:] = torch.tensor([[3.0 if b % 2 else -3.0, -0.4 * b] for b in range(rows)])
    case.bias = window_attn.DistanceBias.from_table(case.rel[torch.tensor(window_attn.log_buckets(rows, most))].T.cuda())
    case.how["bias"] = case.bias
    case.pages.k[0].zero_()
    case.pages.v[0].fill_(-1.0)
    case.pages.v[0][11] = 1.0
    case.pages.store()
    q = rnd(150, 2, 16)
    got = window_attn.prefill(q, case.pages.kv, case.pages.cache.block_table, i32(0, 150), i32(150), 150, **case.how)
    want = case.want(0, q, 0)
    assert np.abs(got.float().cpu().numpy() - want).max() < 1e-2
    for n in range(12, 150):
        one = window_attn.decode(q[n : n + 1], case.pages.kv, case.pages.cache.block_table, i32(n + 1), splits=1 + n % 3, **case.how)
        assert np.abs(one.float().cpu().numpy() - want[n]).max() < 1e-2


# -- latent attention ----------------------------------------------------------------------------------------------------
class Latent:
    """Pages of latent rows of several sequences in scattered pages, and the restatement's answer in latent space."""

    def __init__(self, lens, rank, rot, dtype=BF16):
        from mfq_b200.engine.kv_cache import PlainPagedKVCache
        from mfq_b200.ops.dense import up
        self.lens, self.rank, self.rot, self.cp, self.rp = lens, rank, rot, up(rank), up(rot)
        need = sum(-(-n // 16) for n in lens)
        self.cache = PlainPagedKVCache([(1, self.cp + self.rp, 0)], dtype, num_pages=need + 4, max_seqs=len(lens), max_pages_per_seq=max(-(-n // 16) for n in lens),
                                       device="cuda")
        free = self.cache.allocator.free
        np.random.default_rng(0).shuffle(free)
        self.pool = self.cache.layer(0).k
        self.c, self.r = [rnd(n, rank, dtype=dtype) for n in lens], [rnd(n, rot, dtype=dtype) for n in lens]
        self.store()

    def store(self):
        for b, n in enumerate(self.lens):
            self.cache.assign(b, b, n)
            flat = self.pool.view(-1, self.cp + self.rp)
            at = self.cache.slots(b, 0, n).long().cuda()
            flat[at, : self.rank], flat[at, self.cp : self.cp + self.rot] = self.c[b], self.r[b]

    def query(self, c, r):
        return torch.cat([padded(c, self.cp), padded(r, self.rp)], -1).contiguous()

    def want(self, b, qc, qr, first, window, scale):
        c, r, qc, qr = np64(self.c[b]), np64(self.r[b]), np64(qc), np64(qr)
        see = oracle.visible(first + np.arange(len(qc)), np.arange(self.lens[b]), window)
        return np.stack([oracle.attend((qc[:, n] @ c.T + qr[:, n] @ r.T) * scale, see, c) for n in range(qc.shape[1])], 1)


@pytest.mark.parametrize("heads,rank,rot", [(3, 40, 12), (16, 64, 16), (18, 128, 64), (40, 512, 64), (4, 24, 2), (5, 300, 50)])
@pytest.mark.parametrize("window", [1, 17, 64, 10 ** 9])
def test_attention_in_latent_space(heads, rank, rot, window):
    from mfq_b200.ops import latent_attn
    lens, scale = [1, 16, 17, 70, 129, 333], 0.6 * rank ** -0.5
    case = Latent(lens, rank, rot)
    qc, qr = rnd(6, heads, rank), rnd(6, heads, rot)
    for splits in (1, 3):
        got = latent_attn.decode(case.query(qc, qr), case.pool, case.cache.block_table, i32(*lens), rank=case.cp, window=window, scale=scale, splits=splits)
        for b, n in enumerate(lens):
            close(got[b : b + 1, :, :rank], case.want(b, qc[b : b + 1], qr[b : b + 1], n - 1, window, scale), 2e-2, f"length {n}")
    seq, pos = i32(3, 3, 5, 1, 5, 0), i32(68, 69, 200, 3, 332, 0)  # several queries of a sequence
    how = dict(rank=case.cp, window=window, scale=scale)
    many = latent_attn.decode(case.query(qc, qr), case.pool, case.cache.block_table, pos, tok_seq=seq, splits=2, **how)
    plain = latent_attn.plain(case.query(qc, qr), case.pool, case.cache.block_table, seq, pos, **how)
    for i, (b, p) in enumerate(zip(seq.tolist(), pos.tolist())):
        want = case.want(b, qc[i : i + 1], qr[i : i + 1], p, window, scale)
        close(many[i : i + 1, :, :rank], want, 2e-2)
        close(plain[i : i + 1, :, :rank], want, 1e-2)


def test_attention_in_latent_space_in_full_precision():
    from mfq_b200.ops import latent_attn
    for heads, rank, rot in ((3, 40, 12), (2, 512, 64)):
        case = Latent([70, 200], rank, rot, FP32)
        qc, qr = rnd(4, heads, rank, dtype=FP32), rnd(4, heads, rot, dtype=FP32)
        got = latent_attn.plain(case.query(qc, qr), case.pool, case.cache.block_table, i32(0, 1, 1, 0), i32(69, 199, 30, 0), rank=case.cp, window=33, scale=0.2)
        for i, (b, p) in enumerate(((0, 69), (1, 199), (1, 30), (0, 0))):
            close(got[i : i + 1, :, :rank], case.want(b, qc[i : i + 1], qr[i : i + 1], p, 33, 0.2), 3e-5)


@pytest.mark.parametrize("heads,dim,rot,vdim,rank", [(3, 20, 12, 28, 40), (2, 128, 64, 128, 512), (5, 16, 2, 16, 24), (4, 64, 32, 200, 128)])
@pytest.mark.parametrize("window", [1, 40, 10 ** 9])
def test_attention_over_expanded_rows(heads, dim, rot, vdim, rank, window):
    from mfq_b200.ops import latent_attn
    from mfq_b200.ops.dense import DenseLinear, up
    lens, counts = [150, 300, 70, 33], [150, 60, 2, 17]
    case = Latent(lens, rank, rot)
    d, r, e, c = up(dim), up(rot), up(vdim), up(rank)
    uk, uv = rnd(heads, dim, rank, scale=rank ** -0.5), rnd(heads, vdim, rank, scale=rank ** -0.5)
    expand = torch.zeros(heads, d + r + e, c + r, dtype=BF16, device="cuda")
    expand[:, :dim, :rank], expand[:, d + r : d + r + vdim, :rank] = uk, uv
    expand[:, d : d + r, c:] = torch.eye(r, device="cuda")
    starts, scale = cuts(counts), (dim + rot) ** -0.5
    qn, qr = rnd(sum(counts), heads, dim), rnd(sum(counts), heads, rot)
    q = torch.cat([padded(qn, d), padded(qr, r)], -1).contiguous()
    seq, shift = latent_attn.visible_pages([(n - m, m) for n, m in zip(lens, counts)], window)
    rows = latent_attn.visible_rows(case.pool, case.cache.block_table, i32(*seq), i32(*shift))
    for group in (heads, 2):
        out = torch.zeros(sum(counts), heads, e, dtype=BF16, device="cuda")
        for h0 in range(0, heads, group):
            n = min(group, heads - h0)
            kv = DenseLinear(expand[h0 : h0 + n].reshape(-1, c + r).contiguous())(rows)
            latent_attn.prefill_rows(q, kv, i32(*shift), i32(*starts), i32(*lens), max(counts), head0=h0, heads=n, dk=d + r, dv=e, window=window, scale=scale, out=out)
        for b, (n, m) in enumerate(zip(lens, counts)):
            k, v, kr = np64(case.c[b]) @ np64(uk).transpose(0, 2, 1), np64(case.c[b]) @ np64(uv).transpose(0, 2, 1), np64(case.r[b])
            see = oracle.visible(n - m + np.arange(m), np.arange(n), window)
            a, z = np64(qn[starts[b] : starts[b + 1]]), np64(qr[starts[b] : starts[b + 1]])
            want = np.stack([oracle.attend((a[:, h] @ k[h].T + z[:, h] @ kr.T) * scale, see, v[h]) for h in range(heads)], 1)
            close(out[starts[b] : starts[b + 1], :, :vdim], want, 3e-2, f"sequence {b}")
    check_status()


@BOTH
@pytest.mark.parametrize("owner", [True, False])
def test_stage_behind_the_projections(owner, dtype):
    from mfq_b200.models.bufolorn import _yarn
    from mfq_b200.ops import latent_attn, window_attn
    h, dim, rot, rank, t, n1 = 3, 20, 12, 40, 21, 8
    d, r, c = 32, 16, 48
    sc = {"factor": 4.0, "original": 60, "fast": 4.0, "slow": 0.7}
    rope = window_attn.rope_table(1e4, rot, 500, "cuda", _yarn(sc))
    qn, qr, lat, kr = rnd(t, h, dim, dtype=dtype), rnd(t, h, rot, dtype=dtype), rnd(t, rank, dtype=dtype), rnd(t, rot, dtype=dtype)
    parts = [torch.cat([padded(qn, d), padded(qr, r)], -1).reshape(t, -1)] + ([padded(lat, c), padded(kr, r)] if owner else [])
    proj, pos, w = torch.cat(parts, 1).contiguous(), torch.randint(0, 500, (t,)), rnd(rank, dtype=FP32)
    slots = torch.randperm(48)[:t].int() + 16
    slots[4] = -1
    pages = torch.zeros(5, 1, 16, c + r, dtype=dtype, device="cuda")
    ql, q = latent_attn.finish(proj, pages if owner else None, pos.int().cuda(), slots.cuda(), heads=h, d=d, rank=c, rot=r, real_rank=rank, real_rot=rot,
                               norm_w=torch.nn.functional.pad(w, (0, c - rank)) if owner else None, rope=rope, eps=1e-3, latent_rows=n1)
    turn = lambda x: oracle.rotate_pairs(x, pos.numpy(), *oracle.frequencies(1e4, rot, sc))
    k = 1e-2 if dtype == BF16 else 1e-5
    want = turn(np64(qr))
    close(ql[:, :, c : c + rot], want[:n1], k, "rotated part in latent space")
    close(q[n1:, :, d : d + rot], want[n1:], k, "rotated part")
    assert torch.equal(q[n1:, :, :dim], qn[n1:]) and not q[n1:, :, dim:d].any()
    if owner:
        ok = slots >= 0
        rows = pages.view(-1, c + r)[slots[ok].long().cuda()]
        close(rows[:, :rank], (oracle.rms(np64(lat), 1e-3) * np64(w))[ok.numpy()], k, "latent")
        close(rows[:, c : c + rot], turn(np64(kr)[:, None])[ok.numpy(), 0], k, "rotated key part")
        assert int((pages.view(-1, c + r) != 0).any(-1).sum()) == int(ok.sum())


# -- recurrences -----------------------------------------------------------------------------------------------------------
class Recurrence:
    """Shared by the two kinds: sequences of several lengths on scattered slots."""

    def finish(self, lens, heads, geo, slots, gen):
        self.lens, self.geo, self.heads = lens, geo, heads
        self.slots = slots if slots is not None else list(range(len(lens)))[::-1]
        self.state0 = torch.zeros(len(lens) + 2, heads, geo.dk, geo.dv)
        self.state0[:, :, : geo.dim, : geo.vdim] = torch.randn(len(lens) + 2, heads, geo.dim, geo.vdim, generator=gen)
        self.state, self.starts = self.state0.cuda(), i32(*cuts(lens))

    def check(self, y, tol, state_tol):
        geo, want, states = self.geo, *self.want()
        y = y.view(y.shape[0], self.heads, geo.dv)
        close(y[..., : geo.vdim], want, tol, "y")
        assert not y[..., geo.vdim :].any()
        for slot, s in zip(self.slots, states):
            close(self.state[slot, :, : geo.dim, : geo.vdim], s, state_tol, f"state of slot {slot}")
        for other in set(range(len(self.state0))) - set(self.slots):
            assert torch.equal(self.state[other].cpu(), self.state0[other])


class TimeMix(Recurrence):
    def __init__(self, lens, heads, d, rank, dtype, w0=-2.0, strength=1.0, slots=None):
        from mfq_b200.ops import gla
        from mfq_b200.ops.dense import up
        g = torch.Generator().manual_seed(0)
        t, dk = sum(lens), up(d)
        geo = gla.Geometry(heads, dk, dk, d, d, up(rank), 1.0, 1e-4, decay="exp", scaled=False)
        draw = lambda *s: torch.randn(s, generator=g)
        self.r, self.k, self.v, self.z = (draw(t, heads, d).to(dtype) for _ in range(4))
        self.k = (0.7 * self.r.float() + 0.7 * self.k.float()).to(dtype)
        self.a, self.w2 = draw(t, rank).tanh().to(dtype), (draw(heads, d, rank) * strength * rank ** -0.5).to(dtype)
        self.w0, self.u, self.norm = w0 + draw(heads, d), 0.2 + draw(heads, d).abs(), 1 + 0.3 * draw(heads, d)
        pad = lambda x, n: torch.nn.functional.pad(x, (0, n - x.shape[-1]))
        flat = lambda x: pad(x, dk).reshape(t, -1)
        self.proj = torch.cat([flat(self.r), flat(self.k), flat(self.v), flat(self.z), pad(self.a, geo.rank)], 1).cuda().contiguous()
        w2 = torch.zeros(heads, dk, geo.rank, dtype=dtype)
        w2[:, :d, :rank] = self.w2
        self.args = (w2.reshape(-1, geo.rank).cuda(), pad(self.w0, dk).reshape(-1).cuda(), pad(self.norm, dk).contiguous().cuda())
        self.bonus = pad(self.u, dk).reshape(-1).cuda()
        self.finish(lens, heads, geo, slots, g)

    def want(self):
        out, states, a = [], [], 0
        for n, slot in zip(self.lens, self.slots):
            s = slice(a, a + n)
            w = np.exp(-np.exp(np.einsum("tr,hdr->thd", np64(self.a[s]), np64(self.w2)) + np64(self.w0)))
            state = np64(self.state0[slot, :, : self.geo.dim, : self.geo.dim]).copy()
            o = oracle.rwkv_rule(np64(self.r[s]), np64(self.k[s]), np64(self.v[s]), w, np64(self.u), state)
            out.append(oracle.rms(o, self.geo.eps) * np64(self.norm) * oracle.silu(np64(self.z[s])))
            states.append(state)
            a += n
        return np.concatenate(out), states


MIX_SIZES = [(3, 24, 8), (2, 64, 16), (6, 48, 20), (1, 128, 64), (2, 112, 24), (1, 256, 32), (4, 16, 5)]


@BOTH
@pytest.mark.parametrize("heads,d,rank", MIX_SIZES)
def test_time_mixing_token_by_token(heads, d, rank, dtype):
    from mfq_b200.ops import gla
    case = TimeMix([5, 1, 9, 2], heads, d, rank, dtype, slots=[4, 0, 2, 1])
    y = gla.recurrent(case.proj, *case.args, case.state, i32(*case.slots), case.geo, starts=case.starts, bonus=case.bonus)
    case.check(y, 2e-4 if dtype == FP32 else 2e-2, 1e-5)


@pytest.mark.parametrize("heads,d,rank", MIX_SIZES)
@pytest.mark.parametrize("lens", [[64], [200, 2, 63, 65, 128, 1, 17], [15, 16, 333]])
def test_time_mixing_in_chunks(heads, d, rank, lens):
    from mfq_b200.ops import gla
    case = TimeMix(lens, heads, d, rank, BF16)
    y = gla.chunked(case.proj, *case.args, case.state, i32(*case.slots), case.geo, case.starts, max(lens), bonus=case.bonus)
    case.check(y, 2e-2, 2e-4)


@pytest.mark.parametrize("w0,strength", [(-9.0, 0.5), (-2.0, 1.0), (0.0, 3.0), (2.0, 1.0), (3.0, 6.0), (-3.0, 8.0)])
def test_time_mixing_decays_of_every_strength(w0, strength):
    from mfq_b200.ops import gla
    case = TimeMix([150, 70], 2, 32, 16, BF16, w0, strength)
    case.check(gla.chunked(case.proj, *case.args, case.state, i32(*case.slots), case.geo, case.starts, 150, bonus=case.bonus), 2e-2, 5e-4)
    case = TimeMix([150, 70], 2, 32, 16, FP32, w0, strength)
    case.check(gla.recurrent(case.proj, *case.args, case.state, i32(*case.slots), case.geo, starts=case.starts, bonus=case.bonus), 5e-4, 3e-5)


class Delta(Recurrence):
    def __init__(self, lens, heads, keys, d, e, dtype, ra=12, rg=20, bias=-2.0, strength=1.0, rate=0.0, slots=None):
        from mfq_b200.ops import delta
        from mfq_b200.ops.dense import DenseLinear, up
        g = torch.Generator().manual_seed(1)
        t, dk, dv = sum(lens), up(d), up(e)
        geo = delta.Geometry(heads, keys, dk, dv, d, e, up(ra), up(rg), 4, 1e-4)
        draw = lambda *s: torch.randn(s, generator=g)
        self.q, self.k, self.v = draw(t, keys, d).to(dtype), draw(t, keys, d), draw(t, heads, e).to(dtype)
        self.k = (0.6 * self.q.float() + 0.8 * self.k).to(dtype)
        self.b, self.a, self.g = draw(t, heads).to(dtype), draw(t, ra).to(dtype), draw(t, rg).to(dtype)
        self.a2, self.g2 = (draw(heads, d, ra) * strength * ra ** -0.5).to(dtype), (draw(heads, e, rg) * rg ** -0.5).to(dtype)
        self.dt, self.rate, self.norm = bias + draw(heads, d), (rate + 0.3 * draw(heads)).exp(), 1 + 0.3 * draw(e)
        pad = lambda x, n: torch.nn.functional.pad(x, (0, n - x.shape[-1]))
        self.x = torch.cat([pad(self.q, dk).reshape(t, -1), pad(self.k, dk).reshape(t, -1), pad(self.v, dv).reshape(t, -1)], 1).cuda().contiguous()
        side = torch.cat([pad(self.b, geo.b_cols), pad(self.a, geo.rank_a), pad(self.g, geo.rank_g)], 1)
        self.proj = torch.cat([torch.zeros(t, geo.channels, dtype=dtype), side], 1).cuda().contiguous()
        a2, g2 = torch.zeros(heads, dk, geo.rank_a, dtype=dtype), torch.zeros(heads, dv, geo.rank_g, dtype=dtype)
        a2[:, :d, :ra], g2[:, :e, :rg] = self.a2, self.g2
        self.w = delta.Weights(torch.zeros(4, geo.channels).cuda(), a2.reshape(-1, geo.rank_a).cuda(), pad(self.dt, dk).reshape(-1).cuda(), self.rate.cuda(),
                               DenseLinear(g2.reshape(-1, geo.rank_g).cuda()), pad(self.norm, dv).cuda())
        self.finish(lens, heads, geo, slots, g)

    def want(self):
        out, states, a, rep = [], [], 0, self.heads // self.geo.key_heads
        for n, slot in zip(self.lens, self.slots):
            s = slice(a, a + n)
            z = np.einsum("tr,hdr->thd", np64(self.a[s]), np64(self.a2)) + np64(self.dt)
            g = np.exp(-np64(self.rate)[:, None] * oracle.softplus(z))
            state = np64(self.state0[slot, :, : self.geo.dim, : self.geo.vdim]).copy()
            q, k = (np.repeat(oracle.unit(np64(x[s])), rep, 1) for x in (self.q, self.k))
            o = oracle.delta_rule(q * self.geo.dim ** -0.5, k, np64(self.v[s]), oracle.sigmoid(np64(self.b[s])), g, state)
            gate = oracle.sigmoid(np.einsum("tr,her->the", np64(self.g[s]), np64(self.g2)))
            out.append(oracle.rms(o, self.geo.eps) * np64(self.norm) * gate)
            states.append(state)
            a += n
        return np.concatenate(out), states


DELTA_SIZES = [(4, 2, 24, 40), (2, 2, 64, 64), (3, 1, 48, 112), (2, 1, 128, 128), (6, 3, 16, 16), (1, 1, 112, 256), (4, 4, 80, 32)]


@BOTH
@pytest.mark.parametrize("heads,keys,d,e", DELTA_SIZES + [(1, 1, 256, 256), (2, 1, 256, 512)])
def test_delta_rule_token_by_token(heads, keys, d, e, dtype):
    from mfq_b200.ops import delta
    case = Delta([5, 1, 9, 2], heads, keys, d, e, dtype, slots=[4, 0, 2, 1])
    y = delta.recurrent(case.x, case.proj, case.w, case.state, i32(*case.slots), case.geo, starts=case.starts)
    case.check(y, 2e-4 if dtype == FP32 else 2e-2, 2e-5)


@pytest.mark.parametrize("split", [1, 2, 4, 8])
def test_delta_rule_with_split_columns_and_masked_rows(split):
    from mfq_b200.ops import delta
    case = Delta([1] * 5, 2, 1, 40, 128, FP32, slots=[6, 3, 0, 1, 5])
    case.check(delta.recurrent(case.x, case.proj, case.w, case.state, i32(*case.slots), case.geo, split=split), 2e-4, 2e-5)
    before = case.state.clone()
    delta.recurrent(case.x, case.proj, case.w, case.state, i32(0, -1, 2, -1, -1), case.geo, split=split)
    assert torch.equal(case.state[[1, 3, 4, 5, 6]], before[[1, 3, 4, 5, 6]]) and not torch.equal(case.state[0], before[0])


@pytest.mark.parametrize("heads,keys,d,e", DELTA_SIZES)
@pytest.mark.parametrize("lens", [[64], [200, 2, 63, 65, 128, 1, 17], [15, 16, 333]])
def test_delta_rule_in_chunks(heads, keys, d, e, lens):
    from mfq_b200.ops import delta
    case = Delta(lens, heads, keys, d, e, BF16)
    y = delta.chunked(case.x, case.proj, case.w, case.state, i32(*case.slots), case.geo, case.starts, max(lens))
    case.check(y, 2e-2, 2e-4)
    check_status()


@pytest.mark.parametrize("bias,strength,rate", [(-9.0, 0.5, 0.0), (-2.0, 1.0, 0.0), (1.0, 3.0, 1.0), (4.0, 4.0, 2.0), (-3.0, 12.0, 1.5), (0.0, 1.0, 4.0)])
def test_delta_rule_decays_of_every_strength(bias, strength, rate):
    from mfq_b200.ops import delta
    how = dict(bias=bias, strength=strength, rate=rate)
    case = Delta([150, 70], 2, 1, 32, 48, BF16, **how)
    case.check(delta.chunked(case.x, case.proj, case.w, case.state, i32(*case.slots), case.geo, case.starts, 150), 2e-2, 5e-4)
    case = Delta([150, 70], 2, 1, 32, 48, FP32, **how)
    case.check(delta.recurrent(case.x, case.proj, case.w, case.state, i32(*case.slots), case.geo, starts=case.starts), 5e-4, 5e-5)
    check_status()


def test_delta_rule_of_repeated_keys():
    """The same key again and again with full strength: the triangular system is as far from the identity as it gets."""
    from mfq_b200.ops import delta
    case = Delta([130], 2, 2, 32, 32, BF16, bias=-12.0, strength=0.0)
    case.k[:], case.b[:] = case.k[:1].clone(), 6.0
    dk = case.geo.dk
    case.x[:, 2 * dk : 4 * dk] = case.x[:1, 2 * dk : 4 * dk].clone()
    case.proj[:, case.geo.channels : case.geo.channels + 2] = 6.0
    case.check(delta.chunked(case.x, case.proj, case.w, case.state, i32(0), case.geo, case.starts, 130), 2e-2, 5e-4)


def test_mixed_portions_and_singles_of_both_recurrences():
    from mfq_b200.ops import delta, gla
    lens = [1, 1, 1, 90, 2, 64]
    case = TimeMix(lens, 2, 40, 16, BF16)
    case.check(gla.ragged(case.proj, *case.args, case.state, i32(*case.slots), case.geo, case.starts, 90, 3, bonus=case.bonus), 2e-2, 2e-4)
    case = Delta(lens, 4, 2, 40, 56, BF16)
    delta.recurrent(case.x, case.proj, case.w, case.state, i32(*case.slots[:3]), case.geo, out=(out := torch.empty(159, 4 * 64, dtype=BF16, device="cuda")))
    delta.chunked(case.x, case.proj, case.w, case.state, i32(*case.slots[3:]), case.geo, case.starts[3:], 90, first=3, out=out)
    case.check(out, 2e-2, 2e-4)
    check_status()
