"""Kernels of the Kamedra family, each against the plain restatement: output stages of the products, rotation in pairs, windowed
attention with kept tokens and two maps, the difference of maps, and gated linear attention (token by token and in chunks)."""

import numpy as np
import pytest
import torch

import kamedra_oracle as oracle
from gpu_common import check_status, require_gpu_lib
from test_gpu_tepetar_ops import BF16, FP32, Pages, close, padded, rnd

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module", autouse=True)
def _lib():
    require_gpu_lib()
    from mfq_b200.ops.lib import dense_lib
    dense_lib()


def i32(*x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


# -- products ---------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [BF16, FP32])
@pytest.mark.parametrize("m,n,k", [(1, 16, 8), (3, 48, 72), (8, 592, 264), (16, 1040, 1000), (17, 128, 64), (64, 384, 1096), (130, 272, 320),
                                   (700, 3216, 200)])
def test_output_stages(m, n, k, dtype):
    from mfq_b200.ops import dense
    x, w = rnd(m, k, dtype=dtype), rnd(n, k, dtype=dtype, scale=3 * k ** -0.5)
    y = (x.double() @ w.double().T).cpu().numpy()
    tol = 2e-2 if dtype == BF16 else 2e-5
    close(dense.DenseLinear(w)(x, softcap=2.5), oracle.softcap(y, 2.5), tol, "soft cap")
    stream = rnd(m, n, dtype=FP32)
    want = stream.double().cpu().numpy() + y
    assert dense.DenseLinear(w)(x, add_to=stream) is stream
    close(stream, want, 1e-4 if dtype == BF16 else 2e-5, "added to the stream")  # never rounded to bf16
    gate, up = rnd(n // 2, k, dtype=dtype, scale=2 * k ** -0.5), rnd(n // 2, k, dtype=dtype, scale=2 * k ** -0.5)
    got = dense.DenseLinear(dense.interleave_glu(gate, up), glu="gelu")(x)
    plain = lambda a: (x.double() @ a.double().T).cpu().numpy()
    close(got, oracle.gelu_tanh(plain(gate)) * plain(up), tol, "gelu unit")
    check_status()


@pytest.mark.parametrize("tile", [16, 64, 128, 256])
@pytest.mark.parametrize("splits", [1, 3, 8])
def test_addition_through_every_tile_and_split(tile, splits):
    from mfq_b200.ops import dense
    m, n, k = 2 * tile - 5, 336, 1096
    x, w, stream = rnd(m, k), rnd(n, k, scale=k ** -0.5), rnd(m, n, dtype=FP32)
    want = (stream.double() + x.double() @ w.double().T).cpu()
    close(dense.DenseLinear(w)(x, add_to=stream, tile=tile, splits=splits), want, 1e-4)
    check_status()


# -- per-head stage -----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [BF16, FP32])
@pytest.mark.parametrize("h,g,d,e,rot", [(6, 2, 20, 24, 12), (4, 4, 16, 48, 2), (5, 1, 48, 40, 48), (2, 1, 128, 256, 64), (3, 3, 40, 16, 0)])
def test_heads_between_projection_and_attention(h, g, d, e, rot, dtype):
    from mfq_b200.engine.kv_cache import PlainPagedKVCache
    from mfq_b200.ops import window_attn
    from mfq_b200.ops.dense import up
    dk, dv, t = up(d), up(e), 37
    sc = {"factor": 5.0, "low": 1.0, "high": 6.0, "original": 200}
    pos, slots = torch.randint(0, 900, (t,)), torch.randperm(64)[:t].int() + 16
    slots[5] = -1
    cache = PlainPagedKVCache([(g, 2 * dk, dv)], dtype, num_pages=6, max_seqs=1, max_pages_per_seq=6, device="cuda")
    q, k, v = (torch.randn(t, n, x).to(dtype) for n, x in ((2 * h, d), (2 * g, d), (g, e)))
    rows = torch.cat([padded(q, dk).reshape(t, -1), padded(k, dk).reshape(t, -1), padded(v, dv).reshape(t, -1)], 1)
    table = window_attn.rope_table(3e4, rot, 1000, "cuda", window_attn.FrequencyScaling(*(sc[n] for n in ("factor", "low", "high", "original")))) if rot else None
    how = dict(heads=h, kv_heads=g, dim=d, q_norm=None, k_norm=None, rope=table, rot=rot, eps=1e-5, maps=2, pairs=True)
    got = window_attn.qkv_finish(rows, cache.layer(0), pos.int().cuda(), slots.cuda(), **how)
    tol = 1e-5 if dtype == FP32 else 2e-2
    turn = lambda x: oracle.rotate_pairs(x.double().numpy(), pos.numpy(), oracle.frequencies(3e4, rot, sc))
    close(got[..., :d], turn(q), tol, "q")
    assert not got[..., d:].any()
    ok = slots >= 0
    pg, off = (slots[ok] // 16).long().cuda(), (slots[ok] % 16).long().cuda()
    kept = cache.layer(0).k[pg, :, off].view(-1, 2 * g, dk)
    close(kept[..., :d], turn(k)[ok.numpy()], tol, "k")
    close(cache.layer(0).v[pg, :, off][..., :e], v.double().numpy()[ok.numpy()], tol, "v")
    untouched = torch.ones(96, dtype=torch.bool)
    untouched[slots[ok].long()] = False
    assert not cache.layer(0).k.transpose(1, 2).reshape(96, -1)[untouched.cuda()].any()
    before = cache.layer(0).k.clone()
    alone = window_attn.qkv_finish(rows[:, : 2 * h * dk].contiguous(), None, pos.int().cuda(), slots.cuda(), dk=dk, **how)
    assert torch.equal(alone, got) and torch.equal(cache.layer(0).k, before)


# -- attention ----------------------------------------------------------------------------------------------------------
class TwoMaps:
    """Pages whose rows hold both key maps side by side, and the restatement's answer."""

    def __init__(self, lens, h, g, d, e, dtype=BF16):
        from mfq_b200.ops.dense import up
        self.h, self.g, self.d, self.e, self.dk = h, g, d, e, up(d)
        self.pages = Pages(lens, g, 2 * self.dk, e, dtype)
        if self.dk != d:
            for k in self.pages.k:
                k.view(-1, g, 2, self.dk)[..., d:] = 0
            self.pages.store()
        self.kv, self.table = self.pages.kv, self.pages.cache.block_table

    def order(self, q):
        """``[T, H, 2, d]`` as the kernels take it: ``[KV head][map][head of the KV head]``, padded."""
        t, per = q.shape[0], self.h // self.g
        return padded(q.view(t, self.g, per, 2, self.d).transpose(2, 3).reshape(t, 2 * self.h, self.d), self.dk)

    def maps(self, b, q, first, scale, window, keep):
        """Both maps' outputs ``[T, H, 2, e]``."""
        k = self.pages.k[b].view(-1, self.g, 2, self.dk)[..., : self.d].double().numpy()
        v, q = self.pages.v[b].double().numpy(), q.double().numpy()
        see = oracle.visible(first + np.arange(len(q)), np.arange(self.pages.lens[b]), window, keep)
        per = self.h // self.g
        return np.stack([np.stack([oracle.attend(q[:, n, m], k[:, n // per, m], v[:, n // per], see, scale) for m in (0, 1)], 1)
                         for n in range(self.h)], 1)

    def diff(self, maps, d):
        return oracle.rms(maps[:, :, 0] - d.weight * maps[:, :, 1], d.eps) * d.scale


TWO = [  # heads, kv heads, dim, vdim, window, keep
    (8, 2, 48, 96, 112, 20), (6, 2, 20, 24, 40, 3), (5, 1, 80, 128, 1, 16), (4, 4, 128, 128, 200, 0), (3, 3, 16, 16, 33, 33),
    (24, 1, 32, 64, 17, 1), (2, 1, 128, 256, 150, 64), (12, 2, 64, 128, 1 << 30, 5), (2, 2, 192, 96, 50, 130), (40, 2, 16, 80, 64, 250)]


def spec(d, window, keep, cap=0.0):
    return dict(window=window, keep=keep, scale=1.3 * d ** -0.5, cap=cap)


def combine(e, eps=1e-4):
    from mfq_b200.ops.window_attn import Difference
    return Difference(0.45, 0.7, eps, e)


@pytest.mark.parametrize("h,g,d,e,window,keep", TWO)
def test_attention_of_portions(h, g, d, e, window, keep):
    from mfq_b200.ops import window_attn
    lens, portion = [300, 5, 129, 64, 260], [300, 2, 60, 3, 131]
    tm, how, dd = TwoMaps(lens, h, g, d, e), spec(d, window, keep), combine(e)
    q = [torch.randn((m, h, 2, d)).to(BF16) * 2 for m in portion]
    starts = i32(0, *np.cumsum(portion).tolist())
    maps = window_attn.prefill(tm.order(torch.cat(q)), tm.kv, tm.table, starts, i32(*lens), max(portion), maps=2, **how)
    check_status()
    out = window_attn.difference(maps, g, dd)
    for b, m in enumerate(portion):
        a = int(starts[b])
        want = tm.maps(b, q[b], lens[b] - m, how["scale"], window, keep)
        got = maps[a : a + m, :, :e].view(m, g, 2, h // g, e).transpose(2, 3).reshape(m, h, 2, e)
        close(got, want, 4e-2, f"maps of sequence {b}")
        close(out[a : a + m, :, :e], tm.diff(want, dd), 0.15, f"sequence {b}")
        assert not out[a : a + m, :, e:].any()


@pytest.mark.parametrize("splits", [1, 2, 5])
@pytest.mark.parametrize("h,g,d,e,window,keep", TWO)
def test_attention_of_single_tokens(h, g, d, e, window, keep, splits):
    from mfq_b200.ops import window_attn
    lens = [300, 1, 16, 17, 129, 97, 255]
    tm, how, dd = TwoMaps(lens, h, g, d, e), spec(d, window, keep), combine(e)
    q = torch.randn((len(lens), h, 2, d)).to(BF16) * 2
    out = window_attn.decode(tm.order(q), tm.kv, tm.table, i32(*lens), diff=dd, splits=splits, **how)
    for b, n in enumerate(lens):
        want = tm.diff(tm.maps(b, q[b : b + 1], n - 1, how["scale"], window, keep), dd)
        close(out[b : b + 1, :, :e], want, 0.1, f"sequence of {n}")


@pytest.mark.parametrize("dtype", [BF16, FP32])
@pytest.mark.parametrize("h,g,d,e,window,keep", TWO)
def test_attention_in_fp32(h, g, d, e, window, keep, dtype):
    from mfq_b200.ops import window_attn
    lens = [200, 33]
    tm, how, dd = TwoMaps(lens, h, g, d, e, dtype), spec(d, window, keep), combine(e)
    pick = [(0, 0), (0, 16), (1, 32), (0, 199), (1, 3), (0, 130)]
    q = torch.randn((len(pick), h, 2, d)).to(dtype)
    maps = window_attn.plain(tm.order(q), tm.kv, tm.table, i32(*(p[0] for p in pick)), i32(*(p[1] for p in pick)), maps=2, **how)
    out = window_attn.difference(maps, g, dd)
    for i, (b, p) in enumerate(pick):
        want = tm.diff(tm.maps(b, q[i : i + 1], p, how["scale"], window, keep), dd)
        close(out[i : i + 1, :, :e], want, 2e-5 if dtype == FP32 else 5e-2, f"token {i}")


@pytest.mark.parametrize("hq,hk,d,e,window,keep,cap", [(6, 2, 32, 24, 40, 5, 2.0), (7, 1, 80, 128, 17, 40, 0.0)])
def test_kept_tokens_of_a_single_map(hq, hk, d, e, window, keep, cap):
    """The same windows for plain attention, with and without a score cap."""
    from mfq_b200.ops import window_attn
    from mfq_b200.ops.dense import up
    n, how = 210, spec(d, window, keep, cap)
    pg = Pages([n], hk, d, e)
    q = torch.randn((n, hq, d)).to(BF16) * 2
    see = oracle.visible(range(n), range(n), window, keep)
    k, v = pg.k[0].double().numpy(), pg.v[0].double().numpy()

    def head(i):
        s = np.where(see, oracle.softcap(q[:, i].double().numpy() @ k[:, i * hk // hq].T * how["scale"], cap), -np.inf)
        p = np.exp(s - s.max(-1, keepdims=True))
        return (p / p.sum(-1, keepdims=True)) @ v[:, i * hk // hq]
    want = np.stack([head(i) for i in range(hq)], 1)
    out = window_attn.prefill(padded(q, up(d)), pg.kv, pg.cache.block_table, i32(0, n), i32(n), n, **how)
    close(out[..., :e], want, 4e-2, "portion")
    for splits in (1, 3):
        got = window_attn.decode(padded(q[-1:], up(d)), pg.kv, pg.cache.block_table, i32(n), splits=splits, **how)
        close(got[..., :e], want[-1:], 4e-2, "single")
    check_status()


@pytest.mark.parametrize("window,keep", [(5, 0), (5, 1), (16, 16), (17, 15), (128, 17), (200, 40), (3, 150)])
def test_a_key_at_an_edge_decides(window, keep):
    """One key of the first map matches far better than all others: its value must be the result exactly where it is visible --
    in a portion, as single tokens and in fp32 -- among kept tokens and at the window's two ends."""
    from mfq_b200.ops import window_attn
    h, g, d, e, n = 2, 1, 32, 16, 420
    how = dict(window=window, keep=keep, scale=0.5, cap=0.0)
    tm = TwoMaps([n], h, g, d, e)
    base_k, base_v = tm.pages.k[0].clone(), tm.pages.v[0].clone()
    q = torch.ones((n, h, 2, d)).to(BF16)
    only_first = combine(e)
    for spot in sorted({0, max(0, keep - 1), keep, keep + 1, 15, 16, 37, 151, 200}):
        tm.pages.k[0], tm.pages.v[0] = -base_k.abs(), base_v.clone()
        tm.pages.k[0][spot, :, :32] = 1.5
        tm.pages.v[0][spot] = 9.0
        tm.pages.store()
        maps = window_attn.prefill(tm.order(q), tm.kv, tm.table, i32(0, n), i32(n), n, maps=2, **how).view(n, 2, h, e)
        hit = ((maps[:, 0] - 9.0).abs().amax((1, 2)) < 0.1).cpu().numpy()
        see = oracle.visible(range(n), [spot], window, keep)[:, 0]
        assert (hit == see).all(), (spot, np.flatnonzero(hit != see)[:5])
        assert (maps[:, 1] - 9.0).abs().max() > 1.0
        for p in sorted({spot, spot + window - 1, min(n - 1, spot + window), n - 1, min(n - 1, max(spot, 31)), min(n - 1, spot + 64)}):
            want = tm.diff(tm.maps(0, q[p : p + 1], p, 0.5, window, keep), only_first)
            for splits in (1, 3):
                o = window_attn.decode(tm.order(q[:1]), tm.kv, tm.table, i32(p + 1), diff=only_first, splits=splits, **how)
                close(o, want, 5e-2, f"spot {spot}, position {p}")
            o = window_attn.plain(tm.order(q[:1]), tm.kv, tm.table, i32(0), i32(p), maps=2, **how)
            assert bool((o[:, :h] - 9.0).abs().max() < 0.1) == bool(see[p])
    check_status()


# -- gated linear attention -----------------------------------------------------------------------------------------------
class Gla:
    """Random projections of some portions, states to start from, and the restatement's answer (over the same rounded inputs)."""

    def __init__(self, lens, heads, d, e, rank, tau, dtype, bias=2.0, strength=1.0, slots=None, seed=0):
        from mfq_b200.ops.dense import up
        from mfq_b200.ops.gla import Geometry
        g = torch.Generator().manual_seed(seed)
        t = sum(lens)
        self.lens, self.geo = lens, Geometry(heads, up(d), up(e), d, e, up(rank), tau, 1e-5)
        draw = lambda *s: torch.randn(s, generator=g)
        self.q, self.k, self.v, self.z = (draw(t, heads, x).to(dtype) for x in (d, d, e, e))
        self.a, self.w2 = draw(t, rank).to(dtype), (draw(heads, d, rank) * strength * rank ** -0.5).to(dtype)
        self.bias, self.norm = bias + draw(heads, d), 1 + 0.3 * draw(e)
        pad = lambda x, n: torch.nn.functional.pad(x, (0, n - x.shape[-1]))
        geo = self.geo
        self.proj = torch.cat([pad(self.q, geo.dk).reshape(t, -1), pad(self.k, geo.dk).reshape(t, -1), pad(self.v, geo.dv).reshape(t, -1),
                               pad(self.z, geo.dv).reshape(t, -1), pad(self.a, geo.rank)], 1).cuda().contiguous()
        w2 = torch.zeros(heads, geo.dk, geo.rank, dtype=dtype)
        w2[:, :d, :rank] = self.w2
        self.args = (w2.reshape(-1, geo.rank).cuda(), pad(self.bias, geo.dk).reshape(-1).cuda(), pad(self.norm, geo.dv).cuda())
        self.slots = slots if slots is not None else list(range(len(lens)))[::-1]
        self.state0 = torch.zeros(len(lens) + 2, heads, geo.dk, geo.dv)
        self.state0[:, :, :d, :e] = draw(len(lens) + 2, heads, d, e)
        self.state = self.state0.cuda()
        self.starts = i32(0, *np.cumsum(lens).tolist())

    def want(self):
        """``(y [T, H, e], final states of the sequences)``."""
        geo, out, states, a = self.geo, [], [], 0
        for n, slot in zip(self.lens, self.slots):
            s = slice(a, a + n)
            f = lambda x: x[s].double().numpy()
            alpha = oracle.sigmoid(np.einsum("tr,hdr->thd", f(self.a), self.w2.double().numpy()) + self.bias.double().numpy()) ** (1 / geo.tau)
            state = self.state0[slot, :, : geo.dim, : geo.vdim].double().numpy().copy()
            o = oracle.gated_linear_attention(f(self.q) * geo.dim ** -0.5, f(self.k), f(self.v), alpha, state)
            z = f(self.z)
            out.append(oracle.norm(o, self.norm.double().numpy(), geo.eps) * z * oracle.sigmoid(z))
            states.append(state)
            a += n
        return np.concatenate(out), states

    def check(self, y, tol, state_tol):
        geo = self.geo
        want, states = self.want()
        y = y.view(y.shape[0], geo.heads, geo.dv)
        close(y[..., : geo.vdim], want, tol, "y")
        assert not y[..., geo.vdim :].any()
        for slot, s in zip(self.slots, states):
            close(self.state[slot, :, : geo.dim, : geo.vdim], s, state_tol, f"state of slot {slot}")
            rest = self.state[slot].clone()
            rest[:, : geo.dim, : geo.vdim] = 0
            assert not rest.any()
        for other in set(range(len(self.state0))) - set(self.slots):
            assert torch.equal(self.state[other].cpu(), self.state0[other])


SIZES = [(3, 24, 40, 8), (2, 64, 64, 16), (6, 32, 48, 20), (1, 128, 256, 16), (2, 48, 112, 24), (1, 256, 512, 32), (4, 16, 16, 5), (2, 128, 128, 64)]


@pytest.mark.parametrize("dtype", [BF16, FP32])
@pytest.mark.parametrize("heads,d,e,rank", SIZES)
def test_recurrence_token_by_token(heads, d, e, rank, dtype):
    from mfq_b200.ops import gla
    case = Gla([5, 1, 9, 2], heads, d, e, rank, 4.0, dtype, slots=[4, 0, 2, 1])
    y = gla.recurrent(case.proj, *case.args, case.state, i32(*case.slots), case.geo, starts=case.starts)
    case.check(y, 1e-4 if dtype == FP32 else 2e-2, 1e-5)


@pytest.mark.parametrize("split", [1, 2, 4, 8])
def test_one_token_per_sequence_with_split_columns(split):
    from mfq_b200.ops import gla
    case = Gla([1] * 5, 2, 40, 128, 16, 2.0, FP32, slots=[6, 3, 0, 1, 5])
    out = torch.zeros(5, 2 * 128, device="cuda")
    y = gla.recurrent(case.proj, *case.args, case.state, i32(*case.slots), case.geo, split=split, out=out)
    case.check(y, 1e-4, 1e-5)
    again = Gla([7, 3], 2, 40, 128, 16, 2.0, FP32)
    case = again
    case.check(gla.recurrent(case.proj, *case.args, case.state, i32(*case.slots), case.geo, starts=case.starts, split=split), 1e-4, 1e-5)


def test_masked_rows_keep_their_state():
    from mfq_b200.ops import gla
    case = Gla([1] * 4, 2, 32, 32, 16, 2.0, BF16, slots=[0, 1, 2, 3])
    before = case.state.clone()
    gla.recurrent(case.proj, *case.args, case.state, i32(0, -1, 2, -1), case.geo, split=2)
    assert torch.equal(case.state[[1, 3, 4, 5]], before[[1, 3, 4, 5]]) and not torch.equal(case.state[0], before[0])
    before = case.state.clone()
    long = Gla([70, 70], 2, 32, 32, 16, 2.0, BF16)
    gla.chunked(long.proj, *long.args, case.state, i32(-1, 3), long.geo, long.starts, 70)
    assert torch.equal(case.state[[0, 1, 2, 4, 5]], before[[0, 1, 2, 4, 5]]) and not torch.equal(case.state[3], before[3])


@pytest.mark.parametrize("heads,d,e,rank", SIZES)
@pytest.mark.parametrize("lens", [[64], [200, 2, 63, 65, 128, 1, 17], [15, 16, 333]])
def test_recurrence_in_chunks(heads, d, e, rank, lens):
    from mfq_b200.ops import gla
    case = Gla(lens, heads, d, e, rank, 4.0, BF16)
    y = gla.chunked(case.proj, *case.args, case.state, i32(*case.slots), case.geo, case.starts, max(lens))
    case.check(y, 2e-2, 2e-4)


@pytest.mark.parametrize("tau,bias,strength", [(16.0, 4.0, 1.0), (1.0, 0.0, 1.0), (1.0, -3.0, 6.0), (1.0, -12.0, 10.0), (0.25, -5.0, 40.0), (1.0, 0.0, 60.0)])
def test_decays_of_every_strength(tau, bias, strength):
    """From channels that forget nothing to channels that forget everything within a token; both forms."""
    from mfq_b200.ops import gla
    for lens in ([150, 70],):
        case = Gla(lens, 2, 32, 48, 16, tau, BF16, bias, strength)
        y = gla.chunked(case.proj, *case.args, case.state, i32(*case.slots), case.geo, case.starts, max(lens))
        case.check(y, 2e-2, 2e-4)
        case = Gla(lens, 2, 32, 48, 16, tau, FP32, bias, strength)
        case.check(gla.recurrent(case.proj, *case.args, case.state, i32(*case.slots), case.geo, starts=case.starts), 3e-4, 2e-5)


def test_a_far_key_returns_its_value():
    """One key is met again long after, by the only query that points along it, through channels that do not decay: the value must
    come back from before several chunks and portions."""
    from mfq_b200.ops import gla
    n, heads, d, e = 330, 1, 32, 32
    case = Gla([n], heads, d, e, 8, 16.0, BF16, bias=60.0, strength=0.0)
    case.state0.zero_()
    case.proj[:, : 2 * d] *= 0.02
    for spot in (0, 15, 16, 63, 64, 100):
        proj = case.proj.clone()
        proj[spot, d : 2 * d] = 3.0
        proj[spot, 2 * d : 2 * d + e] = torch.where(torch.arange(e, device="cuda") % 2 == 0, 5.0, -5.0).to(BF16)
        proj[n - 1, :d] = 2.0
        proj[n - 1, 2 * d + e : 2 * d + 2 * e] = 4.0
        outs = []
        for cuts in ([n], [64, n - 64], [spot + 1, 100, n - spot - 101]):
            state, a, y = torch.zeros_like(case.state), 0, None
            for m in cuts:
                y = gla.chunked(proj[a : a + m], *case.args, state, i32(0), case.geo, i32(0, m), m)
                a += m
            outs.append(y[-1])
        state = torch.zeros_like(case.state)
        outs.append(gla.recurrent(proj, *case.args, state, i32(0), case.geo, starts=i32(0, n))[-1])
        for y in outs:
            y = y.float() / (case.args[2] * 4.0)
            assert (y[::2] > 0.8).all() and (y[1::2] < -0.8).all()


def test_mixed_portions_and_singles():
    from mfq_b200.ops import gla
    lens = [1, 1, 1, 90, 2, 64]
    case = Gla(lens, 2, 40, 56, 16, 3.0, BF16)
    y = gla.ragged(case.proj, *case.args, case.state, i32(*case.slots), case.geo, case.starts, 90, 3)
    case.check(y, 2e-2, 2e-4)
    case = Gla([1, 3, 2], 2, 40, 56, 16, 3.0, BF16)
    case.check(gla.ragged(case.proj, *case.args, case.state, i32(*case.slots), case.geo, case.starts, 3, 1), 2e-2, 1e-5)
