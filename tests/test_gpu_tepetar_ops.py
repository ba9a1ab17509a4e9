"""Kernels of the unquantized path, each against a plain restatement: products and their output stages, the fp32 stream, the
per-head stage, and windowed attention over pages."""

import numpy as np
import pytest
import torch

import tepetar_oracle as oracle
from gpu_common import check_status, require_gpu_lib

pytestmark = pytest.mark.gpu
BF16, FP32 = torch.bfloat16, torch.float32


@pytest.fixture(scope="module", autouse=True)
def _lib():
    require_gpu_lib()
    from mfq_b200.ops.lib import dense_lib
    dense_lib()


def close(got, want, tol, what=""):
    """Element by element: the error is within ``tol`` of the value plus the tensor's root mean square."""
    got, want = np.asarray(got.float().cpu(), dtype=np.float64), np.asarray(want, dtype=np.float64)
    assert got.shape == want.shape, (what, got.shape, want.shape)
    worst = (np.abs(got - want) / (np.abs(want) + np.sqrt((want ** 2).mean()) + 1e-12)).max()
    assert worst <= tol, f"{what}: error {worst:.3g} of the value plus rms, allowed {tol:g}"


def rnd(*shape, dtype=BF16, scale=1.0):
    return (torch.randn(shape, device="cuda") * scale).to(dtype)


@pytest.mark.parametrize("dtype", [BF16, FP32])
@pytest.mark.parametrize("m,n,k", [(1, 16, 8), (3, 48, 72), (8, 592, 264), (11, 160, 392), (16, 1040, 1000), (17, 128, 64),
                                   (33, 208, 2048), (64, 384, 1096), (100, 144, 512), (130, 272, 320), (300, 640, 96), (700, 3216, 200)])
def test_products(m, n, k, dtype):
    from mfq_b200.ops import dense
    x, w, b = rnd(m, k + 8, dtype=dtype)[:, :k], rnd(n, k, dtype=dtype, scale=k ** -0.5), rnd(n, dtype=FP32)
    want = x.double() @ w.double().T
    tol = 2e-2 if dtype == BF16 else 2e-5
    close(dense.DenseLinear(w)(x), want.cpu(), tol, "no bias")
    close(dense.DenseLinear(w, b)(x), (want + b.double()).cpu(), tol, "bias")
    half = n // 2
    gate, up = rnd(half, k, dtype=dtype, scale=2 * k ** -0.5), rnd(half, k, dtype=dtype, scale=2 * k ** -0.5)
    glu = dense.DenseLinear(dense.interleave_glu(gate, up), glu=(1.702, 1.3))(x)
    want_glu = oracle.clipped_glu((x.double() @ gate.double().T).cpu().numpy(), (x.double() @ up.double().T).cpu().numpy(), 1.3)
    close(glu, want_glu, tol, "clipped glu")
    table, ids = rnd(13, n, dtype=dtype), torch.randint(0, 13, (m,), device="cuda", dtype=torch.int32)
    got = dense.DenseLinear(w)(x, table=table, ids=ids)
    close(got, oracle.gelu_tanh(want.cpu().numpy()) * table[ids.long()].double().cpu().numpy(), tol, "gelu x table")
    check_status()


@pytest.mark.parametrize("tile", [16, 32, 64, 128, 256])
@pytest.mark.parametrize("splits", [1, 2, 3, 5, 8])
def test_every_tile_and_split(tile, splits):
    from mfq_b200.ops import dense
    m, n, k = 2 * tile - 5, 336, 1096
    x, w, b = rnd(m, k), rnd(n, k, scale=k ** -0.5), rnd(n, dtype=FP32)
    want = (x.double() @ w.double().T + b.double()).cpu()
    close(dense.DenseLinear(w, b)(x, tile=tile, splits=splits), want, 2e-2)
    a = dense.DenseLinear(w, b)(x, tile=tile, splits=splits)
    assert torch.equal(a, dense.DenseLinear(w, b)(x, tile=tile, splits=splits))  # the split order is fixed
    check_status()


@pytest.mark.parametrize("dtype", [BF16, FP32])
@pytest.mark.parametrize("width", [104, 256, 1000, 4096, 8200])
def test_stream(width, dtype):
    from mfq_b200.ops import dense
    w, m, eps = dense.up(width), 7, 1e-3
    pad = lambda t: torch.nn.functional.pad(t, (0, w - width))
    table, ids = pad(rnd(11, width, dtype=dtype)), torch.randint(0, 11, (m,), device="cuda", dtype=torch.int32)
    x, act = dense.embed_scaled(ids, table, 2.5)
    want = table[ids.long()].double() * 2.5
    close(x, want.cpu(), 1e-6, "embed")
    y, f = pad(rnd(m, width, dtype=dtype, scale=0.02)), pad(rnd(width, dtype=FP32))
    dense.norm_add(y, f, x, act, width, eps)
    want = want.cpu().numpy()[:, :width] + oracle.norm_plain(y.double().cpu().numpy()[:, :width], f.double().cpu().numpy()[:width], eps)
    close(x[:, :width], want, 1e-6, "norm_add")
    assert torch.equal(act, x.to(dtype)) and not x[:, width:].any()
    got = dense.norm_out(x, f, width, eps, dtype)
    close(got[:, :width], oracle.norm_plain(want, f.double().cpu().numpy()[:width], eps), 1e-5 if dtype == FP32 else 1.5e-2, "norm_out")


class Pages:
    """Random pages of a few sequences in scattered, interleaved page ids; the logical keys and values stay on the host."""

    def __init__(self, lens, hk, d, e, dtype=BF16, seed=0):
        from mfq_b200.engine.kv_cache import PlainPagedKVCache
        from mfq_b200.ops.dense import up
        g = torch.Generator().manual_seed(seed)
        per = [-(-n // 16) for n in lens]
        self.cache = PlainPagedKVCache([(hk, up(d), up(e))], dtype, num_pages=sum(per) + 4, max_seqs=len(lens),
                                       max_pages_per_seq=max(per) + 1, device="cuda")
        self.kv = self.cache.layer(0)
        ids = (torch.randperm(sum(per) + 3, generator=g) + 1).tolist()
        self.k = [torch.randn((n, hk, d), generator=g).to(dtype) for n in lens]
        self.v = [torch.randn((n, hk, e), generator=g).to(dtype) for n in lens]
        self.lens, self.d, self.e = lens, d, e
        self.pages = []
        for b, n in enumerate(lens):
            mine = [ids.pop() for _ in range(per[b])]
            self.pages.append(mine)
            self.cache.block_table[b, : len(mine)] = torch.tensor(mine, dtype=torch.int32)
        self.store()

    def store(self):
        for b, n in enumerate(self.lens):
            for t in range(n):
                pg = self.pages[b][t // 16]
                self.kv.k[pg, :, t % 16, : self.d] = self.k[b][t].cuda()
                self.kv.v[pg, :, t % 16, : self.e] = self.v[b][t].cuda()

    def want(self, b, q, first, **how):
        return oracle.attend(q.double().numpy(), self.k[b].double().numpy(), self.v[b].double().numpy(), first + np.arange(len(q)),
                             np.arange(self.lens[b]), how["scale"], how["cap"] or 1e30, how["window"])


def padded(q, dk):
    return torch.nn.functional.pad(q, (0, dk - q.shape[-1])).cuda().contiguous()


GEOMETRY = [  # query heads, kv heads, dim, vdim, window, cap
    (8, 2, 64, 80, 112, 30.0), (6, 2, 32, 24, 40, 2.0), (5, 1, 80, 128, 1, 20.0), (4, 4, 128, 128, 200, 0.0), (3, 3, 16, 16, 33, 7.0),
    (32, 2, 128, 64, 130, 30.0), (7, 1, 192, 96, 64, 50.0), (2, 1, 256, 256, 150, 10.0), (40, 2, 48, 200, 1 << 30, 50.0)]


def how_of(d, window, cap):
    return dict(window=window, scale=1.3 * d ** -0.5, cap=cap)


@pytest.mark.parametrize("hq,hk,d,e,window,cap", GEOMETRY)
def test_attention_of_portions(hq, hk, d, e, window, cap):
    from mfq_b200.ops import window_attn
    from mfq_b200.ops.dense import up
    lens, portion = [300, 5, 129, 64, 260], [300, 2, 60, 3, 131]
    pg, how = Pages(lens, hk, d, e), how_of(d, window, cap)
    q = [torch.randn((m, hq, d)).to(BF16) * 2 for m in portion]
    starts = torch.tensor([0] + list(np.cumsum(portion)), dtype=torch.int32, device="cuda")
    out = window_attn.prefill(padded(torch.cat(q), up(d)), pg.kv, pg.cache.block_table, starts,
                              torch.tensor(lens, dtype=torch.int32, device="cuda"), max(portion), **how)
    check_status()
    for b, m in enumerate(portion):
        a = int(starts[b])
        close(out[a : a + m, :, :e], pg.want(b, q[b], lens[b] - m, **how), 4e-2, f"sequence {b}")
        assert not out[a : a + m, :, e:].any()


@pytest.mark.parametrize("splits", [1, 2, 5])
@pytest.mark.parametrize("hq,hk,d,e,window,cap", GEOMETRY)
def test_attention_of_single_tokens(hq, hk, d, e, window, cap, splits):
    from mfq_b200.ops import window_attn
    from mfq_b200.ops.dense import up
    lens = [300, 1, 16, 17, 129, 97, 255]
    pg, how = Pages(lens, hk, d, e), how_of(d, window, cap)
    q = torch.randn((len(lens), hq, d)).to(BF16) * 2
    out = window_attn.decode(padded(q, up(d)), pg.kv, pg.cache.block_table, torch.tensor(lens, dtype=torch.int32, device="cuda"),
                             splits=splits, **how)
    for b, n in enumerate(lens):
        close(out[b : b + 1, :, :e], pg.want(b, q[b : b + 1], n - 1, **how), 4e-2, f"sequence of {n}")


@pytest.mark.parametrize("dtype", [BF16, FP32])
@pytest.mark.parametrize("hq,hk,d,e,window,cap", GEOMETRY)
def test_attention_in_fp32(hq, hk, d, e, window, cap, dtype):
    from mfq_b200.ops import window_attn
    from mfq_b200.ops.dense import up
    lens = [200, 33]
    pg, how = Pages(lens, hk, d, e, dtype), how_of(d, window, cap)
    pick = [(0, 0), (0, 16), (1, 32), (0, 199), (1, 3), (0, 130)]
    q = torch.randn((len(pick), hq, d)).to(dtype)
    seq, pos = (torch.tensor([p[i] for p in pick], dtype=torch.int32, device="cuda") for i in (0, 1))
    out = window_attn.plain(padded(q, up(d)), pg.kv, pg.cache.block_table, seq, pos, **how)
    for i, (b, p) in enumerate(pick):
        close(out[i : i + 1, :, :e], pg.want(b, q[i : i + 1], p, **how), 1e-5 if dtype == FP32 else 1e-2, f"token {i}")


@pytest.mark.parametrize("window", [5, 16, 17, 128, 200])
def test_a_key_at_the_windows_edge_decides(window):
    """One key matches the query far better than all others; the result must be its value while it is the last visible key,
    and must not know it one position later -- in a portion, as single tokens and in fp32."""
    from mfq_b200.ops import window_attn
    hq, hk, d, e, n = 2, 1, 32, 16, 400
    how = dict(window=window, scale=0.5, cap=50.0)
    for spot in (0, 15, 16, 37, 150):
        pg = Pages([n], hk, d, e)
        q = torch.ones((n, hq, d)).to(BF16)
        pg.k[0] = (-pg.k[0].abs()).clone()
        pg.k[0][spot] = 1.5
        pg.v[0][spot] = 9.0
        pg.store()
        seq_lens = torch.tensor([n], dtype=torch.int32, device="cuda")
        out = window_attn.prefill(padded(q, 32), pg.kv, pg.cache.block_table, torch.tensor([0, n], dtype=torch.int32, device="cuda"),
                                  seq_lens, n, **how)
        inside, outside = spot + window - 1, spot + window
        assert (out[inside] - 9.0).abs().max() < 0.1 and (out[outside] - 9.0).abs().min() > 1.0
        assert (out[spot] - 9.0).abs().max() < 0.1 and (spot == 0 or (out[spot - 1] - 9.0).abs().min() > 1.0)
        for p, hit in ((inside, True), (outside, False)):
            one = torch.tensor([p + 1], dtype=torch.int32, device="cuda")
            qd = padded(q[:1], 32)
            for splits in (1, 3):
                o = window_attn.decode(qd, pg.kv, pg.cache.block_table, one, splits=splits, **how)
                assert ((o - 9.0).abs().max() < 0.1) == hit
            o = window_attn.plain(qd, pg.kv, pg.cache.block_table, torch.zeros(1, dtype=torch.int32, device="cuda"), one - 1, **how)
            assert ((o - 9.0).abs().max() < 0.1) == hit
    check_status()


@pytest.mark.parametrize("peak", [0.05, 4.0, 14.0, 16.0, 90.0, 400.0])
def test_scores_small_and_large_against_the_cap(peak):
    """Raw scores of every size relative to the cap: the polynomial form, the exponential form and the saturated range."""
    from mfq_b200.ops import window_attn
    hq, hk, d, e, n, how = 4, 1, 64, 64, 200, dict(window=150, scale=0.125, cap=50.0)
    pg = Pages([n], hk, d, e)
    q = (torch.randn((n, hq, d)) * peak / 3.0).to(BF16)
    want = pg.want(0, q, 0, **how)
    out = window_attn.prefill(padded(q, 64), pg.kv, pg.cache.block_table, torch.tensor([0, n], dtype=torch.int32, device="cuda"),
                              torch.tensor([n], dtype=torch.int32, device="cuda"), n, **how)
    close(out, want, 6e-2, "portion")
    lens = torch.tensor([n], dtype=torch.int32, device="cuda")
    close(window_attn.decode(padded(q[-1:], 64), pg.kv, pg.cache.block_table, lens, **how), want[-1:], 6e-2, "single")
    check_status()


@pytest.mark.parametrize("dtype", [BF16, FP32])
@pytest.mark.parametrize("hq,hk,d,e,rot", [(6, 2, 32, 24, 24), (4, 4, 16, 48, 2), (5, 1, 80, 56, 36), (2, 1, 256, 128, 256), (3, 3, 20, 12, 20)])
def test_heads_between_projection_and_attention(hq, hk, d, e, rot, dtype):
    from mfq_b200.engine.kv_cache import PlainPagedKVCache
    from mfq_b200.ops import window_attn
    from mfq_b200.ops.dense import up
    dk, dv, t, eps, lam = up(d), up(e), 37, 1e-4, 0.3125
    pos = torch.randint(0, 900, (t,))
    slots = torch.randperm(64)[:t].int() + 16
    slots[5] = -1
    cache = PlainPagedKVCache([(hk, dk, dv)], dtype, num_pages=6, max_seqs=1, max_pages_per_seq=6, device="cuda")
    q, k, v, v1 = (torch.randn(t, h, x).to(dtype) for h, x in ((hq, d), (hk, d), (hk, e), (hk, e)))
    qn, kn = torch.randn(d), torch.randn(d)
    pad = torch.nn.functional.pad
    qkv = torch.cat([pad(q, (0, dk - d)).reshape(t, -1), pad(k, (0, dk - d)).reshape(t, -1), pad(v, (0, dv - e)).reshape(t, -1)], 1).cuda()
    first = torch.cat([torch.randn(t, 8).to(dtype), pad(v1, (0, dv - e)).reshape(t, -1)], 1).cuda()[:, 8:]
    got = window_attn.qkv_finish(qkv.contiguous(), cache.layer(0), pos.int().cuda(), slots.cuda(), heads=hq, kv_heads=hk, dim=d,
                                 q_norm=pad(qn, (0, dk - d)).cuda(), k_norm=pad(kn, (0, dk - d)).cuda(),
                                 rope=window_attn.rope_table(3e4, rot, 1000, "cuda"), rot=rot, eps=eps, v_first=first, mix=lam)
    tol = 1e-5 if dtype == FP32 else 2e-2
    turn = lambda x, w: oracle.rotate(oracle.norm_plain(x.double().numpy(), w.double().numpy(), eps), pos.numpy(), 3e4, rot)
    close(got[..., :d], turn(q, qn), tol, "q")
    assert not got[..., d:].any()
    ok = slots >= 0
    pg, off = (slots[ok] // 16).long().cuda(), (slots[ok] % 16).long().cuda()
    close(cache.layer(0).k[pg, :, off][..., :d], turn(k, kn)[ok.numpy()], tol, "k")
    close(cache.layer(0).v[pg, :, off][..., :e], oracle.mix_values(v.double().numpy(), v1.double().numpy(), lam)[ok.numpy()], tol, "v")
    untouched = torch.ones(96, dtype=torch.bool)
    untouched[slots[ok].long()] = False
    flat = cache.layer(0).k.transpose(1, 2).reshape(96, -1)
    assert not flat[untouched.cuda()].any()
