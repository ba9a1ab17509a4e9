"""Bufolorn without a GPU: the plain restatement against itself, configuration and names, weight layout, pages and state."""

import json

import numpy as np
import pytest
import torch

import bufolorn_cases as cases
import bufolorn_oracle as oracle


# -- the restatement ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("size", [1, 2, 7, 64])
def test_portions_of_the_restatement_agree(size):
    cfg = cases.uneven()
    model, toks = oracle.Model(cfg, cases.weights(cfg)), cases.tokens(cfg, 64)
    want, state = model.run(toks), model.start()
    got = np.concatenate([model.run(toks[a : a + size], state) for a in range(0, 64, size)])
    assert np.abs(got - want).max() < 1e-9


def test_mechanisms_of_the_restatement_by_hand():
    see = oracle.visible([0, 4], range(6), 3)
    assert [np.flatnonzero(r).tolist() for r in see] == [[0], [2, 3, 4]] and oracle.visible([3], range(6)).sum() == 4
    assert np.allclose(oracle.rotate_pairs(np.array([[[1.0, 0.0]]]), [3], [0.1], 2.0), [[[2 * np.cos(0.3), 2 * np.sin(0.3)]]])
    f, length = oracle.frequencies(100.0, 4, {"factor": 4.0, "original": 2 * np.pi * 10, "fast": 9.0, "slow": 0.11})
    assert np.allclose(f, [1.0, 0.1 / 4 * 0.5 + 0.1 * 0.5]) and np.isclose(length, 0.1 * np.log(4) + 1)  # ramp over places 0 .. 2
    assert np.allclose(oracle.temperature([0, 2, 3, 8], 2.0, 4), 1 + 2 * np.log([1, 1, 2, 3]))
    assert [oracle.bucket(n, 8, 64) for n in (0, 3, 4, 7, 8, 15, 16, 31, 32, 63, 64, 999)] == [0, 3, 4, 4, 5, 5, 6, 6, 7, 7, 7, 7]
    o = oracle.attend(np.array([[0.0, 0.0, 50.0]]), np.array([[True, True, False]]), np.array([[2.0], [4.0], [9.0]]), np.log(2.0))
    assert np.allclose(o, 6 / 4)
    y, hist = oracle.short_conv(np.array([[1.0], [2.0]]), np.array([[5.0], [7.0]]), np.array([[100.0, 10.0, 1.0]]))
    assert y.reshape(-1).tolist() == [571.0, 712.0] and hist.reshape(-1).tolist() == [1.0, 2.0]
    one = lambda *x: np.array(x, dtype=float).reshape(-1, 1, 1)
    state = np.zeros((1, 1, 1))
    out = oracle.delta_rule(one(2, 2), one(1, 3), one(10, 50), np.array([[0.5], [0.25]]), one(0.5, 0.2), state)
    assert np.allclose(out.reshape(-1), [10.0, 2 * (1 + 3 * 0.25 * (50 - 3 * 1))]) and np.isclose(state[0, 0, 0], 36.25)
    state = np.zeros((1, 1, 1))
    out = oracle.rwkv_rule(one(2, 3), one(1, 5), one(10, 7), one(0.5, 0.25), np.array([[4.0]]), state)
    assert out.reshape(-1).tolist() == [80.0, 3 * (10 + 4 * 35)] and state[0, 0, 0] == 37.5
    assert np.isclose(oracle.delta_decay(np.ones((1, 1)), np.ones((1, 1)), np.full((1, 1), 2.0), np.array([-2.0]), np.array([0.7]), 1)[0, 0, 0],
                      np.exp(-np.exp(0.7) * np.log(2)))
    ids, w = oracle.route(np.array([[1.0]]), np.array([[0.0], [5.0], [-5.0]]), np.array([0.2, 0.0, 9.0]), 2, 3.0)
    s = oracle.sigmoid(np.array([-5.0, 5.0]))
    assert ids.tolist() == [[2, 1]] and np.allclose(w, s / s.sum() * 3)
    x = oracle.layer_norm(np.array([1.0, 3.0]), np.array([2.0, 2.0]), np.array([0.0, 1.0]), 0.0)
    assert np.allclose(x, [-2, 3])


PLANTS = ["window", "scaling", "length", "temperature", "bucket", "sink", "softcap", "key norm", "bonus", "shift", "decay", "delta order", "unit",
          "beta", "conv state", "state", "shared latents", "correction", "top", "router scale", "mult", "left scale", "rotation", "group"]


@pytest.mark.parametrize("plant", PLANTS)
def test_a_planted_mistake_shows_in_the_logits(plant, monkeypatch):
    """The cases the GPU tests compare on are sharp enough: each of these faults moves the logits far beyond rounding."""
    cfg = cases.uneven()
    w, toks = cases.weights(cfg), cases.tokens(cfg, 120)
    want = oracle.Model(cfg, w).run(toks)
    swap = lambda name, f: monkeypatch.setattr(oracle, name, (lambda real: lambda *a, **k: f(real, *a, **k))(getattr(oracle, name)))
    cfg = json.loads(json.dumps(cfg))
    layers, cut = cfg["layers"], False
    if plant == "window":
        swap("visible", lambda real, q, k, n=None: real(q, k, n + 1 if n else n))
    elif plant == "scaling":
        swap("frequencies", lambda real, b, d, s=None: (real(b, d)[0], real(b, d, s)[1]))
    elif plant == "length":
        swap("frequencies", lambda real, b, d, s=None: (real(b, d, s)[0], 1.0))
    elif plant == "temperature":
        swap("temperature", lambda real, p, c, e: real(p, 0.7 * c, e))
    elif plant == "bucket":
        swap("bucket", lambda real, n, rows, most: real(n + 1, rows, most))
    elif plant == "sink":
        swap("attend", lambda real, s, see, v, sink=None: real(s, see, v))
    elif plant == "softcap":
        layers[2]["mixer"]["left"]["softcap"] = None
    elif plant == "key norm":
        swap("rms", lambda real, x, eps: x if x.shape[1:] == (2, 20) else real(x, eps))
    elif plant == "bonus":
        swap("rwkv_rule", lambda real, r, k, v, d, u, s: real(r, k, v, d, np.ones_like(u), s))
    elif plant == "shift":
        swap("shifted", lambda real, h, last: h)
    elif plant == "decay":
        swap("rwkv_decay", lambda real, m, w1, w2, w0: real(m, w1, 0 * w2, w0))
    elif plant == "delta order":
        def early(real, q, k, v, beta, g, s):  # the read-out misses the current token's write
            out = np.zeros(v.shape)
            for t in range(len(q)):
                out[t] = np.einsum("hd,hde->he", q[t] * g[t], s)
                real(q[t : t + 1], k[t : t + 1], v[t : t + 1], beta[t : t + 1], g[t : t + 1], s)
            return out
        swap("delta_rule", early)
    elif plant == "unit":
        swap("unit", lambda real, x: x)
    elif plant == "beta":
        swap("delta_rule", lambda real, q, k, v, beta, g, s: real(q, k, v, np.ones_like(beta), g, s))
    elif plant == "conv state":
        cut = True
        swap("short_conv", lambda real, x, hist, taps: real(x, 0 * hist, taps))
    elif plant == "state":
        cut = True
        swap("delta_rule", lambda real, q, k, v, beta, g, s: real(q, k, v, beta, g, 0 * s))
    elif plant == "shared latents":
        layers[3]["mixer"]["mask"] = layers[1]["mixer"]["mask"]
    elif plant == "correction":
        swap("route", lambda real, h, r, c, *a: real(h, r, 0 * c, *a))
    elif plant == "top":
        layers[1]["mlp"]["router"]["top"] = 2
    elif plant == "router scale":
        layers[1]["mlp"]["router"]["scale"] = 1.0
    elif plant == "mult":
        cfg["residual_mult"] = 0.7
    elif plant == "left scale":
        layers[2]["mixer"]["left_scale"] = 1.0
    elif plant == "rotation":
        swap("rotate_pairs", lambda real, x, p, f, n=1.0: real(x, np.asarray(p), f[::-1], n))
    else:
        swap("attend", lambda real, s, see, v, sink=None: real(np.roll(s, 1, -1), see, v, sink))
    model = oracle.Model(cfg, w)
    if cut:  # shows when the sequence is cut
        state = model.start()
        got = np.concatenate([model.run(toks[:60], state), model.run(toks[60:], state)])
    else:
        got = model.run(toks)
    assert np.sqrt(((got - want) ** 2).mean()) / want.std() > 0.01


def test_spotlights_show_the_edges():
    """The cases of the GPU tests: what a query may not see does not reach its logits, and what it may see does, by far."""
    for shared in (False, True):
        cfg, w = cases.spotlight(9, shared)
        model = oracle.Model(cfg, w)
        for spot in (2, 11):
            toks = [2 + (i * 7) % 17 for i in range(30)]
            blind = model.run(toks)
            toks[spot] = 1
            seen = np.abs(model.run(toks) - blind).max(-1)
            assert (seen[spot : spot + 9] > 0.1).all() and not seen[:spot].any() and seen[spot + 9 :].max() < 1e-9
    cfg, w = cases.far_key()
    model = oracle.Model(cfg, w)
    toks = [2 + (i * 7) % 17 for i in range(300)]
    blind = model.run(toks)
    toks[5] = 1
    assert (np.abs(model.run(toks) - blind).max(-1)[5:] > 0.1).all()


# -- configuration, names, weights ----------------------------------------------------------------------------------
def test_configuration_and_names(tmp_path):
    from mfq_b200.checkpoint import read_hf_directory
    from mfq_b200.models import registry
    from mfq_b200.models.bufolorn import BufolornConfig, DenseSpec, ExpertsSpec, tensor_shapes
    src = cases.uneven()
    raw, tensors, _ = read_hf_directory(cases.write(tmp_path / "m", src, cases.weights(src)))
    assert registry.find(raw).name == "bufolorn" and raw["vocab_size"] == 150 and raw["num_layers"] == 8
    cfg = BufolornConfig.from_dict(json.loads(json.dumps(raw)))
    assert cfg == BufolornConfig.from_source(src)
    known = tensor_shapes(cfg)
    assert set(tensors) == set(known)
    assert all(tuple(tensors[n].shape) == s for n, s in known.items() if 0 not in s)  # ranks and distance tables are the file's
    assert [l.kind for l in cfg.layers] == [l["type"] for l in src["layers"]]
    lat = cfg.layers[1].mixer
    assert (lat.window, lat.kv_rank, lat.rot_scaling.factor, lat.rot_scaling.original_max_position) == (24, 40, 4.0, 40)
    assert cfg.layers[3].mixer.kv_from == 1 and cfg.layers[5].mixer.rot_scaling is None
    assert cfg.layers[0].mlp == DenseSpec(40) and cfg.layers[4].mlp == ExpertsSpec(5, 1, 0.8, 40, 0) and cfg.layers[2].mlp is None
    assert cfg.layers[6].mixer.left.softcap == 0.0 and cfg.layers[6].mixer.left.temp_every == 5 and cfg.layers[6].mixer.right_scale == 0.7
    assert cfg.owners() == [1, 2, 5, 6] and cfg.kv_shapes() == [(1, 48 + 16, 0), (2, 32, 32), (1, 32 + 32, 0), (1, 48, 32)]
    assert cfg.state_shapes() == {(0, "state"): (3, 32, 32), (0, "conv"): (1, 9 * 32), (2, "state"): (3, 32, 32), (2, "last"): (112,),
                                  (4, "state"): (4, 48, 80), (4, "conv"): (4, 4 * 48 + 4 * 80), (6, "state"): (2, 64, 64), (6, "last"): (112,)}
    assert tensors["model.block.1.mlp.experts.up.weight"].shape == (7, 40, 104)
    plain = cases.config([cases.latent(), cases.parallel()])
    plain["layers"][0]["mixer"]["mask"] = None
    plain["layers"][1]["mixer"]["left"].pop("q_temp")
    cfg = BufolornConfig.from_source(plain)
    assert cfg.layers[0].mixer.window > 10 ** 8 and cfg.layers[1].mixer.left.temp_coef == 0.0


def test_configuration_rejects_what_the_kernels_cannot_run():
    from mfq_b200.models.bufolorn import BufolornConfig
    parse = lambda *layers: BufolornConfig.from_source(cases.config(list(layers)))
    odd = cases.delta()
    odd["type"] = "something"
    with pytest.raises(ValueError, match="unknown mixer"):
        parse(odd)
    with pytest.raises(ValueError, match="unknown feed-forward"):
        parse(cases.delta(mlp={"kind": "routed"}))
    odd = cases.latent()
    odd["mixer"]["rot"]["dims"] = 8
    with pytest.raises(ValueError, match="rotated"):
        parse(odd)
    for broken in (cases.latent(rot=3), cases.latent(rank=600), cases.latent(dim=250), cases.latent(scale=0.0), cases.latent(window=-1),
                   cases.parallel(heads=5), cases.parallel(dim=300), cases.parallel(every=0), cases.delta(heads=3), cases.delta(conv=0),
                   cases.delta(conv=9), cases.delta(dim=600, vdim=400), cases.delta(mlp=cases.moe(top=8)), cases.delta(mlp=cases.dense(0))):
        with pytest.raises(ValueError, match="layer 0"):
            parse(broken)
    for later in (cases.latent(kv_from=0), cases.latent(kv_from=2), cases.latent(kv_from=1, rank=32), cases.latent(kv_from=1, base=5.0), cases.latent(kv_from=3)):
        with pytest.raises(ValueError):
            parse(cases.delta(), cases.latent(), later)
    with pytest.raises(ValueError, match="no latents"):
        parse(cases.latent(), cases.latent(kv_from=0), cases.latent(kv_from=1))


def test_devices_and_extensions_are_refused_clearly(tmp_path):
    from mfq_b200.checkpoint import load_engine
    src = cases.config([cases.latent(), cases.delta()])
    path = cases.write(tmp_path / "m", src, cases.weights(src))
    with pytest.raises(RuntimeError, match="CUDA"):
        load_engine(path, "cpu", max_batch=1, max_seq_len=32)
    with pytest.raises(NotImplementedError, match="single rank"):
        load_engine(path, "cpu", max_batch=1, max_seq_len=32, tp_size=2)


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_weights_as_stored_compute_the_same_products(dtype):
    """The padded, stacked and reordered matrices give the plain products at the places the kernels read them from."""
    from mfq_b200.architectures import to_canonical
    from mfq_b200.models.bufolorn import BufolornConfig, BufolornWeights
    from mfq_b200.ops.dense import up
    src = cases.uneven()
    w = cases.weights(src)
    cfg = BufolornConfig.from_source(src)
    packed = BufolornWeights(cfg, {k: torch.from_numpy(np.asarray(v)) for k, v in to_canonical(w, src).items()}, "cpu", dtype)
    rng = np.random.default_rng(0)
    wide = lambda x, n: np.pad(x, (0, n - len(x)))
    x = rng.standard_normal(cfg.hidden_size)
    xp = wide(x, up(cfg.hidden_size))
    for i, (l, layer) in enumerate(zip(cfg.layers, packed.layers)):
        m, p, n = l.mixer, layer.mixer, f"l{i}.mix."
        plain = lambda name: w[n + name] @ x
        mat = lambda lin: lin.w.double().numpy()
        if l.kind == "latent_attention":
            h, d, r, e, c = m.heads, up(m.dim), up(m.rot_dim), up(m.vdim), up(m.kv_rank)
            got = mat(p.proj) @ xp
            q = got[: h * (d + r)].reshape(h, d + r)
            assert np.allclose(np.concatenate([q[:, : m.dim], q[:, d : d + m.rot_dim]], 1).reshape(-1), plain("q")) and not q[:, m.dim : d].any()
            if m.kv_from is None:
                row = got[h * (d + r) :]
                assert np.allclose(np.concatenate([row[: m.kv_rank], row[c : c + m.rot_dim]]), plain("dkv")) and len(row) == m.row
            else:
                assert p.norm is None and len(got) == h * (d + r)
            lat, key = rng.standard_normal(m.kv_rank), rng.standard_normal(m.rot_dim)
            k, v = (w[n + "uk"] @ lat).reshape(h, m.dim), (w[n + "uv"] @ lat).reshape(h, m.vdim)
            a = mat(p.up.absorb).reshape(h, c, d)
            assert np.allclose(np.einsum("hcd,hd,c->h", a, q[:, :d], wide(lat, c)), (q[:, : m.dim] * k).sum(1))
            assert np.allclose((mat(p.up.value_up) @ wide(lat, c)).reshape(h, e)[:, : m.vdim], v)
            assert (p.up.expand is None) == (dtype == torch.float32)
            if p.up.expand is not None:
                kv = (p.up.expand.double().numpy() @ np.concatenate([wide(lat, c), wide(key, r)])).reshape(h, d + r + e)
                assert np.allclose(kv[:, : m.dim], k) and np.allclose(kv[:, d : d + m.rot_dim], key[None]) and np.allclose(kv[:, d + r : d + r + m.vdim], v)
            y, yp = rng.standard_normal((h, m.vdim)), np.zeros((h, e))
            yp[:, : m.vdim] = y
            assert np.allclose((mat(p.o_proj) @ yp.reshape(-1))[: cfg.hidden_size], w[n + "o"] @ y.reshape(-1))
        elif l.kind == "parallel":
            a, t, dk, dv, d = m.left, m.right, up(m.left.dim), up(m.left.vdim), up(m.right.dim)
            got = mat(p.qkv) @ xp + p.qkv.bias.double().numpy()
            parts = np.split(got, np.cumsum([a.heads * dk, a.kv_heads * dk]))
            for s, part, dim, dp in zip("qkv", parts, (a.dim, a.dim, a.vdim), (dk, dk, dv)):
                assert np.allclose(part.reshape(-1, dp)[:, :dim].reshape(-1), plain("left." + s) + w[n + f"left.{s}.b"], atol=1e-6)
            rel = w[n + "left.rel"]
            for dist in (0, 1, 5, 12, 31, 32, 33, 69, 70, 71, 500):
                assert np.allclose(p.bias.table[:, min(dist, p.bias.last)].numpy(), rel[oracle.bucket(dist, len(rel), a.bias_max)])
            assert np.allclose(p.bias.top.numpy(), p.bias.table.numpy().max(1))
            for s, part in zip("rkvg", mat(p.rkvg).reshape(4, -1, len(xp)) @ xp):
                assert np.allclose(part.reshape(t.heads, d)[:, : t.dim].reshape(-1), plain("right." + s))
            assert np.allclose(p.mu[4, : cfg.hidden_size].numpy(), w[n + "right.mu.w"]) and p.geometry.scale == 1.0
            assert np.allclose(p.bonus.view(t.heads, d)[:, : t.dim].numpy(), w[n + "right.u"])
        else:
            geo = p.geometry
            got = mat(p.proj) @ xp
            assert len(got) == geo.width
            parts = np.split(got, np.cumsum([m.kv_heads * geo.dk, m.kv_heads * geo.dk, m.heads * geo.dv, geo.b_cols, geo.rank_a]))
            for s, part, dim, dp in zip("qkv", parts, (m.dim, m.dim, m.vdim), (geo.dk, geo.dk, geo.dv)):
                assert np.allclose(part.reshape(-1, dp)[:, :dim].reshape(-1), plain(s))
            assert np.allclose(parts[3][: m.heads], plain("b")) and np.allclose(parts[5][: len(w[n + "g1"])], plain("g1"))
            taps = p.rule.conv.numpy()[:, : m.kv_heads * geo.dk].reshape(m.taps, m.kv_heads, geo.dk)[..., : m.dim].reshape(m.taps, -1)
            assert np.allclose(taps.T, w[n + "q.conv"]) and np.allclose(p.rule.rate.numpy(), np.exp(w[n + "A_log"]))
        if l.mlp is not None and hasattr(l.mlp, "experts"):
            bank = layer.mlp.bank
            both = bank.gate_up.double().numpy().reshape(l.mlp.experts, -1, 2, 8, len(xp))
            gate, upw = both[:, :, 0].reshape(l.mlp.experts, -1, len(xp)), both[:, :, 1].reshape(l.mlp.experts, -1, len(xp))
            for e in range(l.mlp.experts):
                assert np.allclose((gate[e] @ xp)[: l.mlp.ff], w[f"l{i}.mlp.e{e}.gate"] @ x) and np.allclose((upw[e] @ xp)[: l.mlp.ff], w[f"l{i}.mlp.e{e}.up"] @ x)
            assert (layer.mlp.shared is None) == (l.mlp.shared == 0)
    assert packed.embed.shape == (150, 112) and packed.lm_head.w.shape == (160, 112)


def test_memory_of_a_deployment_counts_pages_and_state():
    from mfq_b200.models.bufolorn import BufolornConfig
    from mfq_b200.server.analysis import model_memory, model_parameters
    own = BufolornConfig.from_source(cases.uneven())
    cfg = own.to_dict()
    got = model_memory(cfg, 1000, batch=2, context=64)["per_gpu"]
    assert got["kv_cache"] == (2 * 4 + 1) * 16 * 2 * (64 + 2 * 64 + 64 + 80)
    assert got["recurrent_state"] == 2 * own.state_bytes() and own.state_bytes() == 4 * sum(int(np.prod(s)) for s in own.state_shapes().values())
    counts = model_parameters(cfg)
    assert counts["attention_layers"] == 6 and counts["experts"] == 7 and counts["top_k"] == 3
    assert counts["total"] - counts["active_per_token"] == 3 * 104 * 40 * ((7 - 3) + (5 - 1) + (7 - 3))
    assert counts["groups"]["time_mixing"] > 0 and "other" not in counts["groups"]


def test_quantization_keeps_what_is_not_a_projection():
    from mfq_b200.checkpoint import quantize_tensors
    rng = np.random.default_rng(0)
    names = ("model.block.0.linear_attention.query_conv.weight", "model.block.0.time_mixing.bonus", "model.block.0.attention.distance.bias",
             "model.block.0.attention.query.weight")
    out = quantize_tensors({n: rng.standard_normal((64, 64)).astype(np.float32) for n in names}, dense="nint8")
    kinds = [type(out[n]).__name__ for n in names]
    assert kinds[0] == kinds[1] == kinds[2] != kinds[3]


def test_state_with_several_parts_per_layer():
    from mfq_b200.engine.recurrent_state import LayerStates
    s = LayerStates({(1, "state"): (2, 4, 8), (1, "conv"): (0, 6), (5, "last"): (9,)}, 3, "cpu")
    for t in s.tensors:
        t.normal_()
    before, out = s.save(), s.export_slot(2)
    s.reset(1)
    assert not s.layer((1, "state"))[1].any() and not s.layer((5, "last"))[1].any() and torch.equal(s.layer((5, "last"))[2], before[2][2])
    s.import_slot(1, out)
    assert torch.equal(s.layer((5, "last"))[1], before[2][2]) and s.layer((1, "conv")).shape == (3, 0, 6)


def test_pages_without_values_are_exported():
    from mfq_b200.engine.kv_cache import PlainPagedKVCache
    cache = PlainPagedKVCache([(1, 48, 0), (2, 16, 32)], torch.float32, num_pages=5, max_seqs=1, max_pages_per_seq=4, device="cpu")
    for l in cache.pools:
        l.k.normal_(), l.v.normal_()
    blob, want = cache.export_pages([3, 1]), cache.layer(0).k[[3, 1]].clone()
    assert blob.nbytes == cache.page_blob_bytes(2)
    cache.import_pages([2, 4], blob)
    assert torch.equal(cache.layer(0).k[[2, 4]], want) and torch.equal(cache.layer(1).v[4], cache.layer(1).v[1])


@pytest.mark.parametrize("window", [1, 15, 16, 17, 40, 1 << 30])
def test_visible_pages_hold_every_key_of_the_window(window):
    from mfq_b200.ops.latent_attn import visible_pages
    portions = [(0, 5), (31, 2), (100, 40), (16, 16), (63, 1)]
    seq, shift = visible_pages(portions, window)
    for b, (start, count) in enumerate(portions):
        mine = {i - shift[b] for i, s in enumerate(seq) if s == b}
        first = max(0, start - window + 1)
        assert mine == set(range(first // 16, (start + count - 1) // 16 + 1))


@pytest.mark.parametrize("rows,most", [(4, 3), (8, 64), (12, 70), (20, 33), (32, 128.0), (32, 4000)])
def test_distance_buckets(rows, most):
    from mfq_b200.ops.window_attn import DistanceBias, log_buckets
    got = log_buckets(rows, most)
    assert got[-1] == rows - 1 and rows - 1 not in got[:-1]
    assert all((got[n] if n < len(got) else rows - 1) == oracle.bucket(n, rows, most) for n in range(int(2 * most) + 5))
    with pytest.raises(ValueError, match="differ"):
        DistanceBias.from_table(torch.tensor([[0.0, 70.0]]))


def test_frequencies_of_the_table_are_those_of_the_restatement():
    from mfq_b200.models.bufolorn import _yarn
    from mfq_b200.ops.window_attn import rope_table
    for dims, base, sc in ((12, 1e4, cases.SCALING), (64, 5e5, {"factor": 8.0, "original": 2048, "fast": 32.0, "slow": 1.0}),
                           (16, 100.0, {"factor": 3.0, "original": 30, "fast": 2.0, "slow": 1.9})):
        table = rope_table(base, dims, 300, "cpu", _yarn(sc)).double().numpy()
        f, length = oracle.frequencies(base, dims, sc)
        a = np.arange(300)[:, None] * f
        assert np.abs(table[..., 0] - length * np.cos(a)).max() < 1e-6 and np.abs(table[..., 1] - length * np.sin(a)).max() < 1e-6
    from mfq_b200.models.rope_scaling import YarnScaling
    y = YarnScaling(4.0, 512)
    assert np.allclose(y.frequencies(64, 1e4), y.inv_freq(64, 1e4).numpy(), rtol=1e-5)


def test_plans():
    from mfq_b200.ops import delta, dense_moe, latent_attn
    for batch in (1, 3, 16, 64):
        for heads in (1, 4, 32):
            for dk in (16, 48, 80, 128, 256):
                for dv in (16, 48, 80, 128, 256, 512):
                    s = delta.column_split(batch, heads, dk, dv)
                    if s == 0:
                        assert dk * dv > 64 * 1024
                        continue
                    groups = dv // s // 4
                    assert s <= 8 and dv % (4 * s) == 0 and -(-dk // min(dk, 256 // groups)) <= 16
            for keys in (1, 100, 4096, 1 << 30):
                assert 1 <= latent_attn.decode_splits(batch, heads, keys) <= 32
    assert dense_moe.token_tile(40, 8, True) == 64 and dense_moe.token_tile(40, 8, False) == 0 and dense_moe.token_tile(4096, 8, False) == 128
