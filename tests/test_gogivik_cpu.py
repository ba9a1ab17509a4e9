"""Gogivik without a GPU: the plain restatement against itself, configuration and names, weight layout, pages and state."""

import json

import numpy as np
import pytest
import torch

import gogivik_cases as cases
import gogivik_oracle as oracle


# -- the restatement ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("size", [1, 2, 7, 64])
def test_portions_of_the_restatement_agree(size):
    cfg = cases.uneven()
    model, toks = oracle.Model(cfg, cases.weights(cfg)), cases.tokens(cfg, 64)
    want, state = model.run(toks), model.start()
    got = np.concatenate([model.run(toks[a : a + size], state) for a in range(0, 64, size)])
    assert np.abs(got - want).max() < 1e-9


def test_mechanisms_of_the_restatement_by_hand():
    see = oracle.in_window([0, 4], range(6), 3)
    assert [np.flatnonzero(r).tolist() for r in see] == [[0], [2, 3, 4]]
    see = oracle.in_chunk([0, 2, 3, 5], range(8), 3)
    assert [np.flatnonzero(r).tolist() for r in see] == [[0], [0, 1, 2], [3], [3, 4, 5]]
    a = np.array([[[1.0, 0.0, 0.0, 2.0, 5.0]]])
    assert np.allclose(oracle.rotate_pairs(a, [3], [0.1, 0.2]), [[[np.cos(0.3), np.sin(0.3), -2 * np.sin(0.6), 2 * np.cos(0.6), 5.0]]])
    assert np.allclose(oracle.rotate_halves(a, [3], [0.1, 0.2]), [[[np.cos(0.3), -2 * np.sin(0.6), np.sin(0.3), 2 * np.cos(0.6), 5.0]]])
    assert np.allclose(oracle.frequencies(100.0, 4, 4.0), [0.25, 0.025])
    o = oracle.attend(np.array([[0.0, 0.0, 50.0]]), np.array([[True, True, False]]), np.array([[2.0], [4.0], [9.0]]), np.log(2.0))
    assert np.allclose(o, 6 / 4)
    y, hist = oracle.causal_conv(np.array([[1.0], [2.0]]), np.array([[5.0], [7.0]]), np.array([[100.0, 10.0, 1.0]]))
    assert y.reshape(-1).tolist() == [571.0, 712.0] and hist.reshape(-1).tolist() == [1.0, 2.0]
    one, state = (lambda *x: np.array(x, dtype=float).reshape(-1, 1, 1)), np.zeros((1, 1, 1))
    dt = np.array([[0.5], [2.0]])
    out = oracle.state_space(one(10, 7), one(3, 4), one(2, 5), dt, np.log([0.25]), np.array([1.5]), state)
    kept = np.exp(-0.5) * 0.5 * 3 * 10
    assert np.allclose(out.reshape(-1), [2 * 15 + 15, 5 * (kept + 2 * 4 * 7) + 10.5]) and np.isclose(state[0, 0, 0], kept + 56)
    assert np.allclose(oracle.rms_parts(np.array([3.0, 3.0, 0.5, 0.5]), 2, 0.0), 1.0)
    assert np.allclose(oracle.squared_unit(np.array([[2.0]]), np.array([[3.0], [-3.0]]), np.array([[1.0, 1.0]])), 36.0)


PLANTS = ["window", "window early", "chunk", "sink", "factor", "halves for pairs", "pairs for halves", "value rotation", "turn back", "value norm",
          "query norm", "query latent norm", "conv bias", "input conv", "input conv of the feed-forward", "input conv state", "order of the taps",
          "one plus", "skip", "decay", "dt bias", "write before reading", "groups", "norm parts", "gate behind the norm", "conv state", "state",
          "squared", "logit scale", "kv heads", "scale"]


@pytest.mark.parametrize("plant", PLANTS)
def test_a_planted_mistake_shows_in_the_logits(plant, monkeypatch):
    """The cases the GPU tests compare on are sharp enough: each of these faults moves the logits far beyond rounding."""
    cfg = cases.uneven()
    w, toks = cases.weights(cfg), cases.tokens(cfg, 120)
    want = oracle.Model(cfg, w).run(toks)
    swap = lambda name, f: monkeypatch.setattr(oracle, name, (lambda real: lambda *a, **k: f(real, *a, **k))(getattr(oracle, name)))
    cfg, w = json.loads(json.dumps(cfg)), dict(w)
    layers, cut = cfg["layers"], False
    every = lambda ending, f: w.update({n: f(t) for n, t in w.items() if n.endswith(ending)})
    if plant == "window":
        swap("in_window", lambda real, q, k, n: real(q, k, n + 1))
    elif plant == "window early":
        swap("in_window", lambda real, q, k, n: real(q, k, max(1, n - 1)))
    elif plant == "chunk":
        swap("in_chunk", lambda real, q, k, n: real(np.asarray(q) + 1, np.asarray(k) + 1, n))
    elif plant == "sink":
        swap("attend", lambda real, s, see, v, sink=None: real(s, see, v))
    elif plant == "factor":
        swap("frequencies", lambda real, b, d, f=1.0: real(b, d))
    elif plant == "halves for pairs":
        monkeypatch.setattr(oracle, "rotate_pairs", oracle.rotate_halves)
    elif plant == "pairs for halves":
        monkeypatch.setattr(oracle, "rotate_halves", oracle.rotate_pairs)
    elif plant == "value rotation":
        swap("rotate_halves", lambda real, x, p, f: x if x.shape[1:] == (2, 28) else real(x, p, f))
    elif plant == "turn back":
        swap("rotate_halves", lambda real, x, p, f: x if p[-1] < 0 else real(x, p, f))
    elif plant == "value norm":
        swap("rms", lambda real, x, eps: x if x.shape[1:] == (2, 28) else real(x, eps))
    elif plant == "query norm":
        swap("rms", lambda real, x, eps: x if x.shape[1:] == (6, 24) else real(x, eps))
    elif plant == "query latent norm":
        swap("rms", lambda real, x, eps: x if x.shape[1:] == (36,) else real(x, eps))
    elif plant == "conv bias":
        every("conv.b", np.zeros_like)
    elif plant == "input conv":
        every("canon1", np.zeros_like)
    elif plant == "input conv of the feed-forward":
        every("canon2", np.zeros_like)
    elif plant == "input conv state":
        cut = True
        swap("causal_conv", lambda real, x, h, taps: real(x, h if x.shape[1] != 104 else 0 * h, taps))
    elif plant == "order of the taps":
        every("canon1", lambda t: t[:, ::-1])
    elif plant == "one plus":
        every(("norm1", "norm2"), lambda t: t - 1)
    elif plant == "skip":
        every("mix.D", np.zeros_like)
    elif plant == "decay":
        every("A_log", lambda t: t + 0.5)
    elif plant == "dt bias":
        swap("softplus", lambda real, z: real(z + 0.3))
    elif plant == "write before reading":
        def late(real, x, b, c, dt, a_log, d, s):  # the read-out misses the current token's write
            out = np.zeros_like(x)
            for t in range(len(x)):
                keep = np.exp(-np.exp(a_log) * dt[t])
                out[t] = (keep[:, None, None] * s * c[t][:, :, None]).sum(1) + d[:, None] * x[t]
                real(x[t : t + 1], b[t : t + 1], c[t : t + 1], dt[t : t + 1], a_log, d, s)
            return out
        swap("state_space", late)
    elif plant == "groups":
        swap("state_space", lambda real, x, b, c, *a: real(x, np.roll(b, 1, 1), c, *a))
    elif plant == "norm parts":
        layers[1]["mixer"]["norm_groups"] = 6
    elif plant == "gate behind the norm":
        swap("silu", lambda real, z: np.ones_like(z) if z.shape[1] in (72, 200, 144) else real(z))
    elif plant == "conv state":
        cut = True
        swap("causal_conv", lambda real, x, h, taps: real(x, h if x.shape[1] == 104 else 0 * h, taps))
    elif plant == "state":
        cut = True
        swap("state_space", lambda real, x, b, c, dt, a, d, s: real(x, b, c, dt, a, d, 0 * s))
    elif plant == "squared":
        swap("squared_unit", lambda real, h, up, down: np.maximum(h @ up.T, 0) @ down.T)
    elif plant == "logit scale":
        cfg["logit_scale"] = 1.0
    elif plant == "kv heads":
        swap("attend", lambda real, s, see, v, sink=None: real(np.roll(s, 1, -1), see, v, sink))
    else:
        layers[0]["mixer"]["scale"] = layers[0]["mixer"]["dim"] ** -0.5
    model = oracle.Model(cfg, w)
    if cut:  # shows when the sequence is cut
        state = model.start()
        got = np.concatenate([model.run(toks[:60], state), model.run(toks[60:], state)])
    else:
        got = model.run(toks)
    assert np.sqrt(((got - want) ** 2).mean()) / want.std() > 0.01


def test_spotlights_show_the_edges():
    """The cases of the GPU tests: what a query may not see does not reach its logits, and what it may see does, by far."""
    for make, last in ((cases.window_spotlight, lambda spot: spot + 8), (cases.chunk_spotlight, lambda spot: spot // 9 * 9 + 8)):
        cfg, w = make(9)
        model = oracle.Model(cfg, w)
        for spot in (2, 8, 9, 12):
            toks = [2 + (i * 7) % 17 for i in range(30)]
            blind = model.run(toks)
            toks[spot] = 1
            seen = np.abs(model.run(toks) - blind).max(-1)
            assert (seen[spot : last(spot) + 1] > 0.1).all() and not seen[:spot].any() and seen[last(spot) + 1 :].max() < 1e-9


# -- configuration, names, weights ----------------------------------------------------------------------------------
def test_configuration_and_names(tmp_path):
    from mfq_b200.checkpoint import read_hf_directory
    from mfq_b200.models import registry
    from mfq_b200.models.gogivik import GogivikConfig, tensor_shapes
    from mfq_b200.ops.window_attn import LinearScaling
    src = cases.uneven()
    raw, tensors, _ = read_hf_directory(cases.write(tmp_path / "m", src, cases.weights(src)))
    assert registry.find(raw).name == "gogivik" and raw["vocab_size"] == 150 and raw["num_layers"] == 9
    cfg = GogivikConfig.from_dict(json.loads(json.dumps(raw)))
    assert cfg == GogivikConfig.from_source(src) and (cfg.conv_taps, cfg.logit_scale, cfg.norm_eps) == (4, 0.7, 1e-4)
    known = tensor_shapes(cfg)
    assert {n: tuple(t.shape) for n, t in tensors.items()} == known and len(known) == len(cases.shapes(src))
    assert [l.kind for l in cfg.layers] == [l["type"] for l in src["layers"]]
    lat, chu, sta = cfg.layers[3].mixer, cfg.layers[0].mixer, cfg.layers[1].mixer
    assert (lat.window, lat.q_rank, lat.kv_rank, lat.rot_dim, lat.rot_base) == (17, 70, 24, 20, 500.0)
    assert (chu.chunk, chu.rotation, chu.value_rotation) == (21, (300.0, 16, LinearScaling(2.5)), (300.0, 28))
    assert (sta.groups, sta.state, sta.taps, sta.norm_groups) == (3, 20, 2, 4)
    assert [l.ff for l in cfg.layers] == [40, 72, 56, 0, 0, 0, 24, 32, 24]
    assert cfg.owners() == [0, 2, 3, 5, 6, 8]
    assert cfg.kv_shapes() == [(2, 32, 32), (1, 48 + 16, 0), (1, 32 + 32, 0), (1, 48, 32), (3, 32, 48), (1, 80 + 16, 0)]
    states = cfg.state_shapes()
    assert states[0, "input"] == states[6, "mlp_input"] == (3, 112) and (3, "mlp_input") not in states
    assert states[1, "state"] == (6, 32, 16) and states[1, "conv"] == (1, 6 * 16 + 2 * 3 * 32) and states[7, "conv"] == (0, 2 * 80 + 4 * 16)
    assert cfg.key_spans() == [(2, 21, 0), (1, 50, 0), (3, 7, 0)]
    bare = cases.config([cases.latent(), cases.chunked()])
    for l in bare["layers"]:
        l["mixer"].pop("mask")
    bare["layers"][1]["mixer"]["rot"].pop("scaling")
    cfg = GogivikConfig.from_source(bare)
    assert cfg.layers[0].mixer.window > 10 ** 8 and cfg.layers[1].mixer.chunk > 10 ** 8 and cfg.layers[1].mixer.rot_factor == 1.0


def test_configuration_rejects_what_the_kernels_cannot_run():
    from mfq_b200.models.gogivik import GogivikConfig
    parse = lambda *layers, **kw: GogivikConfig.from_source(cases.config(list(layers), **kw))
    odd = cases.mamba()
    odd["type"] = "something"
    with pytest.raises(ValueError, match="unknown mixer"):
        parse(odd)
    with pytest.raises(ValueError, match="unknown feed-forward"):
        parse(cases.mamba(mlp={"kind": "routed"}))
    odd = cases.latent()
    odd["mixer"]["rot"]["dims"] = 8
    with pytest.raises(ValueError, match="rotated"):
        parse(odd)
    for broken in (cases.latent(rot=3), cases.latent(rank=600), cases.latent(dim=250), cases.latent(scale=0.0), cases.latent(window=-1), cases.latent(q_rank=0),
                   cases.chunked(heads=5), cases.chunked(dim=300), cases.chunked(vdim=27), cases.chunked(rot=40), cases.chunked(rot=5), cases.chunked(size=-3),
                   cases.chunked(factor=0.0), cases.mamba(heads=3), cases.mamba(conv=0), cases.mamba(conv=9), cases.mamba(norm_groups=3),
                   cases.mamba(state=8000, vdim=400), cases.mamba(mlp=cases.dense(-1))):
        with pytest.raises(ValueError, match="layer 0"):
            parse(broken)
    with pytest.raises(ValueError, match="taps"):
        parse(cases.mamba(), taps=9)


def test_devices_and_extensions_are_refused_clearly(tmp_path):
    from mfq_b200.checkpoint import load_engine
    src = cases.config([cases.latent(), cases.mamba()])
    path = cases.write(tmp_path / "m", src, cases.weights(src))
    with pytest.raises(RuntimeError, match="CUDA"):
        load_engine(path, "cpu", max_batch=1, max_seq_len=32)
    with pytest.raises(NotImplementedError, match="single rank"):
        load_engine(path, "cpu", max_batch=1, max_seq_len=32, tp_size=2)


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_weights_as_stored_compute_the_same_products(dtype):
    """The padded, stacked and reordered matrices give the plain products at the places the kernels read them from."""
    from mfq_b200.architectures import to_canonical
    from mfq_b200.models.gogivik import GogivikConfig, GogivikWeights
    from mfq_b200.ops.dense import up
    src = cases.uneven()
    w = cases.weights(src)
    cfg = GogivikConfig.from_source(src)
    packed = GogivikWeights(cfg, {k: torch.from_numpy(np.asarray(v)) for k, v in to_canonical(w, src).items()}, "cpu", dtype)
    rng = np.random.default_rng(2)
    wide = lambda v, n: np.concatenate([v, np.zeros(n - len(v))])
    x = rng.standard_normal(cfg.hidden_size)
    xp = wide(x, up(cfg.hidden_size))
    mat = lambda lin: lin.w.double().numpy()
    for i, (l, layer) in enumerate(zip(cfg.layers, packed.layers)):
        m, p, n = l.mixer, layer.mixer, f"l{i}.mix."
        plain = lambda name: w[n + name] @ x
        e = up(m.vdim)
        if l.kind == "latent_attention":
            h, d, r, a, c = m.heads, up(m.dim), up(m.rot_dim), up(m.q_rank), up(m.kv_rank)
            low, row = np.split(mat(p.down) @ xp, [a])
            assert np.allclose(low[: m.q_rank], plain("dq")) and not low[m.q_rank :].any()
            assert np.allclose(np.concatenate([row[: m.kv_rank], row[c : c + m.rot_dim]]), plain("dkv")) and len(row) == m.row
            q = (mat(p.query) @ low).reshape(h, d + r)
            assert np.allclose(np.concatenate([q[:, : m.dim], q[:, d : d + m.rot_dim]], 1).reshape(-1), w[n + "uq"] @ plain("dq")) and not q[:, m.dim : d].any()
            lat = rng.standard_normal(m.kv_rank)
            k, v = (w[n + "uk"] @ lat).reshape(h, m.dim), (w[n + "uv"] @ lat).reshape(h, m.vdim)
            assert np.allclose(np.einsum("hcd,hd,c->h", mat(p.up.absorb).reshape(h, c, d), q[:, :d], wide(lat, c)), (q[:, : m.dim] * k).sum(1))
            assert np.allclose((mat(p.up.value_up) @ wide(lat, c)).reshape(h, e)[:, : m.vdim], v) and np.allclose(p.sink.numpy(), w[n + "sink"])
        elif l.kind == "attention":
            parts = np.split(mat(p.qkv) @ xp, np.cumsum([m.heads * up(m.dim), m.kv_heads * up(m.dim)]))
            for s, part, dim in zip("qkv", parts, (m.dim, m.dim, m.vdim)):
                assert np.allclose(part.reshape(-1, up(dim))[:, :dim].reshape(-1), plain(s))
            assert np.allclose(p.k_norm.numpy()[: m.dim], w[n + "k.norm"])
        else:
            geo, got, inner, side = p.geometry, mat(p.proj) @ xp, m.heads * m.vdim, m.groups * m.state
            assert len(got) == geo.row and geo.channels == p.rule.conv.shape[1]
            z, xs, b, c, dt = np.split(plain("in"), np.cumsum([inner, inner, side, side]))
            parts = np.split(got, np.cumsum([m.heads * e, m.groups * geo.state, m.groups * geo.state, m.heads * e]))
            trim = lambda t, d: t.reshape(-1, up(d))[:, :d].reshape(-1)
            assert all(np.allclose(trim(a, d), t) for a, d, t in zip(parts, (m.vdim, m.state, m.state, m.vdim), (xs, b, c, z)))
            assert np.allclose(parts[4][: m.heads], dt)
            for j in range(m.taps):
                rows = np.split(p.rule.conv.numpy()[j], np.cumsum([m.heads * e, m.groups * geo.state]))
                assert np.allclose(np.concatenate([trim(a, d) for a, d in zip(rows, (m.vdim, m.state, m.state))]), w[n + "conv"][:, j])
            assert np.allclose(trim(p.rule.norm.numpy(), m.vdim), w[n + "norm"]) and np.allclose(p.rule.rate.numpy(), np.exp(w[n + "A_log"]))
            assert np.allclose(p.rule.skip.numpy(), w[n + "D"]) and p.rule.norm.numel() == m.heads * e
        y = rng.standard_normal((m.heads, m.vdim))
        assert np.allclose((mat(p.o_proj) @ np.stack([wide(r, e) for r in y]).reshape(-1))[: cfg.hidden_size], w[n + "o"] @ y.reshape(-1))
        assert np.allclose(layer.input.norm.numpy(), wide(1 + w[f"l{i}.norm1"], 112)) and np.allclose(layer.input.conv.numpy()[:, :104].T, w[f"l{i}.canon1"])
        assert (layer.up is None) == (l.ff == 0)
        if l.ff:
            assert layer.up.act == "relu2" and np.allclose((mat(layer.up) @ xp)[: l.ff], w[f"l{i}.mlp.up"] @ x)
            assert np.allclose(layer.mlp_input.conv.numpy()[:, :104].T, w[f"l{i}.canon2"])
    assert np.allclose(packed.final_norm.numpy()[:104], 0.7 * (1 + w["final.norm"])) and packed.lm_head.w.shape == (160, 112)


def test_memory_of_a_deployment_counts_pages_and_state():
    from mfq_b200.models.gogivik import GogivikConfig
    from mfq_b200.server.analysis import model_memory, model_parameters
    own = GogivikConfig.from_source(cases.uneven())
    cfg = own.to_dict()
    got = model_memory(cfg, 1000, batch=2, context=64)["per_gpu"]
    assert got["kv_cache"] == (2 * 4 + 1) * 16 * 2 * (2 * 64 + 64 + 64 + 80 + 3 * 80 + 96)
    assert got["recurrent_state"] == 2 * own.state_bytes() and own.state_bytes() == 4 * sum(int(np.prod(s)) for s in own.state_shapes().values())
    counts = model_parameters(cfg)
    assert counts["attention_layers"] == 6 and counts["experts"] is None and counts["total"] == own.param_count() == counts["active_per_token"]
    assert counts["groups"]["linear_attention"] > 0 and "other" not in counts["groups"]


def test_quantization_keeps_what_is_not_a_projection():
    from mfq_b200.checkpoint import quantize_tensors
    rng = np.random.default_rng(0)
    names = ("model.block.0.attention.input_conv.weight", "model.block.0.linear_attention.in_conv.weight", "model.block.0.linear_attention.in.weight")
    out = quantize_tensors({n: rng.standard_normal((64, 64)).astype(np.float32) for n in names}, dense="nint8")
    kinds = [type(out[n]).__name__ for n in names]
    assert kinds[0] == kinds[1] != kinds[2]


def test_frequencies_of_the_table_are_those_of_the_restatement():
    from mfq_b200.ops.window_attn import LinearScaling, rope_table
    for dims, base, factor in ((12, 1e4, 4.0), (64, 5e5, 1.0), (2, 100.0, 3.0)):
        table = rope_table(base, dims, 300, "cpu", LinearScaling(factor)).double().numpy()
        a = np.arange(300)[:, None] * oracle.frequencies(base, dims, factor)
        assert np.abs(table[..., 0] - np.cos(a)).max() < 1e-6 and np.abs(table[..., 1] - np.sin(a)).max() < 1e-6


def test_plans():
    from mfq_b200.ops import ssd
    for batch in (1, 3, 16, 64):
        for heads in (1, 6, 64):
            for n in (16, 48, 128, 256, 512):
                for p in (16, 48, 64, 80, 128, 256):
                    s = ssd.column_split(batch, heads, n, p)
                    if s == 0:
                        assert n * p > 64 * 1024
                        continue
                    assert p % (4 * s) == 0 and -(-n // min(n, 256 // (p // s // 4))) <= 16
    for heads, groups, n, p in ((6, 2, 32, 32), (64, 1, 128, 64), (80, 8, 256, 64), (7, 7, 16, 48), (4, 1, 512, 128)):
        geo = ssd.Geometry(heads, groups, n, p, p, 4, 1, 1e-5)
        for tokens, longest in ((20, 20), (65, 65), (4096, 4096), (8192, 64)):
            chunk, per = ssd.chunk_plan(geo, tokens, longest)
            assert chunk in (64, 128) and (heads // groups) % per == 0 and (chunk == 64 or geo.chunk_fits(128, per))
