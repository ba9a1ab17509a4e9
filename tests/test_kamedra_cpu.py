"""Kamedra without a GPU: the plain restatement against itself, configuration and names, weight layout, pages and state."""

import json

import numpy as np
import pytest
import torch

import kamedra_cases as cases
import kamedra_oracle as oracle


# -- the restatement ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("size", [1, 2, 7, 64])
def test_portions_of_the_restatement_agree(size):
    cfg = cases.uneven()
    model, toks = oracle.Model(cfg, cases.weights(cfg)), cases.tokens(cfg, 64)
    want, state = model.run(toks), model.start()
    got = np.concatenate([model.run(toks[a : a + size], state) for a in range(0, 64, size)])
    assert np.abs(got - want).max() < 1e-9


def test_mechanisms_of_the_restatement_by_hand():
    see = oracle.visible([0, 4, 5, 9], range(10), 3, 2)
    assert [np.flatnonzero(r).tolist() for r in see] == [[0], [0, 1, 2, 3, 4], [0, 1, 3, 4, 5], [0, 1, 7, 8, 9]]
    assert np.allclose(oracle.rotate_pairs(np.array([[[1.0, 0.0, 5.0]]]), [3], [0.1]), [[[np.cos(0.3), np.sin(0.3), 5.0]]])
    f = oracle.frequencies(100.0, 4)
    assert np.allclose(f, [1.0, 0.1])
    turns = 2 * np.pi
    scaled = lambda original: oracle.frequencies(1.0, 2, {"factor": 4.0, "low": 1.0, "high": 3.0, "original": original * turns})[0]
    assert scaled(0.5) == 0.25 and scaled(4.0) == 1.0 and np.isclose(scaled(2.0), 0.5 * 0.25 + 0.5)
    lam = oracle.mixing_weight(np.array([1.0, 2.0]), np.array([0.5, 0.0]), np.array([0.0]), np.array([9.0]), 0.3)
    assert np.isclose(lam, np.exp(0.5) - 1 + 0.3)
    o = oracle.difference(np.array([3.0, 1.0]), np.array([2.0, 2.0]), 0.5, 0.25, 0.0)
    assert np.allclose(o, np.array([2.0, 0.0]) / np.sqrt(2) * 0.75)
    state = np.zeros((1, 1, 1))
    one = lambda *x: np.array(x).reshape(-1, 1, 1)
    out = oracle.gated_linear_attention(one(1.0, 2.0), one(3.0, 5.0), one(7.0, 11.0), one(0.5, 0.25), state)
    assert out.reshape(-1).tolist() == [21.0, 2 * (0.25 * 21 + 55)] and state[0, 0, 0] == 60.25
    z = oracle.key_decay(np.ones((1, 1)), np.ones((1, 1)), np.full((1, 1), 2.0), np.array([-2.0]), 4.0)
    assert np.isclose(z[0, 0], 0.5 ** 0.25)


@pytest.mark.parametrize("plant", ["window", "keep", "lambda", "second map", "group", "pairs", "scaling", "decay", "state", "shared", "cap"])
def test_a_planted_mistake_shows_in_the_logits(plant, monkeypatch):
    """The cases the GPU tests compare on are sharp enough: each of these faults moves the logits far beyond rounding."""
    cfg = cases.uneven()
    w, toks = cases.weights(cfg), cases.tokens(cfg, 120)
    want = oracle.Model(cfg, w).run(toks)
    see = oracle.visible
    if plant == "window":
        monkeypatch.setattr(oracle, "visible", lambda q, k, n, keep: see(q, k, n + 1, keep))
    elif plant == "keep":
        monkeypatch.setattr(oracle, "visible", lambda q, k, n, keep: see(q, k, n, keep + 1))
    elif plant == "lambda":
        monkeypatch.setattr(oracle, "mixing_weight", lambda a, b, c, d, diff: diff)
    elif plant == "second map":
        real = oracle.difference
        monkeypatch.setattr(oracle, "difference", lambda a1, a2, *a: real(a2, a1, *a))
    elif plant == "group":
        real = oracle.differential_attention
        monkeypatch.setattr(oracle, "differential_attention", lambda q, k, v, *a: real(np.roll(q, 1, 1), k, v, *a))
    elif plant == "pairs":
        def halves(x, pos, freq):
            n = len(freq)
            order = np.r_[np.arange(2 * n).reshape(2, n).T.reshape(-1), np.arange(2 * n, x.shape[-1])]
            back = np.argsort(order)
            return real(x[..., order], pos, freq)[..., back]
        real = oracle.rotate_pairs
        monkeypatch.setattr(oracle, "rotate_pairs", halves)
    elif plant == "scaling":
        real = oracle.frequencies
        monkeypatch.setattr(oracle, "frequencies", lambda b, d, s=None: real(b, d))
    elif plant == "decay":
        real = oracle.key_decay
        monkeypatch.setattr(oracle, "key_decay", lambda h, a, b, bias, tau: real(h, a, b, bias, 1.0))
    elif plant == "state":
        real = oracle.gated_linear_attention
        monkeypatch.setattr(oracle, "gated_linear_attention", lambda q, k, v, a, s: real(q, k, v, a, np.zeros_like(s)))
    elif plant == "shared":
        cfg = json.loads(json.dumps(cfg))
        cfg["layers"][5]["mixer"]["mask"] = cfg["layers"][3]["mixer"]["mask"]
    else:
        cfg = {**cfg, "logit_softcap": None}
    model = oracle.Model(cfg, w)
    if plant == "state":  # shows when the sequence is cut
        state = model.start()
        got = np.concatenate([model.run(toks[:60], state), model.run(toks[60:], state)])
    else:
        got = model.run(toks)
    assert np.sqrt(((got - want) ** 2).mean()) / want.std() > 0.01


# -- configuration, names, weights ----------------------------------------------------------------------------------
def test_configuration_and_names(tmp_path):
    from mfq_b200.checkpoint import read_hf_directory
    from mfq_b200.models import registry
    from mfq_b200.models.kamedra import KamedraConfig, tensor_shapes
    src = cases.uneven()
    raw, tensors, _ = read_hf_directory(cases.write(tmp_path / "m", src, cases.weights(src)))
    assert registry.find(raw).name == "kamedra" and raw["vocab_size"] == 150 and raw["num_layers"] == 7
    cfg = KamedraConfig.from_dict(json.loads(json.dumps(raw)))
    assert cfg == KamedraConfig.from_source(src)
    known = tensor_shapes(cfg)
    assert set(tensors) == set(known)
    assert all(tuple(tensors[n].shape) == s for n, s in known.items() if ".decay_a" not in n and ".decay_b.w" not in n)  # ranks are the file's
    att = cfg.layers[1].mixer
    assert (att.window, att.keep, att.rot_scaling.original, att.diff) == (17, 5, 96, 0.3) and cfg.layers[4].mixer.tau == 1.0
    assert [l.ff for l in cfg.layers] == [0, 72, 0, 40, 56, 0, 0] and cfg.layers[5].mixer.kv_from == 3 and cfg.logit_softcap == 12.0
    assert cfg.owners() == [1, 3, 6] and cfg.kv_shapes() == [(2, 64, 32), (1, 96, 80), (1, 32, 16)]
    assert cfg.state_shapes() == {0: (3, 32, 48), 4: (2, 48, 112)}
    plain = cases.config([cases.attention()])
    plain["layers"][0]["mixer"].update(rot=None, mask={})
    plain["logit_softcap"] = None
    cfg = KamedraConfig.from_source(plain)
    assert cfg.layers[0].mixer.rot_dims == 0 and cfg.layers[0].mixer.keep == 0 and cfg.logit_softcap == 0.0
    assert cfg.layers[0].mixer.window > 10 ** 8


def test_configuration_rejects_what_the_kernels_cannot_run():
    from mfq_b200.models.kamedra import KamedraConfig
    parse = lambda *layers: KamedraConfig.from_source(cases.config(list(layers)))
    odd = cases.attention()
    odd["type"] = "something"
    with pytest.raises(ValueError, match="unknown mixer"):
        parse(odd)
    odd = cases.attention()
    odd["mlp"]["kind"] = "routed"
    with pytest.raises(ValueError, match="unknown feed-forward"):
        parse(odd)
    for broken in (cases.attention(heads=5), cases.attention(dim=300), cases.attention(rot=40), cases.attention(rot=3), cases.attention(scale=0.0),
                   cases.attention(window=-1), cases.gla(tau=0.0), cases.gla(heads=0)):
        with pytest.raises(ValueError):
            parse(broken)
    for later in (cases.attention(kv_from=0), cases.attention(kv_from=2), cases.attention(kv_from=1, vdim=32), cases.attention(kv_from=3)):
        with pytest.raises(ValueError):
            parse(cases.gla(), cases.attention(), later)
    with pytest.raises(ValueError, match="no keys"):
        parse(cases.attention(), cases.attention(kv_from=0), cases.attention(kv_from=1))


def test_devices_and_extensions_are_refused_clearly(tmp_path):
    from mfq_b200.checkpoint import load_engine
    src = cases.config([cases.attention(), cases.gla()])
    path = cases.write(tmp_path / "m", src, cases.weights(src))
    with pytest.raises(RuntimeError, match="CUDA"):
        load_engine(path, "cpu", max_batch=1, max_seq_len=32)
    with pytest.raises(ValueError, match="context extension"):
        load_engine(path, "cpu", max_batch=1, max_seq_len=32, yarn_context_extension=2.0)
    with pytest.raises(NotImplementedError, match="single rank"):
        load_engine(path, "cpu", max_batch=1, max_seq_len=32, tp_size=2)


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_weights_as_stored_compute_the_same_products(dtype):
    """The padded, stacked and reordered matrices give the plain products at the places the kernels read them from."""
    from mfq_b200.architectures import to_canonical
    from mfq_b200.models.kamedra import KamedraConfig, KamedraWeights
    from mfq_b200.ops.dense import up
    src = cases.uneven()
    w = cases.weights(src)
    cfg = KamedraConfig.from_source(src)
    packed = KamedraWeights(cfg, {k: torch.from_numpy(np.asarray(v)) for k, v in to_canonical(w, src).items()}, "cpu", dtype)
    x = np.random.default_rng(0).standard_normal(cfg.hidden_size)
    xp = np.zeros(up(cfg.hidden_size))
    xp[: cfg.hidden_size] = x
    for i, (l, layer) in enumerate(zip(cfg.layers, packed.layers)):
        m, p, n = l.mixer, layer.mixer, f"l{i}.mix."
        dk, dv = up(m.dim), up(m.vdim)
        plain = lambda name: w[n + name] @ x
        if l.linear:
            got = p.proj.w.double().numpy() @ xp
            parts = np.split(got, np.cumsum([m.heads * dk, m.heads * dk, m.heads * dv, m.heads * dv]))
            for name, part, d, dp in zip("qkvg", parts, (m.dim, m.dim, m.vdim, m.vdim), (dk, dk, dv, dv)):
                part = part.reshape(m.heads, dp)
                assert np.allclose(part[:, :d].reshape(-1), plain(name)) and not part[:, d:].any()
            rank = w[n + "a1"].shape[0]
            assert p.geometry.rank == up(rank) and np.allclose(parts[4][:rank], plain("a1")) and not parts[4][rank:].any()
            z = (p.decay_b.double().numpy() @ parts[4] + p.decay_bias.double().numpy()).reshape(m.heads, dk)
            assert np.allclose(z[:, : m.dim].reshape(-1), w[n + "a2"] @ plain("a1") + w[n + "a2.b"], atol=1e-5) and not z[:, m.dim :].any()
        else:
            got = p.qkv.w.double().numpy() @ xp
            g, per = m.kv_heads, m.heads // m.kv_heads
            q = got[: 2 * m.heads * dk].reshape(g, 2, per, dk).transpose(0, 2, 1, 3)[..., : m.dim]
            assert np.allclose(q.reshape(-1), plain("q"))
            if m.kv_from is None:
                k, v = np.split(got[2 * m.heads * dk :], [2 * g * dk])
                assert np.allclose(k.reshape(-1, dk)[:, : m.dim].reshape(-1), plain("k")) and np.allclose(v.reshape(g, dv)[:, : m.vdim].reshape(-1), plain("v"))
            else:
                assert p.qkv.w.shape[0] == 2 * m.heads * dk
            lam = oracle.mixing_weight(*(w[n + k] for k in ("lq1", "lk1", "lq2", "lk2")), m.diff)
            assert np.isclose(p.difference.weight, lam, rtol=1e-5) and np.isclose(p.difference.scale, 1 - m.diff)
        y = np.random.default_rng(1).standard_normal(m.heads * m.vdim)
        yp = np.zeros((m.heads, dv))
        yp[:, : m.vdim] = y.reshape(m.heads, m.vdim)
        assert np.allclose((p.o_proj.w.double().numpy() @ yp.reshape(-1))[: cfg.hidden_size], w[n + "o"] @ y)
        assert (layer.gate_up is None) == (l.ff == 0) and np.allclose(layer.norm[: cfg.hidden_size].numpy(), w[f"l{i}.norm1"])
    assert packed.embed.shape == (160, 112) and packed.lm_head.w is packed.embed


def test_memory_of_a_deployment_counts_pages_and_state():
    from mfq_b200.models.kamedra import KamedraConfig
    from mfq_b200.server.analysis import model_memory, model_parameters
    cfg = KamedraConfig.from_source(cases.uneven()).to_dict()
    got = model_memory(cfg, 1000, batch=2, context=64)["per_gpu"]
    assert got["kv_cache"] == (2 * 4 + 1) * 16 * 2 * (2 * (64 + 32) + 96 + 80 + 32 + 16)
    assert got["recurrent_state"] == 2 * 4 * (3 * 32 * 48 + 2 * 48 * 112)
    counts = model_parameters(cfg)
    assert counts["attention_layers"] == 5 and counts["groups"]["dense_mlp"] == 3 * 104 * (72 + 40 + 56) + 3 * 104
    assert counts["groups"]["embeddings"] == 150 * 104 and "head" not in counts["groups"]


def test_budget_sets_the_state_aside_and_takes_models_without_pages():
    from mfq_b200.engine.kv_budget import plan
    how = dict(layers=0, kv_heads=1, head_dim=1, max_batch=4, max_seq_len=64)
    assert plan(budget_bytes=10_000, token_bytes=0, state_bytes_per_row=1000, **how).num_pages == 17
    assert plan(budget_bytes=4000 + 6 * 160, token_bytes=10, state_bytes_per_row=1000, **how).num_pages == 6
    with pytest.raises(MemoryError):
        plan(budget_bytes=3000, token_bytes=0, state_bytes_per_row=1000, **how)


def test_state_slots_are_zeroed_saved_and_moved():
    from mfq_b200.engine.recurrent_state import LayerStates
    s = LayerStates({1: (2, 4, 8), 5: (3, 4, 4)}, 3, "cpu")
    for t in s.tensors:
        t.normal_()
    assert s.layer(5).shape == (3, 3, 4, 4) and s.bytes_per_slot() == 4 * (64 + 48)
    before, out = s.save(), s.export_slot(2)
    s.reset(1)
    assert not s.layer(1)[1].any() and torch.equal(s.layer(1)[2], before[0][2])
    s.import_slot(1, out)
    assert torch.equal(s.layer(5)[1], before[1][2])
    s.load(before)
    assert all(torch.equal(a, b) for a, b in zip(s.tensors, before))


def test_frequencies_of_the_table_are_those_of_the_restatement():
    from mfq_b200.ops.window_attn import FrequencyScaling, rope_table
    sc = cases.SCALING
    scaling = FrequencyScaling(sc["factor"], sc["low"], sc["high"], sc["original"])
    table = rope_table(1e4, 24, 300, "cpu", scaling).double().numpy()
    a = np.arange(300)[:, None] * oracle.frequencies(1e4, 24, sc)
    assert np.abs(table[..., 0] - np.cos(a)).max() < 1e-6 and np.abs(table[..., 1] - np.sin(a)).max() < 1e-6


def test_spotlights_show_the_edges():
    """The cases of the GPU tests: what a query may not see does not reach its logits, and what it may see does, by far."""
    for shared in (False, True):
        cfg, w = cases.spotlight(9, 4, shared)
        model = oracle.Model(cfg, w)
        for spot, last in ((2, None), (3, None), (4, 12), (11, 19)):
            toks = [2 + (i * 7) % 17 for i in range(30)]
            blind = model.run(toks)
            toks[spot] = 1
            seen = np.abs(model.run(toks) - blind).max(-1)
            assert (seen[spot : (last or 29) + 1] > 0.1).all() and not seen[:spot].any()
            assert last is None or seen[last + 1 :].max() < 1e-9


def test_plan_of_column_splits():
    from mfq_b200.ops.gla import _split
    for batch in (1, 3, 16, 64):
        for heads in (1, 4, 16):
            for dv in (16, 48, 80, 128, 256, 512):
                s = _split(batch, heads, dv)
                assert 1 <= s <= 8 and dv % (4 * s) == 0 and (s == 1 or batch * heads * s <= 148)
