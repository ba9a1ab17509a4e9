"""Tepetar without a GPU: the plain restatement against itself, configuration and names, weight layout, unquantized pages,
mixed batches of the scheduler, and trace replay on a stand-in engine."""

import io
import json

import numpy as np
import pytest
import torch

import tepetar_cases as cases
import tepetar_oracle as oracle


# -- the restatement ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("size", [1, 2, 7, 64])
def test_portions_of_the_restatement_agree(size):
    cfg = cases.uneven()
    model, toks = oracle.Model(cfg, cases.weights(cfg)), cases.tokens(cfg, 64)
    want, state = model.run(toks), model.start()
    got = np.concatenate([model.run(toks[a : a + size], state) for a in range(0, 64, size)])
    assert np.abs(got - want).max() < 1e-9


def test_attention_of_the_restatement_by_hand():
    q, k = np.array([[[2.0]], [[1.0]]]), np.array([[[1.0]], [[3.0]]])
    v = np.array([[[10.0]], [[20.0]]])
    out = oracle.attend(q, k, v, [0, 1], [0, 1], 0.5, 4.0, 2)
    s = 4 * np.tanh(np.array([0.5, 1.5]) / 4)
    p = np.exp(s) / np.exp(s).sum()
    assert out[0, 0, 0] == 10.0 and np.isclose(out[1, 0, 0], p @ [10.0, 20.0])
    assert oracle.attend(q, k, v, [0, 1], [0, 1], 0.5, 4.0, 1)[1, 0, 0] == 20.0  # a window of one token sees itself
    assert np.allclose(oracle.rotate(np.array([[[1.0, 0.0, 5.0]]]), [3], 100.0, 2), [[[np.cos(3), np.sin(3), 5.0]]])
    assert np.allclose(oracle.clipped_glu(np.array([9.0, -9.0]), np.array([-9.0, 9.0]), 2.0),
                       [2 / (1 + np.exp(-3.404)) * -1, -9 / (1 + np.exp(1.702 * 9)) * 3])


@pytest.mark.parametrize("plant", ["window", "lambda", "first", "cap", "group", "norm", "side", "clamp"])
def test_a_planted_mistake_shows_in_the_logits(plant, monkeypatch):
    """The cases the GPU tests compare on are sharp enough: each of these faults moves the logits far beyond rounding."""
    cfg = cases.uneven()
    w, toks = cases.weights(cfg), cases.tokens(cfg, 120)
    want = oracle.Model(cfg, w).run(toks)
    if plant == "window":
        monkeypatch.setattr(oracle, "visible", lambda q, k, n: (lambda d: (d >= 0) & (d <= n))(np.asarray(q)[:, None] - np.asarray(k)[None]))
    elif plant == "lambda":
        monkeypatch.setattr(oracle, "mix_values", lambda v, f, l: l * v + (1 - l) * f)
    elif plant == "first":
        monkeypatch.setattr(oracle, "mix_values", lambda v, f, l: v)
    elif plant == "cap":
        monkeypatch.setattr(oracle, "softcap", lambda s, c: s)
    elif plant == "group":
        real = oracle.attend
        monkeypatch.setattr(oracle, "attend", lambda q, k, v, *a: real(q, np.roll(k, 1, 1), np.roll(v, 1, 1), *a))
    elif plant == "norm":
        monkeypatch.setattr(oracle, "norm_centered", oracle.norm_plain)
    elif plant == "side":
        real_side = oracle.token_side
        monkeypatch.setattr(oracle, "token_side", lambda x, t, w, p, i, d, e: real_side(x, t, w, p, 0, d, e))
    else:
        monkeypatch.setattr(oracle, "clipped_glu", lambda g, u, l: g / (1 + np.exp(-1.702 * g)) * (u + 1))
    err = np.sqrt(((oracle.Model(cfg, w).run(toks) - want) ** 2).mean()) / want.std()
    assert err > 0.02


# -- configuration, names, weights ----------------------------------------------------------------------------------
def test_configuration_and_names(tmp_path):
    from mfq_b200.checkpoint import read_hf_directory
    from mfq_b200.models import registry
    from mfq_b200.models.tepetar import TepetarConfig, tensor_shapes
    src = cases.uneven()
    raw, tensors, _ = read_hf_directory(cases.write(tmp_path / "m", src, cases.weights(src)))
    assert registry.find(raw).name == "tepetar" and raw["vocab_size"] == 150 and raw["num_layers"] == 5
    cfg = TepetarConfig.from_dict(json.loads(json.dumps(raw)))
    assert {k: tuple(v.shape) for k, v in tensors.items()} == tensor_shapes(cfg)
    assert [l.window for l in cfg.layers] == [17, 40, 1, 100, 33] and cfg.layers[0].ff == 0 and not cfg.layers[2].v_mix
    assert cfg.layers[3].softcap == 2.0 and cfg.layers[3].rot_base == 7e5 and cfg.layers[1].scale == 0.4 and cfg.norm_eps == 1e-5


def test_configuration_rejects_what_the_kernels_cannot_run():
    from mfq_b200.models.tepetar import TepetarConfig
    bad = cases.config([cases.layer()])
    bad["layers"][0]["type"] = "something"
    with pytest.raises(ValueError, match="unknown mixer"):
        TepetarConfig.from_source(bad)
    bad = cases.config([cases.layer()])
    bad["layers"][0]["mlp"]["kind"] = "routed"
    with pytest.raises(ValueError, match="unknown feed-forward"):
        TepetarConfig.from_source(bad)
    for broken in (cases.layer(heads=5), cases.layer(dim=300), cases.layer(rot=40), cases.layer(scale=0.0), cases.layer(window=-1)):
        with pytest.raises(ValueError):
            TepetarConfig.from_source(cases.config([broken]))
    with pytest.raises(ValueError, match="share values"):
        TepetarConfig.from_source(cases.config([cases.layer(), cases.layer(vdim=32)]))


def test_element_types_and_devices_are_refused_clearly(tmp_path):
    from mfq_b200.checkpoint import load_engine
    from mfq_b200.models import registry
    src = cases.config([cases.layer()])
    path = cases.write(tmp_path / "m", src, cases.weights(src))
    with pytest.raises(RuntimeError, match="CUDA"):
        load_engine(path, "cpu", max_batch=1, max_seq_len=32)
    with pytest.raises(ValueError, match="context extension"):
        load_engine(path, "cpu", max_batch=1, max_seq_len=32, yarn_context_extension=2.0)
    with pytest.raises(registry.UnsupportedDtype, match="float32"):
        registry.find({"num_layers": 1}).check_dtype("float32")


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_weights_as_stored_compute_the_same_products(dtype):
    """The padded, stacked and interleaved matrices give the plain products at the places the kernels read them from."""
    from mfq_b200.architectures import to_canonical
    from mfq_b200.models.tepetar import TepetarConfig, TepetarWeights
    from mfq_b200.ops.dense import up
    src = cases.uneven()
    w = cases.weights(src)
    cfg = TepetarConfig.from_source(src)
    packed = TepetarWeights(cfg, {k: torch.from_numpy(np.asarray(v)) for k, v in to_canonical(w, src).items()}, "cpu", dtype)
    x = np.random.default_rng(0).standard_normal(cfg.hidden_size)
    xp = np.zeros(up(cfg.hidden_size))
    xp[: cfg.hidden_size] = x
    for i, (l, p) in enumerate(zip(cfg.layers, packed.layers)):
        q = oracle.linear(x, w[f"l{i}.mix.q"], w[f"l{i}.mix.q.b"]).reshape(l.heads, l.dim)
        v = oracle.linear(x, w[f"l{i}.mix.v"], w[f"l{i}.mix.v.b"]).reshape(l.kv_heads, l.vdim)
        got = oracle.linear(xp, p.qkv.w.double().numpy(), p.qkv.bias.double().numpy())
        dk, dv = up(l.dim), up(l.vdim)
        gq, gv = got[: l.heads * dk].reshape(l.heads, dk), got[(l.heads + l.kv_heads) * dk :].reshape(l.kv_heads, dv)
        assert np.allclose(gq[:, : l.dim], q) and not gq[:, l.dim :].any() and np.allclose(gv[:, : l.vdim], v) and not gv[:, l.vdim :].any()
        assert np.allclose(p.attn_post_norm[: cfg.hidden_size].numpy(), 1 + w[f"l{i}.norm1"]) and not p.attn_post_norm[cfg.hidden_size :].any()
        assert torch.equal(p.side_table[:, : cfg.side_dim].float(), torch.from_numpy(w["side.embed"][:, i * cfg.side_dim : (i + 1) * cfg.side_dim]))
        assert abs(p.value_mix - float(w[f"l{i}.mix.vmix"])) < 1e-7 and (p.gate_up is None) == (l.ff == 0)
        if l.ff:
            both = oracle.linear(xp, p.gate_up.w.double().numpy()).reshape(-1, 2, 8)
            assert np.allclose(both[:, 0].reshape(-1)[: l.ff], oracle.linear(x, w[f"l{i}.mlp.gate"]))
            assert np.allclose(both[:, 1].reshape(-1)[: l.ff], oracle.linear(x, w[f"l{i}.mlp.up"]))
    assert packed.lm_head.w.shape == (160, 112) and not packed.lm_head.w[150:].any()


def test_product_plan_stays_within_the_kernels_limits():
    from mfq_b200.ops import dense
    for m in (1, 8, 9, 16, 17, 64, 65, 128, 129, 300, 513, 4096):
        for n in (16, 256, 6144, 28672, 128256):
            for k in (8, 72, 256, 4096, 14336):
                tile, splits = dense.plan(m, n, k)
                assert (tile == 0 and m <= 16 and splits == 1) or (tile in (16, 32, 64, 128, 256) and 1 <= splits <= 8)


def test_decode_splits_leave_pages_for_everyone():
    from mfq_b200.ops.window_attn import decode_splits
    for batch in (1, 2, 7, 32, 64, 256):
        for heads in (1, 2, 8, 40):
            for keys in (1, 63, 64, 400, 4096, 1 << 20):
                s = decode_splits(batch, heads, keys)
                assert 1 <= s <= 16 and (s == 1 or keys // s >= 64)


def test_memory_of_a_deployment_counts_unquantized_pages():
    from mfq_b200.models.tepetar import TepetarConfig
    from mfq_b200.server.analysis import model_memory
    cfg = TepetarConfig.from_source(cases.uneven()).to_dict()
    per_token = 2 * (4 * (48 + 32) + 2 * (32 + 32) + (80 + 64) + 2 * (32 + 32) + 2 * (16 + 32))
    assert model_memory(cfg, 1000, batch=2, context=64)["per_gpu"]["kv_cache"] == (2 * 4 + 1) * 16 * per_token


# -- pages ----------------------------------------------------------------------------------------------------------
def test_unquantized_pages_move_between_caches():
    from mfq_b200.engine.kv_cache import PlainPagedKVCache
    make = lambda: PlainPagedKVCache([(2, 16, 32), (1, 48, 16)], torch.bfloat16, num_pages=9, max_seqs=2, max_pages_per_seq=4, device="cpu")
    a, b = make(), make()
    a.assign(0, 7, 33)
    b.assign(1, 3, 20)
    b.assign(0, 4, 40)
    for pool in a.pools:
        pool.k.normal_()
        pool.v.normal_()
    pa, pb = a.allocator.owned[7], b.allocator.owned[4]
    blob = a.export_pages(pa)
    assert blob.nbytes == a.page_blob_bytes(3) == 3 * 16 * a.bytes_per_token() and pa != pb
    b.import_pages(pb, blob)
    for i in range(2):
        assert torch.equal(a.layer(i).k[pa], b.layer(i).k[pb]) and torch.equal(a.layer(i).v[pa], b.layer(i).v[pb])
        assert not b.layer(i).k[b.allocator.owned[3]].any()
    assert a.slots(7, 15, 3).tolist() == [pa[0] * 16 + 15, pa[1] * 16, pa[1] * 16 + 1]
    a.release(7)
    assert a.allocator.free_pages == 8


# -- scheduler ------------------------------------------------------------------------------------------------------
class MixedBackend:
    """A backend whose next token is a hash of the whole context, with pages to run out of; it records every batch."""

    max_batch, mixed_batches, prefill_chunk = 4, True, 2048

    def __init__(self, pages=100):
        self.pages, self.rows, self.batches = pages, {}, []

    def _need(self, tokens):
        return -(-tokens // 4)

    def free_tokens(self):
        return (self.pages - sum(self._need(len(r["ids"]) + 1) for r in self.rows.values())) * 4

    def tokens_needed(self, tokens):
        return self._need(tokens) * 4

    def begin_prompt(self, row, tokens, params, **extra):
        assert row not in self.rows
        self.rows[row] = {"ids": list(tokens), "read": 0}
        return len(tokens)

    def _next(self, row):
        r = self.rows[row]
        tok = next_token(r["ids"])
        r["ids"].append(tok)
        return tok

    def mixed_step(self, rows, portions):
        self.batches.append((list(rows), list(portions)))
        out = {}
        for row, count in portions:
            r = self.rows[row]
            r["read"] += count
            assert count > 0 and r["read"] <= len(r["ids"]) and row not in rows
            if r["read"] == len(r["ids"]):
                out[row] = self._next(row)
        return {**out, **{row: self._next(row) for row in rows}}

    def decode(self, rows):
        self.batches.append((list(rows), []))
        assert all(r["read"] > 0 for r in self.rows.values())
        return {row: self._next(row) for row in rows}

    def can_grow(self, row):
        return self.free_tokens() >= 0

    def release(self, row):
        self.rows.pop(row, None)


def next_token(ids):
    return (sum((i + 1) * t for i, t in enumerate(ids)) * 31 + 7) % 97


def continuation(prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(next_token(ids))
    return ids[len(prompt):]


@pytest.mark.parametrize("budget", [1, 3, 8, 1000])
def test_prompts_are_read_beside_decoding_rows(budget):
    from mfq_b200.engine.scheduler import ContinuousBatchScheduler, Request, SamplingParams
    back = MixedBackend()
    sched = ContinuousBatchScheduler(back, mixed_tokens=budget)
    prompts = [list(range(1, n)) for n in (6, 12, 3, 21, 2, 9)]
    reqs = [Request(prompt=p, params=SamplingParams(max_tokens=7)) for p in prompts]
    for r in reqs[:2]:
        sched.submit(r)
    for _ in range(4):
        sched.step()
    for r in reqs[2:]:
        sched.submit(r)
    sched.run_until_idle()
    assert [r.generated for r in reqs] == [continuation(p, 7) for p in prompts] and not back.rows
    assert all(sum(c for _, c in portions) <= budget for _, portions in back.batches)
    assert any(rows and portions for rows, portions in back.batches)  # the point of it
    assert sched.stats.mixed_steps == sum(1 for _, portions in back.batches if portions)


def test_mixed_batches_survive_retraction_stop_tokens_and_failures():
    from mfq_b200.engine.scheduler import ContinuousBatchScheduler, Request, SamplingParams
    back = MixedBackend(pages=14)
    sched = ContinuousBatchScheduler(back, mixed_tokens=4)
    prompts = [list(range(1, n)) for n in (10, 9, 8)]
    reqs = [Request(prompt=p, params=SamplingParams(max_tokens=25)) for p in prompts]
    for r in reqs:
        sched.submit(r)
    sched.run_until_idle()
    assert [r.generated for r in reqs] == [continuation(p, 25) for p in prompts] and sched.stats.retractions > 0
    stop = continuation(prompts[0], 3)[2]
    first = continuation(prompts[0], 25).index(stop)
    r = Request(prompt=prompts[0], params=SamplingParams(max_tokens=25, stop_token_ids=(stop,)))
    sched.submit(r)
    sched.run_until_idle()
    assert r.finish_reason == "stop" and len(r.generated) == first + 1
    broken = Request(prompt=[1, 2], params=SamplingParams(max_tokens=3))
    good = Request(prompt=[3, 4], params=SamplingParams(max_tokens=3))
    begin = back.begin_prompt

    def refuse(row, tokens, params, **extra):
        if list(tokens) == [1, 2]:
            raise RuntimeError("no")
        return begin(row, tokens, params, **extra)
    back.begin_prompt = refuse
    sched.submit(broken)
    sched.submit(good)
    sched.run_until_idle()
    assert broken.error is not None and good.generated == continuation([3, 4], 3) and sched.healthy
    long = Request(prompt=list(range(30)), params=SamplingParams(max_tokens=4))
    sched.submit(long)
    sched.step()
    assert sched.cancel(long.id) and not back.rows and not sched.reading
    back.mixed_step = lambda rows, portions: (_ for _ in ()).throw(RuntimeError("device lost"))
    last = Request(prompt=[5, 6, 7], params=SamplingParams(max_tokens=4))
    sched.submit(last)
    sched.run_until_idle()
    assert last.error is not None and last.finish_reason == "backend_failure" and not sched.healthy


# -- trace replay ---------------------------------------------------------------------------------------------------
class ReplayEngine:
    """Answers with (row's length so far, token) instead of logits."""

    max_batch, device = 2, torch.device("cpu")

    def __init__(self):
        self.rows, self.opened = {}, []

    def open_row(self, row):
        assert row not in self.rows
        self.rows[row] = []
        self.opened.append(row)

    def release(self, row):
        del self.rows[row]

    def extend(self, portions, wanted):
        out = []
        for (row, toks), want in zip(portions, wanted):
            base = len(self.rows[row])
            self.rows[row] += toks
            out += [[base + w, toks[w]] for w in want]
        return torch.tensor(out, dtype=torch.float32) if out else None


def test_replay_keeps_requests_rows_and_order(tmp_path):
    from mfq_b200.engine.trace_runner import run
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [5, 6, 7], "want": [2, 0]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": [9], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": [1, 2], "want": [1]}, {"id": "a", "tokens": [8], "want": [0]}], "end": ["a"]},
             {"step": 4, "entries": [{"id": "c", "tokens": [3], "want": [0]}], "end": ["b", "c"]}]
    engine, said = ReplayEngine(), []
    run(engine, io.StringIO("\n".join(map(json.dumps, steps)) + "\n\n"), tmp_path, said.append)
    assert said == ["done 0", "done 1", "done 2", "done 4"] and engine.opened == [0, 1, 0] and not engine.rows
    read = lambda n: np.fromfile(tmp_path / f"{n}.f32", dtype="<f4").reshape(-1, 2).tolist()
    assert read(0) == [[2, 7], [0, 5]] and read(2) == [[2, 2], [3, 8]] and read(4) == [[0, 3]]
    assert not (tmp_path / "1.f32").exists()


def test_replay_refuses_float32_of_a_family_without_it(tmp_path):
    from mfq_b200.engine.trace_runner import main
    (tmp_path / "config.json").write_text(json.dumps({"model_type": "llama", "vocab_size": 8, "hidden_size": 8, "num_hidden_layers": 1,
                                                      "num_attention_heads": 1}))
    assert main(["--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "64"]) == 3
