"""The Gogivik family through the framework's engine, loader and scheduler, against the plain restatement."""

import io
import json

import numpy as np
import pytest
import torch

import gogivik_cases as cases
import gogivik_oracle as oracle
from gpu_common import check_status, require_gpu_lib
from test_gpu_tepetar import engine_of, whole

pytestmark = pytest.mark.gpu
BOTH = pytest.mark.parametrize("dtype", ["float32", "bfloat16"])


@pytest.fixture(scope="module", autouse=True)
def _lib():
    require_gpu_lib()


def agree(got, want, dtype, what=""):
    """fp32: the worst position; bf16: nearly all positions (a run of channels whose sum nearly cancels is normed up, with its rounding),
    none far off."""
    got, want = np.asarray(got.float().cpu(), dtype=np.float64), np.asarray(want)
    assert got.shape == want.shape
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    e = np.sqrt((d ** 2).mean(-1)) / np.sqrt(((want - want.mean(-1, keepdims=True)) ** 2).mean())
    if dtype == "float32":
        assert e.max() < 2e-4, (what, e.max())
    else:
        assert np.quantile(e, 0.97) < 0.06 and e.max() < 0.5, (what, np.quantile(e, 0.97), e.max())


def latent_only():
    return cases.config([cases.latent(mlp=cases.dense()), cases.latent(window=70, heads=17), cases.latent(q_rank=130, rank=100, rot=16, dim=100, vdim=130, window=9)], taps=2)


def chunked_only():
    return cases.config([cases.chunked(mlp=cases.dense(40)), cases.chunked(heads=20, kv_heads=1, dim=64, vdim=64, rot=64, size=33, factor=1.0, scale=0.2)], taps=3)


def recurrent_only():
    return cases.config([cases.mamba(mlp=cases.dense(40)), cases.mamba(heads=1, groups=1, state=64, vdim=16, conv=1, norm_groups=1)], taps=8)


def one_of_everything():
    """A single head, group, tap and token of whatever can be one."""
    return cases.config([cases.latent(heads=1, window=1), cases.chunked(heads=1, kv_heads=1, size=1), cases.mamba(heads=1, groups=1, conv=1, norm_groups=1),
                         cases.chunked(heads=2, kv_heads=2, size=10 ** 10), cases.latent(heads=1, rot=2, window=10 ** 10, mlp=cases.dense(16))], taps=1, logit_scale=1.0)


@BOTH
@pytest.mark.parametrize("make", [cases.uneven, latent_only, chunked_only, recurrent_only, one_of_everything])
def test_whole_prompts_and_every_layer(tmp_path, make, dtype):
    cfg = make()
    w, toks = cases.weights(cfg), cases.tokens(cfg, 150)
    eng = engine_of(tmp_path, cfg, w, dtype)
    trace = []
    want = oracle.Model(cfg, w).run(toks, trace=trace)
    agree(whole(eng, 0, toks), want, dtype)
    eng.open_row(1)
    eng.cache.assign(1, eng.row_seq[1], len(toks))
    layers = []
    ids = torch.tensor(toks, dtype=torch.int32, device="cuda")
    eng.model.forward(eng._ragged_step([(1, 0, len(toks))], ids), eng.cache, prefill=True, layer_outputs=layers)
    assert len(layers) == len(trace)
    for i, (a, b) in enumerate(zip(layers, trace)):
        rel = np.abs(a.double().cpu().numpy() - b) / np.sqrt((b ** 2).mean())
        assert rel.max() < 2e-4 if dtype == "float32" else np.quantile(rel, 0.98) < 0.1, f"layer {i}"
    check_status()


@BOTH
@pytest.mark.parametrize("size", [1, 2, 3, 16, 17, 50, 65])
def test_portions_and_decoding_agree_with_the_whole(tmp_path, size, dtype):
    cfg = cases.uneven()
    w, toks = cases.weights(cfg), cases.tokens(cfg, 140)
    eng = engine_of(tmp_path, cfg, w, dtype)
    want = oracle.Model(cfg, w).run(toks)
    eng.open_row(2)
    got = [eng.extend([(2, toks[a : a + size])], [range(len(toks[a : a + size]))]) for a in range(0, len(toks), size)]
    agree(torch.cat(got), want, dtype)
    check_status()


@BOTH
def test_unequal_requests_in_one_batch_reused_pages_and_slots(tmp_path, dtype):
    """Requests of different ages and portions share every step; rows, pages and state slots go round several times in a pool that
    holds no more than the live requests."""
    cfg = cases.uneven()
    w = cases.weights(cfg)
    eng = engine_of(tmp_path, cfg, w, dtype, num_pages=36, max_seq_len=256)
    model, rng = oracle.Model(cfg, w), np.random.default_rng(3)
    live, made = {}, 0
    for _ in range(70):
        while len(live) < 3 and made < 12:
            toks = cases.tokens(cfg, int(rng.integers(1, 170)), seed=100 + made)
            row = next(r for r in range(4) if r not in live)
            eng.open_row(row)
            live[row] = [toks, 0, model.run(toks), []]
            made += 1
        batch = {}
        for row in sorted(live, key=lambda r: -r):
            toks, at = live[row][:2]
            n = min(len(toks) - at, int(rng.choice([1, 1, 2, 7, 40, 90])))
            if rng.random() < 0.8:
                batch[row] = n
        if not batch:
            continue
        out = eng.extend([(r, live[r][0][live[r][1] : live[r][1] + n]) for r, n in batch.items()], [range(n) for n in batch.values()])
        for r, n in batch.items():
            live[r][3].append(out[:n])
            out = out[n:]
            live[r][1] += n
            if live[r][1] == len(live[r][0]):
                agree(torch.cat(live[r][3]), live[r][2], dtype)
                eng.release(r)
                del live[r]
    assert made == 12 and not live
    check_status()


@BOTH
@pytest.mark.parametrize("make,size", [(cases.window_spotlight, n) for n in (2, 16, 31, 64, 65)] + [(cases.chunk_spotlight, n) for n in (2, 16, 31, 64, 65)])
def test_edges_of_windows_and_chunks(tmp_path, make, size, dtype):
    cfg, w = make(size)
    eng = engine_of(tmp_path, cfg, w, dtype)
    model = oracle.Model(cfg, w)
    for spot in (0, 1, 15, 16, 40):
        last = spot + size - 1 if make is cases.window_spotlight else spot // size * size + size - 1
        n = last + 5
        toks = [2 + (i * 7) % 17 for i in range(n)]
        toks[spot] = 1
        want = model.run(toks)
        blind = model.run([2 + (spot * 7) % 17 if t == 1 else t for t in toks])
        seen = np.abs(want - blind).max(-1)
        assert seen[last] > 0.1 and seen[last + 1] < 1e-9  # the case shows the edge
        agree(whole(eng, 0, toks), want, dtype)
        eng.open_row(1)
        eng.extend([(1, toks[: max(1, spot)])])
        got = [eng.extend([(1, [t])], [[0]]) for t in toks[max(1, spot) :]]
        agree(torch.cat(got), want[max(1, spot) :], dtype)
        eng.open_row(2)  # the last portion starts inside and ends behind the edge
        eng.extend([(2, toks[: spot + 1])])
        agree(eng.extend([(2, toks[spot + 1 :])], [range(n - spot - 1)]), want[spot + 1 :], dtype)


@BOTH
def test_the_first_tokens_reach_far_through_the_state(tmp_path, dtype):
    cfg, w = cases.memory()
    eng = engine_of(tmp_path, cfg, w, dtype)
    toks = cases.tokens(cfg, 300)
    model = oracle.Model(cfg, w)
    want = model.run(toks)
    other = model.run(toks[3:])[-1]
    assert np.abs(want[-1] - other).max() > 5e-3 * want.std()
    for size in (300, 128, 64, 63, 7, 1):
        eng.open_row(0)
        got = [eng.extend([(0, toks[a : a + size])], [range(len(toks[a : a + size]))]) for a in range(0, 300, size)]
        agree(torch.cat(got), want, dtype)
    eng.open_row(0)  # the slot starts from zero again
    agree(eng.extend([(0, toks[3:])], [[296]]), other[None], dtype)


@BOTH
def test_long_decoding(tmp_path, dtype):
    cfg = cases.config([cases.latent(window=50), cases.mamba(conv=4), cases.chunked(size=90, mlp=cases.dense()), cases.latent(window=20)])
    w, toks = cases.weights(cfg), cases.tokens(cfg, 400)
    eng = engine_of(tmp_path, cfg, w, dtype)
    want = oracle.Model(cfg, w).run(toks)
    eng.open_row(0)
    got = [eng.extend([(0, toks[:40])], [[39]])]
    got += [eng.extend([(0, [t])], [[0]]) for t in toks[40:]]
    agree(torch.cat(got), want[39:], dtype)


def margin_prompts(cfg, w, count, new):
    """Prompts whose greedy continuation never meets a near-tie, so that rounding cannot change a token."""
    model, found = oracle.Model(cfg, w), []
    for seed in range(400):
        prompt = cases.tokens(cfg, 5 + 13 * (seed % 7), seed=1000 + seed)
        state, ids, safe = model.start(), [], True
        logits = model.run(prompt, state)[-1]
        for _ in range(new):
            top = np.sort(logits)[-2:]
            safe = safe and top[1] - top[0] > 0.02 * logits.std()
            ids.append(int(logits.argmax()))
            logits = model.run(ids[-1:], state)[-1]
        if safe:
            found.append((prompt, ids))
        if len(found) == count:
            break
    assert len(found) == count
    return found


def mixed_model():
    return cases.config([cases.latent(mlp=cases.dense()), cases.mamba(), cases.chunked(mlp=cases.dense(32)), cases.latent(window=30)])


def test_greedy_generation_through_engine_and_scheduler(tmp_path):
    from mfq_b200.engine.scheduler import ContinuousBatchScheduler, Request, SamplingParams
    cfg = mixed_model()
    w = cases.weights(cfg)
    want = margin_prompts(cfg, w, 6, 10)
    for graphs in (False, True):
        eng = engine_of(tmp_path, cfg, w, "float32", use_graphs=graphs)
        for _ in range(2):  # the second time on used slots and captured graphs
            res = eng.generate([torch.tensor(p) for p, _ in want[:4]], 10)
            assert res.tokens.tolist() == [ids for _, ids in want[:4]]
    for mixed_tokens in (7, 64, 4096):
        eng = engine_of(tmp_path, cfg, w, "float32")
        sched = ContinuousBatchScheduler(eng, mixed_tokens=mixed_tokens)
        reqs = [Request(prompt=p, params=SamplingParams(max_tokens=10)) for p, _ in want]
        for r in reqs:
            sched.submit(r)
        sched.run_until_idle()
        assert [r.generated for r in reqs] == [ids for _, ids in want]
        assert sched.stats.mixed_steps > 0 and eng.cache.allocator.free_pages == eng.cache.num_pages - 1
    check_status()


def test_captured_decode_steps_in_bf16(tmp_path):
    """A captured step and an eager one give the same tokens; the longest context grows past several split plans."""
    cfg = mixed_model()
    w = cases.weights(cfg)
    outs = []
    for graphs in (False, True):
        eng = engine_of(tmp_path, cfg, w, "bfloat16", use_graphs=graphs)
        outs.append(eng.generate([torch.tensor(cases.tokens(cfg, n, seed=n)) for n in (3, 40, 100)], 80).tokens.tolist())
    assert outs[0] == outs[1]
    check_status()


def test_sampling_scoring_and_retraction(tmp_path):
    """Scores are the oracle's log probabilities; a pool that is too small retracts (and rebuilds the state of the retracted rows) and
    still finishes with the same tokens; seeded sampling does not depend on how the prompt was read."""
    from mfq_b200.engine.scheduler import ContinuousBatchScheduler, Request, SamplingParams
    cfg = mixed_model()
    w = cases.weights(cfg)
    eng = engine_of(tmp_path, cfg, w, "float32")
    prompt = cases.tokens(cfg, 40)
    outs = []
    for mixed_tokens in (5, 500):
        sched = ContinuousBatchScheduler(eng, mixed_tokens=mixed_tokens)
        reqs = [Request(prompt=prompt, params=SamplingParams(max_tokens=8, temperature=0.8, top_k=20, seed=s)) for s in (1, 2, 1)]
        for r in reqs:
            sched.submit(r)
        sched.run_until_idle()
        outs.append([r.generated for r in reqs])
    assert outs[0] == outs[1] and outs[0][0] == outs[0][2]
    logits = oracle.Model(cfg, w).run(prompt)
    logp = logits - np.log(np.exp(logits - logits.max(-1, keepdims=True)).sum(-1, keepdims=True)) - logits.max(-1, keepdims=True)
    assert np.allclose(eng.score(0, prompt, 10), [logp[i - 1, prompt[i]] for i in range(10, 40)], atol=3e-3)
    want, retracted = margin_prompts(cfg, w, 4, 40), 0
    for pages in (9, 12, 16):
        small = engine_of(tmp_path, cfg, w, "float32", num_pages=pages, max_seq_len=128)
        sched = ContinuousBatchScheduler(small)
        sched.new_token_ratio = 0.0  # admits as if nobody would grow
        reqs = [Request(prompt=p, params=SamplingParams(max_tokens=40)) for p, _ in want]
        for r in reqs:
            sched.submit(r)
        sched.run_until_idle()
        assert [r.generated for r in reqs] == [ids for _, ids in want] and small.cache.allocator.free_pages == pages - 1
        retracted += sched.stats.retractions
    assert retracted > 0


def test_a_conversation_continues_from_its_snapshot(tmp_path):
    from mfq_b200.engine.session_cache import SessionSnapshotCache
    cfg = mixed_model()
    w, toks = cases.weights(cfg), cases.tokens(cfg, 90)
    eng = engine_of(tmp_path, cfg, w)
    eng.session_cache = SessionSnapshotCache()
    plain = eng.prefill(1, toks)
    eng.prefill(0, toks[:70], session="talk")
    eng.save_session(0, "talk", toks[:70])
    eng.release(0)
    assert eng.prefill(0, toks, session="talk") == plain and eng.session_cache.stats["restored"] == 1


def test_quantized_checkpoint_and_replay(tmp_path):
    """The family as an .mfq file (unquantized), and the replay of a trace on top of it; a quantized one loads too."""
    from mfq_b200.checkpoint import load_engine, quantize_tensors, read_hf_directory, save_checkpoint
    from mfq_b200.engine.trace_runner import run
    cfg = cases.uneven()
    w, toks = cases.weights(cfg), cases.tokens(cfg, 30)
    raw, tensors, assets = read_hf_directory(cases.write(tmp_path / "src", cfg, w))
    save_checkpoint(tmp_path / "m.mfq", raw, quantize_tensors(tensors, dense="bf16"), assets)
    eng = load_engine(tmp_path / "m.mfq", "cuda", dtype="float32", max_batch=4, max_seq_len=64, num_pages=9)[0]
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:9], "want": [0, 8]}, {"id": "y", "tokens": toks[:1], "want": []}], "end": ["y"]},
             {"step": 1, "entries": [{"id": "z", "tokens": toks[:20], "want": []}, {"id": "x", "tokens": toks[9:10], "want": [0]}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[10:], "want": [19, 3]}], "end": ["x", "z"]}]
    said = []
    run(eng, io.StringIO("\n".join(map(json.dumps, steps))), tmp_path, said.append)
    assert said == ["done 0", "done 1", "done 2"]
    want = oracle.Model(cfg, w).run(toks)
    for step, places in ((0, [0, 8]), (1, [9]), (2, [29, 13])):
        got = torch.from_numpy(np.fromfile(tmp_path / f"{step}.f32", dtype="<f4").reshape(len(places), cfg["vocab"]))
        agree(got, want[places], "float32")
    assert eng.cache.allocator.free_pages == 8
    save_checkpoint(tmp_path / "q.mfq", raw, quantize_tensors(tensors, dense="nint8"), assets)
    eng = load_engine(tmp_path / "q.mfq", "cuda", max_batch=2, max_seq_len=64)[0]
    got = np.asarray(whole(eng, 0, toks).float().cpu(), dtype=np.float64)
    assert np.isfinite(got).all() and np.corrcoef(got.reshape(-1), want.reshape(-1))[0, 1] > 0.9


def test_command_line_runtime_serves_the_checkpoint(tmp_path):
    """`mfq runtime` on the checkpoint's own directory: ready, two prompts at once, shutdown."""
    import subprocess
    import sys
    from pathlib import Path
    cfg = mixed_model() | {"vocab": 300}
    path = cases.write(tmp_path / "m", cfg, cases.weights(cfg))
    ask = lambda i, n: {"v": 1, "id": i, "op": "generate", "params": {"model": "m", "input": {"benchmark_prompt_tokens": n},
                                                                      "sampling": {"temperature": 0.0, "max_new_tokens": 6}, "stream": False}}
    frames = [ask("a", 37), ask("b", 90), {"v": 1, "op": "shutdown"}]
    run = subprocess.run([sys.executable, "-m", "mfq_b200.cli", "runtime", "--model", str(path), "--ctx-size", "256",
                          "--continuous-batching", "4"], input="".join(json.dumps(f) + "\n" for f in frames), capture_output=True,
                         text=True, timeout=240, cwd=Path(__file__).resolve().parents[1])
    said = [json.loads(l) for l in run.stdout.splitlines()]
    assert run.returncode == 0, run.stderr[-2000:]
    results = {f["id"]: f["data"] for f in said if f["type"] == "result"}
    assert said[0]["type"] == "ready" and not [f for f in said if f["type"] == "error"]
    for i, n in (("a", 37), ("b", 90)):
        usage = results[i]["usage"]
        assert usage["prompt_tokens"] == n and (usage["completion_tokens"] == 6 or results[i]["finish_reason"] == "stop")
