"""Meronex through the framework's engine against the oracle: prompts, portions, mixed batches, decoding, generation."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from tests import meronex_helpers as H

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]
NAMES = sorted(H.CONFIGS)


def _weights(cfg, seed, dtype):
    return H.weights(cfg, seed, decided=dtype == torch.bfloat16)


def _check(got, want, dtype, what=""):
    err = H.error(got, want)
    assert err < H.TOL[dtype], (what, err)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_prompts_portions_and_decoding_agree_with_the_oracle(name, dtype):
    from arctic_platform_b200.ops import _lib
    cfg = H.CONFIGS[name]
    w, toks = _weights(cfg, 0, dtype), H.tokens(cfg, 150)
    want = H.expected(cfg, w, toks)
    eng = H.engine(cfg, w, dtype, tokens=256)          # room for one sequence: pages and slot are used again every time
    for cuts in ([150], [1], [2], [3, 5, 31, 2, 64], [16], [17, 15], [100, 1], [149, 1], [8, 9], [33], [69, 2, 1]):
        _check(H.feed(eng, toks, cuts), want, dtype, cuts)
    _lib.check_status("serving")
    assert eng.pages.free_count() == eng.num_pages


@pytest.mark.parametrize("dtype", DTYPES)
def test_layers_one_by_one(dtype):
    cfg = H.CONFIGS["mixed-layers"]
    w, toks = _weights(cfg, 4, dtype), H.tokens(cfg, 40, 4)
    runs = H.oracle.forward(cfg, w, toks)[1]
    eng = H.engine(cfg, w, dtype)
    got = []
    eng.step([(eng.open_sequence(), toks, [])], on_layer=lambda r, x: got.append(x.cpu()))
    assert len(got) == len(runs)
    for i, (a, b) in enumerate(zip(got, runs)):
        assert float((a - b).abs().max() / b.pow(2).mean().sqrt()) < 2 * H.TOL[dtype], i


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed-layers", "wide-heads"])
def test_mixed_batches_equal_each_request_alone(name, dtype):
    """Unequal requests join and leave, pause, and use each other's pages and slots; portions beside single tokens."""
    cfg = H.CONFIGS[name]
    w = _weights(cfg, 1, dtype)
    lens = [180, 3, 65, 16, 120, 17, 33, 90]
    toks = [H.tokens(cfg, n, 10 + i) for i, n in enumerate(lens)]
    want = [H.expected(cfg, w, t) for t in toks]
    eng = H.engine(cfg, w, dtype, tokens=28 * 16, slots=3)
    rng = np.random.default_rng(0)
    todo, live, got = list(range(len(lens))), {}, [[] for _ in lens]
    at = [0] * len(lens)

    def held(extra):
        return sum((at[i] + extra.get(i, 0) + 15) // 16 for i in live)

    while todo or live:
        while todo and len(live) < 3:
            i = todo.pop(0)
            live[i] = eng.open_sequence()
        work, extra = [], {}
        for i in list(live):
            if len(live) > 1 and rng.random() < 0.25:
                continue                                      # left out of this step
            n = int(min(rng.choice([1, 1, 2, 5, 17, 40]), lens[i] - at[i]))
            extra[i] = n
            if held(extra) > eng.num_pages:
                extra.pop(i)
                continue
            work.append((i, n))
        if not work:
            continue
        out = eng.step([(live[i], toks[i][at[i]:at[i] + n], list(range(n))) for i, n in work]).cpu()
        r = 0
        for i, n in work:
            got[i].append(out[r:r + n])
            r, at[i] = r + n, at[i] + n
            if at[i] == lens[i]:
                eng.close_sequence(live.pop(i))
    for i in range(len(lens)):
        _check(torch.cat(got[i]), want[i], dtype, i)
    assert eng.pages.free_count() == eng.num_pages


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed-layers", "long-range"])
def test_long_decoding(name, dtype):
    cfg = H.CONFIGS[name]
    w, toks = _weights(cfg, 2, dtype), H.tokens(cfg, 420, 2)
    want = H.expected(cfg, w, toks)
    _check(H.feed(H.engine(cfg, w, dtype), toks, [20, 1]), want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_prompts(dtype):
    """Several query tiles and key blocks, chunks and segments of the recurrences, then decoding far behind them."""
    cfg = H.CONFIGS["long-range"]
    w, toks = _weights(cfg, 3, dtype), H.tokens(cfg, 900, 3)
    want = H.expected(cfg, w, toks)
    eng = H.engine(cfg, w, dtype, tokens=1024)
    for cuts in ([900], [511, 2, 300, 1], [880, 1]):
        _check(H.feed(eng, toks, cuts), want, dtype, cuts)


def test_logits_do_not_depend_on_pages_slots_or_the_batch():
    """The same request alone, and later in other pages and another slot beside others: equal to fp32 rounding."""
    cfg = H.CONFIGS["mixed-layers"]
    w, toks = H.weights(cfg, 11), [H.tokens(cfg, 90, i) for i in range(3)]
    eng = H.engine(cfg, w, torch.float32, tokens=512)
    alone = H.feed(eng, toks[0], [60, 7, 1])
    other = eng.open_sequence()
    eng.step([(other, toks[1], [])])
    mine, third = eng.open_sequence(), eng.open_sequence()
    got, at = [], 0
    for n in (60, 7) + (1,) * 23:
        work = [(third, toks[2][at:at + n], []), (mine, toks[0][at:at + n], list(range(n)))]
        got.append(eng.step(work).cpu())
        at += n
    assert mine != 0 and H.error(torch.cat(got), alone) < 1e-5


def test_step_interface_refuses_what_does_not_fit():
    cfg = H.CONFIGS["plain"]
    eng = H.engine(cfg, H.weights(cfg), torch.float32, tokens=64, slots=2, max_seq_len=100)
    a, b = eng.open_sequence(), eng.open_sequence()
    with pytest.raises(RuntimeError, match="slots"):
        eng.open_sequence()
    with pytest.raises(RuntimeError, match="open"):
        eng.generate([[1, 2]], {"max_tokens": 1})
    eng.step([(a, [1] * 40, [])])
    with pytest.raises(RuntimeError, match="KV cache"):
        eng.step([(b, [1] * 40, [])])
    with pytest.raises(ValueError, match="max_seq_len"):
        eng.step([(a, [1] * 70, [])])
    with pytest.raises(ValueError, match="wanted"):
        eng.step([(b, [1, 2], [2])])
    assert eng.step([(b, [1] * 16, [15])]).shape == (1, cfg["vocab"])
    eng.close_sequence(a)
    eng.close_sequence(b)
    assert eng.pages.free_count() == eng.num_pages == 4


# ---------------------------------------------------------------------------- generation
def _follow(cfg, w, prompt, rec, tol):
    """Every generated token is the oracle's arg-max (up to ties within rounding) and its log-prob the oracle's."""
    seq = list(prompt) + rec["token_ids"]
    lp = torch.log_softmax(H.expected(cfg, w, seq), -1)
    for i, (t, l) in enumerate(zip(rec["token_ids"], rec["logprobs"])):
        row = lp[len(prompt) - 1 + i]
        assert float(row.max() - row[t]) < tol, (i, float(row.max() - row[t]))
        assert abs(float(row[t]) - l) < tol, i


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 1e-3), (torch.bfloat16, 0.25)])
@pytest.mark.parametrize("graph", [False, True])
def test_greedy_generation(dtype, tol, graph):
    """More prompts than slots, prompts cut into portions, several samples per prompt, slots used again."""
    from arctic_platform_b200.ops import _lib
    cfg = H.CONFIGS["mixed-layers"]
    w = _weights(cfg, 5, dtype)
    eng = H.engine(cfg, w, dtype, tokens=1024, slots=8, max_seq_len=256, prefill_tokens=23, sync_interval=4,
                   use_cuda_graph=graph)
    prompts = [H.tokens(cfg, n, n) for n in (37, 16, 1, 64, 5, 33, 2)]
    outs = eng.generate(prompts, {"n": 2, "temperature": 0.0, "max_tokens": 19, "ignore_eos": True})
    _lib.check_status("generate")
    assert len(outs) == 14 and eng.pages.free_count() == eng.num_pages
    for o in outs:
        assert len(o["token_ids"]) == 19 and o["finish_reason"] == "length"
        _follow(cfg, w, prompts[o["prompt_index"]], o, tol)
    for a, b in zip(outs[::2], outs[1::2]):
        assert dtype != torch.float32 or a["token_ids"] == b["token_ids"]
    # a second call on the same engine, now with a stop token
    stop = outs[0]["token_ids"][3]
    again = eng.generate(prompts[:1], {"temperature": 0.0, "max_tokens": 19, "stop_token_ids": [stop]})[0]
    first = outs[0]["token_ids"].index(stop)
    if dtype == torch.float32:
        assert again["token_ids"] == outs[0]["token_ids"][:first + 1] and again["finish_reason"] == "stop"


def test_a_checkpoint_with_another_rank_replaces_captured_steps():
    cfg = H.CONFIGS["mixed-layers"]
    w, other = H.weights(cfg, 5), H.weights(cfg, 6, rank=40)
    eng = H.engine(cfg, w, torch.float32, slots=4, max_seq_len=128)
    p, sp = H.tokens(cfg, 20, 1), {"temperature": 0.0, "max_tokens": 8, "ignore_eos": True}
    _follow(cfg, w, p, eng.generate([p], sp)[0], 1e-3)
    for n, t in other.items():
        eng.model.load_named_tensor(n, t)
    eng.weights_updated()
    _follow(cfg, other, p, eng.generate([p], sp)[0], 1e-3)


def test_sampling_is_seeded_filtered_and_reports_log_probs():
    cfg = H.CONFIGS["mixed-layers"]
    w = H.weights(cfg, 6)
    eng = H.engine(cfg, w, torch.float32, slots=8, max_seq_len=128)
    p = H.tokens(cfg, 20, 1)
    a = eng.generate([p], {"n": 8, "temperature": 1.0, "max_tokens": 12, "seed": 3})
    b = eng.generate([p], {"n": 8, "temperature": 1.0, "max_tokens": 12, "seed": 3})
    assert [x["token_ids"] for x in a] == [x["token_ids"] for x in b]
    assert len({tuple(x["token_ids"]) for x in a}) > 4
    for rec in a[:3]:
        lp = torch.log_softmax(H.expected(cfg, w, p + rec["token_ids"]), -1)
        for i, (t, l) in enumerate(zip(rec["token_ids"], rec["logprobs"])):
            assert abs(float(lp[len(p) - 1 + i, t]) - l) < 1e-3
    k1 = eng.generate([p], {"n": 2, "temperature": 1.0, "top_k": 1, "max_tokens": 6})
    assert k1[0]["token_ids"] == k1[1]["token_ids"] == \
        eng.generate([p], {"temperature": 0.0, "max_tokens": 6})[0]["token_ids"]


def test_worker_serves_a_checkpoint_directory(tmp_path):
    """The entry point every client uses: a sampling job named by its directory; sleep, wake, weight hand-over."""
    from arctic_platform_b200.engine.stateful_sampler import StatefulSampler
    from arctic_platform_b200.engine.worker import EngineWorker
    cfg = H.CONFIGS["mixed-layers"]
    w = H.weights(cfg, 7, decided=True)
    worker = EngineWorker("cuda:0")
    worker.initialize({"model_name": str(H.save(cfg, w, tmp_path / "m")), "job_type": "sampling",
                       "vllm_config": {"kv_cache_tokens": 4096, "max_num_seqs": 8, "max_model_len": 256}})
    assert isinstance(worker.sampler, StatefulSampler)
    prompts = [H.tokens(cfg, n, n) for n in (30, 12)]
    sp = {"temperature": 0.0, "max_tokens": 8, "ignore_eos": True}
    first = worker.sampler.generate(prompts, sp)
    for o in first:
        _follow(cfg, w, prompts[o["prompt_index"]], o, 0.25)
    scored = worker.score_completions(prompts, [o["token_ids"] for o in first], top_k=3)
    for o, lp, top in zip(first, scored["log_probs"], scored["top_log_probs"]):
        assert np.abs(np.array(lp) - np.array(o["logprobs"])).max() < 0.2
        assert all(len(t) == 3 and abs(max(t.values()) - v) < 0.2 for t, v in zip(top, lp))
    worker.sampler.sleep(1)
    with pytest.raises(RuntimeError, match="asleep"):
        worker.sampler.generate(prompts, sp)
    worker.sampler.wake()
    assert worker.sampler.generate(prompts, sp)[0]["token_ids"] == first[0]["token_ids"]
    new = H.weights(cfg, 8, decided=True)
    worker.sampler.sleep(2)
    worker.sampler.wake(["weights"])
    assert worker.load_weights(list(new.items())) == len(new)
    worker.sampler.wake(["kv_cache"])
    for o in worker.sampler.generate(prompts, sp):
        _follow(cfg, new, prompts[o["prompt_index"]], o, 0.25)
    norm = worker.sampler.weight_norm()["norm"]
    assert abs(norm - sum(float(t.double().pow(2).sum()) for t in new.values()) ** 0.5) < 1e-3 * norm


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_replaying_a_trace(tmp_path, dtype):
    root = Path(__file__).resolve().parents[1]
    cfg = H.CONFIGS["odd-sizes"]
    w = _weights(cfg, 9, getattr(torch, dtype))
    model = H.save(cfg, w, tmp_path / "m")
    toks = {"a": H.tokens(cfg, 50, 1), "b": H.tokens(cfg, 21, 2), "c": H.tokens(cfg, 40, 3)}
    want = {k: H.expected(cfg, w, t) for k, t in toks.items()}
    plan = [[("a", 30)], [("a", 1), ("b", 20)], [("b", 1)], [("a", 19), ("c", 2)], [("c", 38)]]
    at, lines, rows = {k: 0 for k in toks}, [], []
    for n, step in enumerate(plan):
        entries, r = [], []
        for k, c in step:
            places = sorted({0, c - 1})
            entries.append({"id": k, "tokens": toks[k][at[k]:at[k] + c], "want": [] if n == 2 else places})
            r += [] if n == 2 else [want[k][at[k] + p] for p in places]
            at[k] += c
        rows.append(r)
        lines.append(json.dumps({"step": n, "entries": entries, "end": [k for k, c in step if at[k] == len(toks[k])]}))
    (tmp_path / "out").mkdir()
    res = subprocess.run([sys.executable, str(root / "bin" / "trace_run"), "--model", str(model), "--dtype", dtype,
                          "--out", str(tmp_path / "out"), "--max-tokens", "128"], input="\n".join(lines) + "\n",
                         capture_output=True, text=True, timeout=300)
    assert res.returncode == 0, res.stderr[-2000:]
    assert [x for x in res.stdout.splitlines() if x.startswith("done")] == [f"done {n}" for n in range(len(plan))]
    assert not (tmp_path / "out" / "2.f32").exists()
    for n, r in enumerate(rows):
        if r:
            got = torch.from_numpy(np.fromfile(tmp_path / "out" / f"{n}.f32", "<f4").reshape(len(r), -1))
            _check(got, torch.stack(r), getattr(torch, dtype), n)
