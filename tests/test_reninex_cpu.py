"""Reninex without a GPU: configuration, checkpoint names, step planning, and the oracle's own sharpness."""
import json

import numpy as np
import pytest
import torch

from tests import reninex_helpers as H
from tests import reninex_oracle as oracle


@pytest.mark.parametrize("name", sorted(H.CONFIGS))
def test_config_round_trip_and_tensor_names(name):
    from arctic_platform_b200.models.reninex import ReninexConfig
    cfg = H.CONFIGS[name]
    rc = ReninexConfig.from_dict(json.loads(json.dumps(cfg)))
    assert ReninexConfig.from_dict(rc.to_hf_dict()) == rc
    assert sorted(rc.tensor_names()) == sorted(H.weights(cfg))
    assert rc.layer_runs() == oracle.layer_order(cfg)
    assert rc.num_parameters() == sum(t.numel() for t in H.weights(cfg).values())


@pytest.mark.parametrize("name", sorted(H.CONFIGS))
def test_checkpoint_round_trip_through_the_fused_layouts(name, tmp_path):
    from arctic_platform_b200.models import registry
    from arctic_platform_b200.models.config import resolve_config
    from arctic_platform_b200.models.hf_io import iter_hf_tensors, load_hf_checkpoint, save_hf_checkpoint
    cfg, w = H.CONFIGS[name], H.weights(H.CONFIGS[name], 3)
    src = H.save(cfg, w, tmp_path / "a")
    rc = resolve_config(str(src))
    assert registry.is_stateful(rc)
    model = registry.new_model(rc, "cpu", torch.bfloat16)
    assert load_hf_checkpoint(model, src) == len(w)
    back = dict(iter_hf_tensors(model))
    assert set(back) == set(w)
    for n, t in w.items():
        assert back[n].shape == t.shape and torch.equal(back[n], t), n
    save_hf_checkpoint(model, tmp_path / "b")
    again = registry.new_model(resolve_config(str(tmp_path / "b")), "cpu", torch.bfloat16)
    load_hf_checkpoint(again, tmp_path / "b")
    assert all(torch.equal(a, b) for a, b in zip(model.parameters(), again.parameters()))


def test_fused_padding_stays_zero():
    from arctic_platform_b200.models.reninex import ReninexConfig, ReninexLM
    cfg = H.CONFIGS["odd-sizes"]
    model = ReninexLM(ReninexConfig.from_dict(cfg), "cpu", torch.float32)
    for n, t in H.weights(cfg).items():
        model.load_named_tensor(n, torch.ones_like(t))
    blk = model.blocks[0]
    for cols, w in ((blk.in_cols, blk.w_in), (blk.out_cols, blk.w_out.t())):
        used = torch.zeros(w.shape[0], dtype=torch.bool)
        for o, n in cols.values():
            assert o % 8 == 0
            used[o:o + n] = True
        assert (w[used] == 1).all() and (w[~used] == 0).all()


def test_bad_configurations_and_tensors_are_refused(tmp_path):
    from arctic_platform_b200.models.config import resolve_config
    from arctic_platform_b200.models.hf_io import load_hf_checkpoint
    from arctic_platform_b200.models.reninex import ReninexConfig, ReninexLM

    def broken(**kw):
        d = json.loads(json.dumps(H.CONFIGS["bare"]))
        d["layers"][0].update(kw.pop("entry", {}))
        d["layers"][0]["mixer"]["right"].update(kw.pop("right", {}))
        d["layers"][0]["mixer"]["left"].update(kw.pop("left", {}))
        d.update(kw)
        return d

    for bad in (broken(entry={"type": "other"}), broken(right={"decay": [0.5]}), broken(left={"kv_heads": 3}),
                broken(right={"rot": {"dims": 64, "base": 1.0}}), broken(loop={"start": 0, "stop": 4, "times": 2}),
                broken(entry={"mlp": {"kind": "routed", "ff": 8}})):
        with pytest.raises(ValueError):
            ReninexConfig.from_dict(bad)
    (tmp_path / "m").mkdir()
    (tmp_path / "m" / "config.json").write_text(json.dumps(broken(architecture="Unheard")))
    with pytest.raises(ValueError, match="Unheard"):
        resolve_config(str(tmp_path / "m"))
    cfg, w = H.CONFIGS["bare"], H.weights(H.CONFIGS["bare"])
    model = ReninexLM(ReninexConfig.from_dict(cfg), "cpu", torch.float32)
    with pytest.raises(ValueError):
        model.load_named_tensor("embed", torch.zeros(3, 3))
    for name in ("bigram", "l0.canon1", "l7.norm1", "l0.mix.left.g", "nothing"):
        with pytest.raises(KeyError):
            model.load_named_tensor(name, torch.zeros(1))
    w.pop("l0.norm1")
    with pytest.raises(KeyError, match="l0.norm1"):
        load_hf_checkpoint(model, H.save(cfg, w, tmp_path / "part"))


def test_step_plan_tables():
    from arctic_platform_b200.ops.serving import StepBatch, StepEntry
    pages = np.arange(40, dtype=np.int32)[::-1]
    p = StepBatch.plan([StepEntry(2, np.arange(19), 5, pages[:2]), StepEntry(0, np.array([7]), 16, pages[4:6])])
    assert p["start"].tolist() == [0, 19] and p["len"].tolist() == [19, 1] and p["slot"].tolist() == [2, 0]
    assert p["row_entry"].tolist() == [0] * 19 + [1] and p["pos0"].tolist() == [5, 16]
    assert p["tiles"].tolist() == [[0, 0], [0, 8], [0, 16], [1, 0]]
    assert p["table"].tolist() == [[39, 38], [35, 34]]
    with pytest.raises(ValueError, match="pages"):
        StepBatch.plan([StepEntry(0, np.arange(17), 0, pages[:1])])
    with pytest.raises(ValueError, match="once"):
        StepBatch.plan([StepEntry(0, np.arange(1), 0, pages), StepEntry(0, np.arange(1), 1, pages)])
    with pytest.raises(ValueError):
        StepBatch.plan([StepEntry(0, np.arange(0), 0, pages)])


def test_prompt_portions_cover_every_prompt_in_order():
    from arctic_platform_b200.engine.stateful_sampler import StatefulSampler
    eng = object.__new__(StatefulSampler)
    for budget in (1, 5, 16, 1000):
        eng.prefill_tokens = budget
        lens = [3, 17, 1, 40]
        steps = eng._plan_portions(lens)
        seen = {i: 0 for i in range(4)}
        for st in steps:
            assert sum(n for _, _, n in st) <= budget and len({i for i, _, _ in st}) == len(st)
            for i, at, n in st:
                assert at == seen[i] and n > 0
                seen[i] += n
        assert list(seen.values()) == lens


def test_served_only_on_a_gpu_and_only_as_a_sampler(tmp_path):
    from arctic_platform_b200.engine.stateful_sampler import StatefulSampler
    from arctic_platform_b200.engine.worker import EngineWorker
    from arctic_platform_b200.models.reninex import PRESETS
    with pytest.raises(RuntimeError, match="CUDA"):
        StatefulSampler(PRESETS["reninex-tiny"], "cpu")
    for job, match in (("training", "sampling"), ("log_prob", "sampling")):
        with pytest.raises(ValueError, match=match):
            EngineWorker(device="cpu").initialize({"model_name": "reninex-tiny", "job_type": job})


@pytest.mark.parametrize("fault", ["no_bigram_start", "conv_shift", "window:60", "state_reset:70", "no_bias"])
def test_the_oracle_would_show_a_mistake(fault):
    """The inputs of the engine tests are sharp enough: each planted mistake moves some logits far over the tolerance."""
    cfg = H.CONFIGS["mixed-layers"]
    w, toks = H.weights(cfg), H.tokens(cfg, 100)
    good, bad = H.expected(cfg, w, toks), H.expected(cfg, w, toks, (fault,))
    assert H.error(bad, good) > 2 * H.TOL[torch.bfloat16], fault


def test_oracle_retention_equals_the_quadratic_form():
    g = torch.Generator().manual_seed(0)
    q, k, v = (torch.randn(20, 2, n, generator=g, dtype=torch.float64) for n in (6, 6, 5))
    decay = [0.9, 0.5]
    o = oracle.retention(q, k, v, decay)
    i, j = torch.arange(20)[:, None], torch.arange(20)[None]
    for h in range(2):
        w = torch.where(j <= i, decay[h] ** (i - j).clamp(min=0).double(), torch.zeros(()).double())
        assert torch.allclose(((q[:, h] @ k[:, h].t()) * w) @ v[:, h], o[:, h])


@pytest.mark.parametrize("heads,kv", [(4, 2), (3, 1), (5, 5), (6, 2), (1, 1)])
def test_attention_work_items_cover_every_row_and_head_once(heads, kv):
    from arctic_platform_b200.ops.serving import tile_work
    host = np.array([[0, 300, 1, 40], [300, 5, 0, 1000], [305, 129, 2, 0], [434, 128, 3, 7]])
    work = tile_work(host, heads, kv, 17)
    seen = {}
    for en, blocks, g, _, *groups in work.tolist():
        last = 0
        for row, valid, head, keys in (groups[:4], groups[4:]):
            if valid == 0:
                continue
            start, n, _, pos0 = host[en]
            assert head // (heads // kv) == g and keys == pos0 + (row - start) + 1 and row + valid <= start + n
            last = max(last, keys + valid - 1)
            for r in range(row, row + valid):
                seen[r, head] = seen.get((r, head), 0) + 1
        assert blocks == -(-last // 128)
    rows = [r for s, n, _, _ in host.tolist() if n > 16 for r in range(s, s + n)]
    assert seen == {(r, h): 1 for r in rows for h in range(heads)}
    assert (np.diff(work[:, 1]) <= 0).all()


@pytest.mark.parametrize("lens,slices,slots", [([2100, 700, 1, 64], 8, 296), ([500] * 200, 32, 296), ([2], 1, 296),
                                               ([8192], 32, 296), ([257, 31], 4, 40)])
def test_retention_segments_cover_every_long_entry_in_order(lens, slices, slots):
    from arctic_platform_b200.ops.serving import segment_plan
    host = np.array([[0, n, i, 0] for i, n in enumerate(lens)])
    plan = segment_plan(host, slices, slots)
    at, used = {}, set()
    for i, (en, t, n, before, out, last) in enumerate(plan["seg"].tolist()):
        assert t == at.get(en, 0) and n > 0
        at[en] = t + n
        assert last == (at[en] == lens[en]) and (out >= 0) == (before >= 0 and not last)
        assert last or n % 32 == 0
        if before >= 0:
            assert before not in used and (last or out == before + 1)
            used.add(before)
    assert at == {i: n for i, n in enumerate(lens) if n > 1}
    assert used == set(range(plan["states"]))
    for en, base, k, first in plan["chains"].tolist():
        assert k > 1 and plan["seg"][first:first + k, 0].tolist() == [en] * k
        assert plan["seg"][first:first + k, 3].tolist() == list(range(base, base + k))
