"""Titatar without a GPU: configuration, checkpoint names, caches, planning tables, and the oracle's own sharpness."""
import json
import math
import re

import numpy as np
import pytest
import torch

from tests import titatar_helpers as H
from tests import titatar_oracle as oracle


@pytest.mark.parametrize("name", sorted(H.CONFIGS))
def test_config_round_trip_and_tensor_names(name):
    from arctic_platform_b200.models.titatar import TitatarConfig
    cfg = H.CONFIGS[name]
    rc = TitatarConfig.from_dict(json.loads(json.dumps(cfg)))
    assert TitatarConfig.from_dict(rc.to_hf_dict()) == rc and rc.to_hf_dict() == cfg
    w = H.weights(cfg)
    assert sorted(rc.tensor_names()) == sorted(w)
    assert rc.num_parameters() == sum(t.numel() for t in w.values())
    assert rc.num_parameters() - rc.num_parameters(False) == w["embed"].numel() + w["head"].numel()


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
    assert all(torch.equal(a, b) for a, b in zip(model.state_dict().values(), again.state_dict().values()))
    assert all(torch.equal(a, b) for a, b in zip(model.buffers(), again.buffers()))
    for i, s in enumerate(cfg["layers"]):
        if s["type"] == "latent_attention":                          # what is derived from the weights
            m, mix = s["mixer"], again.blocks[i].mixer
            uk = w[f"l{i}.mix.uk"].view(m["heads"], m["dim"], m["kv_rank"])
            assert torch.equal(mix.w_absorb.view(m["heads"], m["kv_rank"], -1)[..., :m["dim"]], uk.transpose(1, 2))
            assert torch.equal(mix.sink32, w[f"l{i}.mix.sink"].float())


def test_fused_padding_stays_zero():
    from arctic_platform_b200.models.titatar import TitatarConfig, TitatarLM
    cfg = H.CONFIGS["odd-sizes"]
    model = TitatarLM(TitatarConfig.from_dict(cfg), "cpu", torch.float32)
    w = H.weights(cfg)
    for n, t in w.items():
        model.load_named_tensor(n, torch.ones_like(t))
    assert sum(float(p.sum()) for p in model.parameters()) == sum(t.numel() for t in w.values())
    for blk in model.blocks:
        for cols in (blk.mixer.in_cols, getattr(blk.mixer, "exp_cols", {})):
            assert all(o % 8 == 0 for o, _ in cols.values())
        assert blk.mixer.w_out.shape[1] % 8 == 0


def test_bad_configurations_and_tensors_are_refused(tmp_path):
    from arctic_platform_b200.models.hf_io import load_hf_checkpoint
    from arctic_platform_b200.models.titatar import TitatarConfig, TitatarLM

    def broken(layer=0, entry={}, mixer={}, router={}, **kw):
        d = json.loads(json.dumps(H.CONFIGS["mixed-layers"]))
        d["layers"][layer].update(entry)
        d["layers"][layer]["mixer"].update(mixer)
        if router:
            d["layers"][layer]["mlp"]["router"].update(router)
        d.update(kw)
        return d

    for bad in (broken(entry={"type": "other"}), broken(1, mixer={"kv_heads": 3}), broken(1, mixer={"rot": {"dims": 64, "base": 9.0}}),
                broken(1, mixer={"rot": {"dims": 3, "base": 9.0}}), broken(0, mixer={"rot": {"dims": 8, "base": 9.0}}),
                broken(0, mixer={"rot": {"dims": 15, "base": 9.0}, "rot_dim": 15}), broken(entry={"mlp": {"kind": "routed", "ff": 8}}),
                broken(1, router={"top": 10}), broken(1, router={"top": 0}), broken(1, router={"experts": 600}),
                broken(1, mixer={"mask": {"size": -1}}), broken(loop={"start": 2, "stop": 2, "times": 1}),
                broken(loop={"start": 2, "stop": 6, "times": 1}), broken(loop={"start": 0, "stop": 1, "times": 0})):
        with pytest.raises(ValueError):
            TitatarConfig.from_dict(bad)
    cfg, w = H.CONFIGS["mixed-layers"], H.weights(H.CONFIGS["mixed-layers"])
    model = TitatarLM(TitatarConfig.from_dict(cfg), "cpu", torch.float32)
    for name, shape in (("embed", (3, 3)), ("l0.mix.dkv", (48, 128)), ("l1.mix.q", (64, 128)), ("l1.mlp.router", (6, 128))):
        with pytest.raises(ValueError):
            model.load_named_tensor(name, torch.zeros(shape))
    for name in ("l3.norm2", "l3.mlp.gate", "l2.mlp.shared.up", "l1.mlp.e6.up", "l0.mlp.router", "l1.mix.sink", "l0.mix.q", "l9.norm1",
                 "nothing"):
        with pytest.raises(KeyError):
            model.load_named_tensor(name, torch.zeros(1))
    w.pop("l1.mlp.e3.up")
    with pytest.raises(KeyError, match="l1.mlp.e3.up"):
        load_hf_checkpoint(model, H.save(cfg, w, tmp_path / "part"))


def test_every_pass_has_a_cache_and_a_latent_layer_keeps_one_row():
    from arctic_platform_b200.engine.stateful_sampler import StateCache
    from arctic_platform_b200.models.titatar import TitatarConfig, TitatarLM
    rc = TitatarConfig.from_dict(H.CONFIGS["mixed-layers"])
    assert rc.layer_runs() == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None), (4, None)]
    model = TitatarLM(rc, "cpu", torch.float32)
    c = StateCache(model.cache_layout(), 6, 2, "cpu", torch.float32)
    assert len(c.k) == 9 and len({id(t) for t in c.k}) == 9
    assert c.k[0].shape == (6, 1, 16, 48 + 16) and c.v[0] is None and c.v[2] is None
    assert c.k[1].shape == (6, 2, 16, 32) and c.v[1].shape == (6, 2, 16, 48)
    c.k[0][2] = 5.0
    c.copy_pages(torch.tensor([2]), torch.tensor([3]))
    assert (c.k[0][3] == 5.0).all() and (c.k[0][4] == 0).all()


def test_presets_resolve_and_are_served_only_on_a_gpu():
    from arctic_platform_b200.engine.stateful_sampler import StatefulSampler
    from arctic_platform_b200.engine.worker import EngineWorker
    from arctic_platform_b200.models import registry
    from arctic_platform_b200.models.config import resolve_config
    cfg = resolve_config("titatar-tiny")
    assert cfg.architecture == "Titatar" and "Titatar" in registry.architectures()
    model = registry.new_model(cfg, "cpu", torch.float32).init_weights(1)
    assert sum(t.numel() for _, t in model.iter_named_tensors()) == cfg.num_parameters()
    with pytest.raises(RuntimeError, match="CUDA"):
        StatefulSampler(cfg, "cpu")
    with pytest.raises(ValueError, match="sampling"):
        EngineWorker(device="cpu").initialize({"model_name": "titatar-tiny", "job_type": "training"})


@pytest.mark.parametrize("dims,base,yarn", [(16, 2000.0, (4.0, 64.0, 8.0, 1.0)), (64, 1e4, (40.0, 4096.0, 32.0, 1.0)), (6, 500.0, None),
                                            (8, 1e6, (1.5, 8.0, 64.0, 32.0)), (32, 100.0, (2.0, 1e6, 2.0, 1.0))])
def test_position_tables(dims, base, yarn):
    from arctic_platform_b200.ops import norm
    rot = {"dims": dims, "base": base}
    if yarn:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    freqs, gain = oracle.frequencies(rot)
    cos, sin = norm.rope_tables(300, dims, base, "cpu", norm.Yarn(*yarn) if yarn else None)
    for i, f in enumerate(freqs):
        assert abs(float(cos[299, i]) - math.cos(299 * f) * gain) < 1e-6 and abs(float(sin[299, i]) - math.sin(299 * f) * gain) < 1e-6


FAULTS = [f for f in re.findall(r"``(\w+)``", oracle.__doc__.split("a set of names")[1])]


@pytest.mark.parametrize("decided", [False, True])
def test_the_oracle_would_show_a_mistake(decided):
    """The inputs of the engine tests are sharp enough: each planted mistake moves some logits far over the tolerance."""
    assert len(FAULTS) > 25
    cfg = H.CONFIGS["mixed-layers"]
    w, toks = H.weights(cfg, decided=decided), H.tokens(cfg, 150)
    good = H.expected(cfg, w, toks)
    assert H.error(oracle.forward(cfg, w, toks, torch.float32)[0], good) < H.TOL[torch.float32] / 10
    for fault in FAULTS:
        if decided and fault == "scores_of_experts":                # the chosen experts differ, their number of weights too
            continue
        assert H.error(H.expected(cfg, w, toks, (fault,)), good) > 2 * H.TOL[torch.bfloat16], fault


def test_oracle_windows_sinks_and_routing():
    seen = oracle.visible(8, 3)
    assert seen.sum(-1).tolist() == [1, 2, 3, 3, 3, 3, 3, 3] and not torch.triu(seen, 1).any()
    s = torch.tensor([[0.5, 2.0], [1.0, -1.0]], dtype=torch.float64)
    p = oracle.sink_softmax(s, torch.ones(2, 2, dtype=torch.bool), torch.tensor(0.0, dtype=torch.float64))
    assert torch.allclose(p, s.exp() / (1 + s.exp().sum(-1, keepdim=True)))
    z = torch.tensor([[1.0, 2.0, 0.0, 1.5]], dtype=torch.float64)
    w = oracle.route(z, torch.tensor([0.0, -1.0, 0.0, 0.0], dtype=torch.float64), 2)
    soft = torch.softmax(z, -1)
    assert w[0, 1] == 0 and w[0, 2] == 0 and torch.allclose(w[0, [0, 3]], soft[0, [0, 3]])


def test_runs_of_short_entries():
    from arctic_platform_b200.ops.serving import entry_runs
    host = np.array([[0, 1, 0, 5], [1, 40, 1, 0], [41, 2, 2, 9], [43, 1, 3, 7], [44, 90, 4, 0]])
    assert entry_runs(host, 5, 16) == [(0, 1), (2, 4)] and entry_runs(host, 5, 100) == [(0, 5)] and entry_runs(None, 7, 1) == [(0, 7)]


@pytest.mark.parametrize("window", [0, 1, 50, 128, 200, 4096])
@pytest.mark.parametrize("heads,kv", [(4, 2), (3, 1), (5, 5)])
def test_attention_work_items_cover_every_row_once_and_walk_all_visible_keys(heads, kv, window):
    from arctic_platform_b200.ops.serving import PAGE, flash_tiles
    host = np.array([[0, 300, 1, 40], [300, 5, 0, 1000], [305, 129, 2, 0], [434, 128, 3, 7], [562, 17, 4, 2047]])
    work = flash_tiles(host, heads, kv, 17, window, np.arange(5) * 10000)
    seen, keys = {}, []
    for en, g, k0, base, *tiles in work.tolist():
        start, n, _, pos0 = host[en]
        assert k0 % PAGE == 0 and base == en * 10000 and tiles[1] > 0
        ends = []
        for row, valid, head, pos in (tiles[:4], tiles[4:]):
            if not valid:
                continue
            assert head // (heads // kv) == g and 0 < valid <= 128 and row + valid <= start + n and pos - pos0 == row - start
            assert k0 <= max(0, pos - window + 1 if window else 0)
            ends.append(pos + valid)
            for r in range(row, row + valid):
                seen[r, head] = seen.get((r, head), 0) + 1
        keys.append(max(ends) - k0)
    rows = [r for s, n, _, _ in host.tolist() if n > 16 for r in range(s, s + n)]
    assert seen == {(r, h): 1 for r in rows for h in range(heads)}
    assert (np.diff(keys) <= 0).all()
    assert flash_tiles(host, heads, kv, 1000, window).shape == (0, 12)


def test_contexts_are_expanded_in_groups_of_bounded_size():
    from arctic_platform_b200.ops.serving import PAGE, expansion_plan
    host = np.array([[0, 40, 1, 100], [40, 3, 0, 900], [43, 60, 2, 0], [103, 64, 3, 1000]])
    plans = expansion_plan(host, 2, 33, 256)
    assert [sorted({int(e) for e in p["pages"][:, 0]}) for p in plans] == [[0, 2], [3]]
    for p in plans:
        rows = p["pages"][:, 2]
        assert rows.tolist() == list(range(0, len(rows) * PAGE, PAGE)) and (p["pages"][:, 3] == PAGE).all()
        for en, _, _, base, *_ in p["work"].tolist():
            mine = p["pages"][p["pages"][:, 0] == en]
            assert mine[0, 2] == base and mine[:, 1].tolist() == list(range(-(-(host[en, 3] + host[en, 1]) // PAGE)))


def test_splits_of_wide_rows():
    from arctic_platform_b200.ops.serving import MAX_WIDE_SPLITS, wide_splits
    assert wide_splits(1, 148) == MAX_WIDE_SPLITS and wide_splits(128, 148) == 1 and wide_splits(64, 148) == 2
    assert all(1 <= wide_splits(n, 148) <= MAX_WIDE_SPLITS for n in range(1, 2000, 37))
