"""Rigulorn without a GPU: configuration, checkpoint names, shared caches, work tables, and the oracle's own sharpness."""
import json

import numpy as np
import pytest
import torch

from tests import rigulorn_helpers as H
from tests import rigulorn_oracle as oracle


@pytest.mark.parametrize("name", sorted(H.CONFIGS))
def test_config_round_trip_and_tensor_names(name):
    from arctic_platform_b200.models.rigulorn import RigulornConfig
    cfg = H.CONFIGS[name]
    rc = RigulornConfig.from_dict(json.loads(json.dumps(cfg)))
    assert RigulornConfig.from_dict(rc.to_hf_dict()) == rc and rc.to_hf_dict() == cfg
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
    assert all(torch.equal(a, b) for a, b in zip(model.parameters(), again.parameters()))
    for i, s in enumerate(cfg["layers"]):
        if s["type"] == "attention":
            lam = oracle.map_weight(*(w[f"l{i}.mix.{n}"].float() for n in ("lq1", "lk1", "lq2", "lk2")), s["mixer"]["diff"])
            assert abs(float(again.blocks[i].mixer.lam) - float(lam)) < 1e-5


def test_fused_padding_stays_zero():
    from arctic_platform_b200.models.rigulorn import RigulornConfig, RigulornLM
    cfg = H.CONFIGS["odd-sizes"]
    model = RigulornLM(RigulornConfig.from_dict(cfg), "cpu", torch.float32)
    for n, t in H.weights(cfg).items():
        model.load_named_tensor(n, torch.ones_like(t))
    for blk in model.blocks:
        used = torch.zeros(blk.mixer.w_in.shape[0], dtype=torch.bool)
        for o, n in blk.mixer.in_cols.values():
            assert o % 8 == 0
            used[o:o + n] = True
        assert (blk.mixer.w_in[used] == 1).all() and (blk.mixer.w_in[~used] == 0).all()
        out = blk.mixer.w_out
        n = blk.mixer.m.inner if hasattr(blk.mixer.m, "inner") else blk.mixer.n_out
        assert out.shape[1] % 8 == 0 and (out[:, :n] == 1).all() and (out[:, n:] == 0).all()


def test_bad_configurations_and_tensors_are_refused(tmp_path):
    from arctic_platform_b200.models.hf_io import load_hf_checkpoint
    from arctic_platform_b200.models.rigulorn import RigulornConfig, RigulornLM

    def broken(layer=0, entry={}, mixer={}, **kw):
        d = json.loads(json.dumps(H.CONFIGS["mixed-layers"]))
        d["layers"][layer].update(entry)
        d["layers"][layer]["mixer"].update(mixer)
        d.update(kw)
        return d

    for bad in (broken(entry={"type": "other"}), broken(mixer={"kv_heads": 3}), broken(mixer={"rot": {"dims": 64, "base": 1.0}}),
                broken(mixer={"rot": {"dims": 3, "base": 1.0}}), broken(entry={"mlp": {"kind": "routed", "ff": 8}}),
                broken(1, mixer={"groups": 4}), broken(1, mixer={"norm_groups": 5}), broken(1, mixer={"conv": 0}),
                broken(3, mixer={"kv_from": 1}), broken(3, mixer={"kv_from": 3}), broken(3, mixer={"kv_from": 4}),
                broken(3, mixer={"vdim": 40}), broken(2, mixer={"kv_from": 3}), broken(streams=0)):
        with pytest.raises(ValueError):
            RigulornConfig.from_dict(bad)
    cfg, w = H.CONFIGS["mixed-layers"], H.weights(H.CONFIGS["mixed-layers"])
    model = RigulornLM(RigulornConfig.from_dict(cfg), "cpu", torch.float32)
    for name, shape in (("embed", (3, 3)), ("l1.mix.in", (5, 128)), ("l0.mix.q", (128, 128))):
        with pytest.raises(ValueError):
            model.load_named_tensor(name, torch.zeros(shape))
    for name in ("l2.norm2", "l2.hc2.in", "l3.mix.k", "l3.mix.v", "l1.mix.q", "l0.mix.conv", "l9.norm1", "l2.mlp.gate", "nothing"):
        with pytest.raises(KeyError):
            model.load_named_tensor(name, torch.zeros(1))
    w.pop("l0.hc1.mix")
    with pytest.raises(KeyError, match="l0.hc1.mix"):
        load_hf_checkpoint(model, H.save(cfg, w, tmp_path / "part"))


def test_borrowed_keys_share_one_cache():
    from arctic_platform_b200.engine.stateful_sampler import StateCache
    from arctic_platform_b200.models.rigulorn import RigulornConfig, RigulornLM
    model = RigulornLM(RigulornConfig.from_dict(H.CONFIGS["wide-heads"]), "cpu", torch.float32)
    c = StateCache(model.cache_layout(), 6, 2, "cpu", torch.float32)
    assert c.k[1] is c.k[2] is c.k[3] and c.v[1] is c.v[3] and c.k[0] is None and c.state[2] is None
    assert c.k[1].shape == (6, 4, 16, 128) and c.state[0].shape == (2, 2, 128, 136) and c.conv[0] is None     # one tap
    assert c.num_bytes() == 4 * (c.k[1].numel() + c.v[1].numel() + c.state[0].numel()) + 4 * 4
    c.k[1][2] = 5.0
    c.copy_pages(torch.tensor([2]), torch.tensor([3]))
    assert (c.k[3][3] == 5.0).all() and (c.k[3][4] == 0).all()


def test_presets_resolve_and_are_served_only_on_a_gpu():
    from arctic_platform_b200.engine.stateful_sampler import StatefulSampler
    from arctic_platform_b200.engine.worker import EngineWorker
    from arctic_platform_b200.models import registry
    from arctic_platform_b200.models.config import resolve_config
    cfg = resolve_config("rigulorn-tiny")
    assert cfg.architecture == "Rigulorn" and "Rigulorn" in registry.architectures()
    model = registry.new_model(cfg, "cpu", torch.float32).init_weights(1)
    assert sum(t.numel() for _, t in model.iter_named_tensors()) == cfg.num_parameters()
    with pytest.raises(RuntimeError, match="CUDA"):
        StatefulSampler(cfg, "cpu")
    with pytest.raises(ValueError, match="sampling"):
        EngineWorker(device="cpu").initialize({"model_name": "rigulorn-tiny", "job_type": "training"})


FAULTS = ["chunk_early", "chunk_late", "no_chunks", "chunks_from:7", "no_softcap", "one_map", "no_diff_scale", "half_rotation",
          "own_keys", "conv_shift", "state_reset:70", "late_gate", "one_norm", "no_limit", "mix_transposed", "in_order_mix"]


@pytest.mark.parametrize("fault", FAULTS)
def test_the_oracle_would_show_a_mistake(fault):
    """The inputs of the engine tests are sharp enough: each planted mistake moves some logits far over the tolerance."""
    cfg = H.CONFIGS["mixed-layers"]
    w, toks = H.weights(cfg), H.tokens(cfg, 150)
    good, bad = H.expected(cfg, w, toks), H.expected(cfg, w, toks, (fault,))
    assert H.error(bad, good) > 2 * H.TOL[torch.bfloat16], fault


def test_oracle_state_space_equals_the_quadratic_form():
    g = torch.Generator().manual_seed(0)
    T, Hh, G, N, E = 20, 4, 2, 6, 5
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    x, B, C, dt, A, D = rnd(T, Hh, E), rnd(T, G, N), rnd(T, G, N), rnd(T, Hh).abs(), rnd(Hh), rnd(Hh)
    y = oracle.state_space(x, B, C, dt, A, D)
    for h in range(Hh):
        cum = torch.cumsum(-torch.exp(A[h]) * dt[:, h], 0)
        w = torch.exp(cum[:, None] - cum[None]) * dt[None, :, h] * (C[:, h // 2] @ B[:, h // 2].t())
        assert torch.allclose(torch.tril(w) @ x[:, h] + D[h] * x[:, h], y[:, h])


def test_oracle_streams_and_chunks():
    g = torch.Generator().manual_seed(1)
    x, y, mix, out = (torch.randn(*s, generator=g) for s in ((3, 5, 4), (5, 4), (3, 3), (3,)))
    new = oracle.streams_out(x, y, mix, out)
    assert torch.allclose(new, torch.einsum("st,snw->tnw", mix, x) + out[:, None, None] * y, atol=1e-5)
    seen = oracle.chunk_visible(10, 4)
    assert seen.sum(-1).tolist() == [1, 2, 3, 4, 1, 2, 3, 4, 1, 2] and not torch.triu(seen, 1).any()


@pytest.mark.parametrize("chunk", [0, 1, 50, 128, 200, 4096])
@pytest.mark.parametrize("heads,kv", [(4, 2), (3, 1), (5, 5)])
def test_attention_work_items_cover_every_row_once_and_stay_in_a_chunk(heads, kv, chunk):
    from arctic_platform_b200.ops.serving import PAGE, chunk_tiles
    host = np.array([[0, 300, 1, 40], [300, 5, 0, 1000], [305, 129, 2, 0], [434, 128, 3, 7], [562, 17, 4, 2047]])
    work = chunk_tiles(host, heads, kv, 17, chunk)
    seen, keys = {}, []
    for en, g, head, row, valid, pos, first_page, first in work.tolist():
        start, n, _, pos0 = host[en]
        assert head // (heads // kv) == g and 0 < valid <= 128 and row + valid <= start + n and pos - pos0 == row - start
        assert first == (pos // chunk * chunk if chunk else 0) and first_page == first // PAGE * PAGE
        assert not chunk or (pos + valid - 1) // chunk == pos // chunk
        keys.append(pos + valid - first_page)
        for r in range(row, row + valid):
            seen[r, head] = seen.get((r, head), 0) + 1
    rows = [r for s, n, _, _ in host.tolist() if n > 16 for r in range(s, s + n)]
    assert seen == {(r, h): 1 for r in rows for h in range(heads)}
    assert (np.diff(keys) <= 0).all()
    assert chunk_tiles(host, heads, kv, 1000, chunk).shape == (0, 8)


def test_row_tiles_skip_single_tokens():
    from arctic_platform_b200.ops.serving import row_tiles
    host = np.array([[0, 33, 0, 0], [33, 1, 1, 9], [34, 16, 2, 0]])
    assert row_tiles(host, 16).tolist() == [[0, 0], [0, 16], [0, 32], [2, 0]]


def test_a_serving_process_compiles_only_its_own_kernels():
    from arctic_platform_b200 import _build
    from arctic_platform_b200.models import registry
    own = {a: set(registry.kernel_sources(a)) for a in registry.architectures()}
    names = {p.stem for p in _build.cuda_sources()}
    assert all(k and k <= names and not k & set(_build.SERVE_STEMS) for k in own.values())
    assert not own["Rigulorn"] & own["Reninex"] and set(_build.SERVE_STEMS) <= names
    assert _build.serve_lib("Rigulorn") != _build.serve_lib("Reninex")
