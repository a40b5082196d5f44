"""Meronex without a GPU: configuration, checkpoint names, caches, planning tables, and the oracle's own sharpness."""
import json
import re

import numpy as np
import pytest
import torch

from tests import meronex_helpers as H
from tests import meronex_oracle as oracle


def _rank_surplus(cfg, w):
    """Weights that the configuration cannot know: the checkpoint's rank against the default."""
    from arctic_platform_b200.models.meronex import DEFAULT_RANK
    out = 0
    for n, t in w.items():
        if n.endswith(".right.w1"):
            out += (t.shape[0] - DEFAULT_RANK) * (t.shape[1] + w[n[:-1] + "2"].shape[0])
    return out


@pytest.mark.parametrize("name", sorted(H.CONFIGS))
def test_config_round_trip_and_tensor_names(name):
    from arctic_platform_b200.models.meronex import MeronexConfig
    cfg = H.CONFIGS[name]
    rc = MeronexConfig.from_dict(json.loads(json.dumps(cfg)))
    assert MeronexConfig.from_dict(rc.to_hf_dict()) == rc and rc.to_hf_dict() == cfg
    w = H.weights(cfg)
    assert sorted(rc.tensor_names()) == sorted(w)
    assert rc.num_parameters() + _rank_surplus(cfg, w) == sum(t.numel() for t in w.values())
    assert rc.num_parameters() - rc.num_parameters(False) == w["embed"].numel() + w["head"].numel()
    assert rc.flops_per_token(100) > 2 * w["head"].numel()


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


def test_fused_padding_stays_zero():
    from arctic_platform_b200.models.meronex import MeronexConfig, MeronexLM
    cfg = H.CONFIGS["odd-sizes"]
    model = MeronexLM(MeronexConfig.from_dict(cfg), "cpu", torch.float32)
    w = H.weights(cfg)
    for n, t in w.items():
        model.load_named_tensor(n, torch.ones_like(t))
    assert sum(float(p.sum()) for p in model.parameters()) == sum(t.numel() for t in w.values())
    for blk in model.blocks:
        assert all(o % 8 == 0 for o, _ in blk.mixer.in_cols.values())
        assert all(o % 8 == 0 for o, _ in blk.mlp.z_cols.values())


def test_a_checkpoint_decides_the_rank_of_the_decay():
    from arctic_platform_b200.models.meronex import DEFAULT_RANK, MeronexConfig, MeronexLM
    cfg = H.CONFIGS["wide-heads"]
    model = MeronexLM(MeronexConfig.from_dict(cfg), "cpu", torch.float32)
    mixer = model.blocks[0].mixer
    assert mixer.rank == DEFAULT_RANK
    model.load_named_tensor("l0.mix.right.r", torch.ones(128, 256))
    for rank in (5, 200):
        model.load_named_tensor("l0.mix.right.w2", torch.full((128, rank), 2.0))
        model.load_named_tensor("l0.mix.right.w1", torch.full((rank, 256), 3.0))
        assert mixer.rank == rank and mixer.w_rank.shape == (128, -(-rank // 8) * 8)
        assert (mixer.w_shift.shape[0] - 4 * mixer.step) % 128 == 0 and (mixer.place("right.r") == 1).all()
        assert float(mixer.w_shift.sum()) == 128 * 256 + 3 * rank * 256 and float(mixer.w_rank.sum()) == 2 * rank * 128
    with pytest.raises(ValueError):
        model.load_named_tensor("l0.mix.right.w1", torch.zeros(200, 255))


def test_bad_configurations_and_tensors_are_refused(tmp_path):
    from arctic_platform_b200.models.hf_io import load_hf_checkpoint
    from arctic_platform_b200.models.meronex import MeronexConfig, MeronexLM

    def broken(layer=0, entry={}, mixer={}, left={}, router={}, **kw):
        d = json.loads(json.dumps(H.CONFIGS["mixed-layers"]))
        d["layers"][layer].update(entry)
        d["layers"][layer]["mixer"].update(mixer)
        if left:
            d["layers"][layer]["mixer"]["left"].update(left)
        if router:
            d["layers"][layer]["mlp"]["router"].update(router)
        d.update(kw)
        return d

    for bad in (broken(entry={"type": "other"}), broken(left={"kv_heads": 3}), broken(left={"rot": {"dims": 64, "base": 9.0}}),
                broken(left={"rot": {"dims": 3, "base": 9.0}}), broken(2, mixer={"kv_heads": 3}), broken(2, mixer={"conv": 0}),
                broken(entry={"mlp": {"kind": "dense", "ff": 8}}), broken(router={"top": 7}), broken(router={"top": 0}),
                broken(router={"experts": 600}), broken(norm={"eps": 1e-5, "groups": 3})):
        with pytest.raises(ValueError):
            MeronexConfig.from_dict(bad)
    cfg, w = H.CONFIGS["mixed-layers"], H.weights(H.CONFIGS["mixed-layers"])
    model = MeronexLM(MeronexConfig.from_dict(cfg), "cpu", torch.float32)
    for name, shape in (("embed", (3, 3)), ("l0.mix.left.v", (48, 128)), ("l1.mix.q", (64, 128)), ("l1.mlp.router", (5, 128)),
                        ("l2.mix.q.conv", (64, 4)), ("l0.mix.right.u", (72,)), ("l0.rg1", (128, 64))):
        with pytest.raises(ValueError):
            model.load_named_tensor(name, torch.zeros(shape))
    for name in ("l2.norm2", "l2.rg2", "l2.rg2.b", "l2.mlp.router", "l1.mlp.e6.up", "l0.mix.q", "l1.mix.left.q", "l1.mix.b", "l2.mix.i.b", "l2.mix.g.conv",
                 "l0.mix.right.mu.x", "l0.mix.right.mu.", "l0.mix.rg", "l0.mlp.rg", "l0.rg1.c", "l0.rg3", "l9.norm1", "nothing"):
        with pytest.raises(KeyError):
            model.load_named_tensor(name, torch.zeros(1))
    w.pop("l1.mlp.e3.up")
    with pytest.raises(KeyError, match="l1.mlp.e3.up"):
        load_hf_checkpoint(model, H.save(cfg, w, tmp_path / "part"))


def test_what_a_layer_keeps_per_sequence():
    from arctic_platform_b200.engine.stateful_sampler import StateCache
    from arctic_platform_b200.models.meronex import MeronexConfig, MeronexLM
    model = MeronexLM(MeronexConfig.from_dict(H.CONFIGS["mixed-layers"]), "cpu", torch.float32)
    c = StateCache(model.cache_layout(), 6, 3, "cpu", torch.bfloat16)
    # attention and time mixing side by side
    assert c.k[0].shape == (6, 2, 16, 32) and c.v[0].shape == (6, 2, 16, 48) and c.state[0].shape == (3, 3, 24, 24)
    assert c.conv[0].shape == (3, 2, 1, 128) and c.aux[0] is None
    # matrix memory, delta rule
    assert c.k[1] is None and c.state[1].shape == (3, 3, 32, 48) and c.aux[1].shape == (3, 3, 33) and c.conv[1] is None
    assert c.state[2].shape == (3, 4, 32, 40) and c.conv[2].shape == (3, 2, 2, 2 * 64 + 160) and c.aux[2] is None
    assert all(t.dtype == torch.float32 for t in c.state + c.aux + c.conv if t is not None)
    for t in (c.state[1], c.aux[1], c.conv[2]):
        t[0] = 5.0
    c.copy_slots(torch.tensor([0]), torch.tensor([2]))
    assert all((t[2] == 5.0).all() and (t[1] == 0).all() for t in (c.state[1], c.aux[1], c.conv[2]))
    one_tap = MeronexLM(MeronexConfig.from_dict(H.CONFIGS["plain"]), "cpu", torch.float32)
    assert StateCache(one_tap.cache_layout(), 1, 1, "cpu", torch.float32).conv[0] is None


def test_presets_resolve_and_are_served_only_on_a_gpu():
    from arctic_platform_b200 import _build
    from arctic_platform_b200.engine.stateful_sampler import StatefulSampler
    from arctic_platform_b200.engine.worker import EngineWorker
    from arctic_platform_b200.models import registry
    from arctic_platform_b200.models.config import resolve_config
    cfg = resolve_config("meronex-tiny")
    assert cfg.architecture == "Meronex" and "Meronex" in registry.architectures()
    assert all((_build.CSRC / f"{s}.cu").is_file() for s in registry.kernel_sources("Meronex"))
    model = registry.new_model(cfg, "cpu", torch.float32).init_weights(1)
    assert sum(t.numel() for _, t in model.iter_named_tensors()) == cfg.num_parameters()
    with pytest.raises(RuntimeError, match="CUDA"):
        StatefulSampler(cfg, "cpu")
    with pytest.raises(ValueError, match="sampling"):
        EngineWorker(device="cpu").initialize({"model_name": "meronex-tiny", "job_type": "training"})


def test_parameter_block_of_the_recurrent_kernels_matches_its_declaration():
    """The fields and their order, read from the header."""
    from arctic_platform_b200 import _build
    from arctic_platform_b200.ops.serving import _RecurrentParams
    text = (_build.CSRC / "recurrent.cuh").read_text()
    body = re.sub(r"//[^\n]*", "", text[text.index("struct RecurrentParams {"):].split("};")[0].split("{", 1)[1])
    want = [("start", "p"), ("len", "p"), ("slot", "p"), ("pos0", "p")]                # ServeEntries
    for decl in body.split(";")[1:]:
        decl = decl.strip()
        if not decl:
            continue
        kind, names = re.match(r"((?:const )?(?:void|float|int|long long)\*?)\s+(.*)", decl, re.S).groups()
        code = "p" if "*" in kind else {"int": "i", "float": "f", "long long": "l"}[kind]
        want += [(n.strip(), code) for n in names.split(",")]
    codes = {_RecurrentParams._p: "p", _RecurrentParams._i: "i", _RecurrentParams._f: "f", _RecurrentParams._l: "l"}
    assert [(n, codes[t]) for n, t in _RecurrentParams._fields_] == want


FAULTS = [f for f in re.findall(r"``(\w+)``", oracle.__doc__.split("a deliberate mistake")[1])]
# the head's norm takes the scale of a memory's output away: these show through the norm's eps only (and in the mechanism alone)
SCALE = ["no_floor", "signed_denominator", "unscaled_q"]


def test_the_oracle_would_show_a_mistake():
    """The inputs of the engine tests are sharp enough: each planted mistake moves some logits far over the tolerance."""
    assert len(FAULTS) == 39
    cfg = H.CONFIGS["mixed-layers"]
    w, toks = H.weights(cfg), H.tokens(cfg, 150)
    good = H.expected(cfg, w, toks)
    assert H.error(oracle.forward(cfg, w, toks, torch.float32)[0], good) < H.TOL[torch.float32] / 10
    for fault in FAULTS:
        if fault not in SCALE:
            assert H.error(H.expected(cfg, w, toks, (fault,)), good) > 2 * H.TOL[torch.bfloat16], fault


def test_the_memory_inputs_show_its_scale():
    g = torch.Generator().manual_seed(0)
    q, k, v = (torch.randn(60, 2, 16, generator=g, dtype=torch.float64) for _ in range(3))
    li, lf = oracle.memory_gates(torch.randn(60, 2, generator=g, dtype=torch.float64) * 3 - 2, torch.randn(60, 2, generator=g, dtype=torch.float64) * 3, 6.0)
    good = oracle.rms(oracle.matrix_memory(q / 4, k, v, li, lf), 0.5)
    for fault in ("no_floor", "signed_denominator"):
        bad = oracle.rms(oracle.matrix_memory(q / 4, k, v, li, lf, (fault,)), 0.5)
        assert float((bad - good).abs().max()) > 0.2, fault
    assert float((oracle.rms(oracle.matrix_memory(q, k, v, li, lf), 0.5) - good).abs().max()) > 0.2


def test_recurrences_against_their_closed_forms():
    g = torch.Generator().manual_seed(1)
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    T, D, E = 9, 4, 3
    q, k, v = rnd(T, 1, D), rnd(T, 1, D), rnd(T, 1, E)
    # memory: weights exp(sum of log forget gates + log input gate) over the past
    li, lf = rnd(T, 1), -rnd(T, 1).abs()
    F = lf.cumsum(0)[:, 0]
    a = ((q[:, 0] @ k[:, 0].t()) * torch.exp(F[:, None] - F[None] + li[None, :, 0])).tril()
    den, m = a.sum(-1).abs(), torch.stack([max([F[t]] + [F[t] - F[j] + li[j, 0] for j in range(t + 1)]) for t in range(T)])
    want = (a @ v[:, 0]) / (torch.maximum(den, torch.ones(())) + 1e-6 * torch.exp(m))[:, None]
    assert torch.allclose(oracle.matrix_memory(q, k, v, li, lf)[:, 0], want)
    # time mixing: products of the decays between the tokens, a bonus for the current one
    w, u = torch.rand(T, 1, D, generator=g, dtype=torch.float64), rnd(1, D)
    for t in range(T):
        want = (q[t, 0] * u[0] * k[t, 0]).sum() * v[t, 0]
        for j in range(t):
            want = want + (q[t, 0] * k[j, 0] * w[j + 1:t, 0].prod(0)).sum() * v[j, 0]
        assert torch.allclose(oracle.channel_decay_recurrence(q, k, v, w, u)[t, 0], want)
    # delta rule with beta 1 and no decay: the state maps the last key to its value
    kn = k / k.norm(dim=-1, keepdim=True)
    one = torch.ones(T, 1, dtype=torch.float64)
    assert torch.allclose(oracle.delta_rule(kn, kn, v, one, one), v)


def test_chunks_of_long_entries():
    from arctic_platform_b200.ops.serving import first_tiles, row_tiles, segment_chunks, segment_plan
    host = np.array([[0, 1, 0, 5], [1, 40, 1, 0], [41, 2, 2, 9], [43, 1, 3, 7], [44, 96, 4, 0]])
    tiles, heads = row_tiles(host, 32), first_tiles(host, 32)
    assert tiles.tolist() == [[1, 0], [1, 32], [2, 0], [4, 0], [4, 32], [4, 64]]
    assert heads.tolist() == [[1, 0], [2, 2], [4, 3]]
    assert all(tiles[at].tolist() == [en, 0] for en, at in heads.tolist())
    host = np.array([[0, 2000, 0, 0], [2000, 1, 1, 4], [2001, 700, 2, 16]])
    plan, tiles = segment_plan(host, 1, 296), row_tiles(host, 32)
    at = segment_chunks(host, plan["seg"])
    assert len(at) == len(plan["seg"]) > 2
    for (en, t, *_), i in zip(plan["seg"].tolist(), at.tolist()):
        assert tiles[i].tolist() == [en, t]
