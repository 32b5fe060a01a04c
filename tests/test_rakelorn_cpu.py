"""Rakelorn without a GPU: the oracle's mechanisms against hand computation, the configuration, the weight layout, the states
beside the cache, the registry and the command line."""
import json
import math

import pytest
import torch

from mojo_linuxperiments_b200.models import layered_config as LC
from mojo_linuxperiments_b200.models import layered_weights as LW
from mojo_linuxperiments_b200.models import registry
from mojo_linuxperiments_b200.models.config import RuntimeConfig
from mojo_linuxperiments_b200.models.kvcache import KVState
from mojo_linuxperiments_b200.ops import dense as D
from mojo_linuxperiments_b200.ops import latent as LT
from mojo_linuxperiments_b200.oracle import rakelorn as R

F64 = torch.float64


def test_oracle_norm_and_shift_by_hand():
    x = torch.tensor([[3.0, 4.0], [0.0, 1e-3]], dtype=F64)
    y = R.scalar_norm(x, 2.0, 1e-2)
    assert y[0].tolist() == pytest.approx([6 / math.sqrt(12.5 + 0.01), 8 / math.sqrt(12.5 + 0.01)])
    assert y[1, 1].item() == pytest.approx(2e-3 / math.sqrt(5e-7 + 0.01))
    h = torch.tensor([[1.0, 2.0], [3.0, 5.0], [-1.0, 0.0]], dtype=F64)
    got = R.token_shift(h, torch.tensor([0.25, 1.0], dtype=F64))
    assert got.tolist() == [[0.75, 0.0], [2.5, 2.0], [0.0, 5.0]]        # row 2 leans on row 1 as it was, not as it became


def test_oracle_rotation_by_hand():
    x = torch.arange(1.0, 5.0, dtype=F64).view(1, 4)
    y = R.rotate_pairs(x, torch.tensor([3]), 100.0, 4)[0].tolist()
    c, s = math.cos(3.0), math.sin(3.0)
    assert y[:2] == pytest.approx([c - 2 * s, 2 * c + s])
    c, s = math.cos(0.3), math.sin(0.3)
    assert y[2:] == pytest.approx([3 * c - 4 * s, 4 * c + 3 * s])


def test_oracle_recurrence_by_hand():
    assert R.mingru_candidate(torch.tensor([0.0, 2.0, -1.0], dtype=F64)).tolist() == pytest.approx([0.5, 2.5, 1 / (1 + math.e)])
    z = torch.tensor([[0.5], [1.0], [0.0], [0.25]], dtype=F64)
    c = torch.tensor([[4.0], [3.0], [9.0], [-1.0]], dtype=F64)
    assert R.mingru_states(z, c).flatten().tolist() == [2.0, 3.0, 3.0, 0.75 * 3 - 0.25]


def test_oracle_routing_by_hand():
    # softmax of log p is p; outputs 0 1 | 2 3 | 4 5
    p = torch.tensor([[0.30, 0.05, 0.20, 0.25, 0.08, 0.12]], dtype=F64)
    corr = torch.tensor([0.0, 0.0, 0.0, 0.0, 0.3, 0.0], dtype=F64)
    i, w = R.route(p.log(), corr, {"groups": {"count": 3, "keep": 2}, "top": 3, "scale": 2.0})
    # best of the groups: 0.30, 0.25, 0.38 -> the middle group is out although its 0.25 and 0.20 beat what is left
    assert i.tolist() == [[4, 0, 5]] and w[0].tolist() == pytest.approx([0.16, 0.6, 0.24])
    i, w = R.route(p.log(), corr - 5.0, {"top": 2, "scale": 1.0})              # negative choice scores, no groups
    assert i.tolist() == [[4, 0]] and w[0].tolist() == pytest.approx([0.08, 0.30])
    h = torch.tensor([[1.0, -2.0]], dtype=F64)
    one = torch.eye(2, dtype=F64)
    mlp = {"router": torch.zeros((3, 2), dtype=F64), "correction": torch.tensor([0.0, 1.0, 2.0], dtype=F64),
           "e0.up": one, "e0.down": one, "e1.up": 3 * one, "e1.down": 2 * one}
    out = R.mixture(h, mlp, {"experts": 2, "identity": 1, "top": 2, "scale": 1.5})
    assert out[0].tolist() == pytest.approx([0.5 * 1 + 0.5 * 18, 0.5 * -2])    # identity + the second expert, a third each times 1.5


def test_oracle_attention_sees_itself_and_the_past():
    g = torch.Generator().manual_seed(0)
    m = {"heads": 2, "dim": 4, "rot_dim": 2, "vdim": 3, "kv_rank": 5, "q_rank": 6, "scale": 0.02, "rot": {"base": 10.0, "dims": 2}}
    shapes = {"dq": (6, 7), "dq.norm": (6,), "uq": (12, 6), "dkv": (7, 7), "dkv.norm": (5,), "uk": (8, 5), "uv": (6, 5), "g": (2, 7), "o": (7, 6)}
    mix = {k: torch.randn(s, generator=g, dtype=F64) for k, s in shapes.items()}
    h = torch.randn((9, 7), generator=g, dtype=F64)
    y = R.latent_attention(h, mix, m, 1e-6)
    k = h.clone()
    k[5] += 1
    z = R.latent_attention(k, mix, m, 1e-6)
    assert torch.allclose(z[:5], y[:5], atol=1e-12) and (z[5:] - y[5:]).abs().amax(-1).min() > 1e-4
    # a single token attends to itself alone: its value, gated
    v = (R.rms(h[:1] @ mix["dkv"][:5].t(), 1e-6) * mix["dkv.norm"]) @ mix["uv"].t()
    gate = torch.sigmoid(h[:1] @ mix["g"].t()).repeat_interleave(3, 1)
    assert torch.allclose(R.latent_attention(h[:1], mix, m, 1e-6), (v * gate) @ mix["o"].t(), atol=1e-12)


def test_schedule_and_runs_agree():
    base = LC.tiny_rakelorn()
    for loop in (None, LC.Loop(0, 2, 3), LC.Loop(1, 2, 1), LC.Loop(2, 4, 4), LC.Loop(0, 4, 2)):
        cfg = LC.LayeredConfig("Rakelorn", 10, 8, base.layers, loop=loop)
        assert [(r.layer, r.step) for r in cfg.runs] == R.schedule(cfg.to_dict())
        assert not any(r.add_embedding for r in cfg.runs)
        assert len(cfg.cache_layout(RuntimeConfig())) == len(cfg.state_layout()) == len(cfg.runs)
        assert sum(r.step is not None for r in cfg.runs) == (loop.times if loop else 0)


def test_config_round_trip_defaults_and_rejections():
    cfg = LC.tiny_rakelorn()
    assert LC.LayeredConfig.from_json(cfg.to_json()) == cfg
    d = cfg.to_dict()
    assert [l["type"] for l in d["layers"]] == ["latent_attention", "mingru", "latent_attention", "mingru"] and d["layers"][1]["mlp"] is None
    assert "residual_mult" not in d and d["layers"][0]["mlp"]["router"]["groups"] == {"count": 3, "keep": 2}
    for path, value in [(("layers", 0, "type"), "convolution"), (("layers", 0, "mlp", "kind"), "routed"), (("architecture",), "Else"),
                        (("loop", "stop"), 9), (("layers", 0, "mixer", "rot", "dims"), 15), (("layers", 0, "mixer", "rot", "dims"), 18),
                        (("layers", 0, "mlp", "router", "groups", "count"), 4), (("layers", 0, "mlp", "router", "groups", "keep"), 5),
                        (("layers", 3, "mlp", "router", "top"), 6)]:
        bad = json.loads(json.dumps(d))
        at = bad
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(ValueError):
            LC.LayeredConfig.from_dict(bad)
    # what a model may leave out: loop, groups, identity experts, the router's factor
    d.pop("loop")
    r = d["layers"][0]["mlp"]["router"]
    r.pop("groups"), r.pop("identity"), r.pop("scale")
    m = LC.LayeredConfig.from_dict(d)
    assert m.loop is None and m.layers[0].mlp == LC.MoE(6, 3, 112)


def test_weight_layout():
    a = LC.LatentSpec(3, 20, 6, 12, 18, 28, 0.3, LC.Rotary(100.0, 6))
    cfg = LC.LayeredConfig("Rakelorn", 19, 22, (LC.LayerSpec(a, LC.MoE(3, 2, 9, 1.0, 1, 2, 1)), LC.LayerSpec(LC.MinGRUSpec(13), None)), loop=LC.Loop(0, 1, 2))
    t = LW.init_master(cfg, 1)
    assert set(t) == set(LW.tensor_shapes(cfg)) and t["l0.norm1"].shape == () and t["loop.step"].shape == (2, 22) and "l1.norm2" not in t
    w = LW.place(cfg, RuntimeConfig(dtype="float32"), t, "cpu")
    L = w["layers"][0]
    dn, dr, dv, rank, qr = a.dn, a.dr, a.dv, a.rank, a.qr
    assert (dn, dr, dv, rank, qr) == (24, 8, 16, 32, 24)
    down = L["down"]
    assert down.n == qr + rank + dr + 3
    assert torch.equal(down.data[:18, :22], t["l0.mix.dq"].float()) and down.data[18:24].abs().max() == 0
    assert torch.equal(down.data[24:52, :22], t["l0.mix.dkv"][:28].float()) and torch.equal(down.data[56:62, :22], t["l0.mix.dkv"][28:].float())
    assert torch.equal(down.data[64:67, :22], t["l0.mix.g"].float())
    for h in range(3):
        head = L["uq"].data[h * 32:(h + 1) * 32]
        src = t["l0.mix.uq"][h * 26:(h + 1) * 26].float()
        assert torch.equal(head[:20, :18], src[:20]) and torch.equal(head[24:30, :18], src[20:]) and head[20:24].abs().max() == 0 and head[30:].abs().max() == 0
        uk, uv = t["l0.mix.uk"][h * 20:(h + 1) * 20].float(), t["l0.mix.uv"][h * 12:(h + 1) * 12].float()
        assert torch.equal(L["uk"].data[h * 32:h * 32 + 28, :20], uk.t()) and L["uk"].data[h * 32 + 28:(h + 1) * 32].abs().max() == 0
        assert torch.equal(L["ukv"].data[h * 24:h * 24 + 20, :28], uk)
        assert torch.equal(L["ukv"].data[72 + h * 16:72 + h * 16 + 12, :28], uv)
        assert torch.equal(L["uv"].data[h * 16:h * 16 + 12, :28], uv)
        assert torch.equal(L["o"].data[:, h * 16:h * 16 + 12], t["l0.mix.o"][:, h * 12:(h + 1) * 12].float())
    up, dw = L["experts_up"], L["experts_down"]
    assert (up.groups, up.n, up.k) == (3, 16, 22) and (dw.n, dw.k) == (24, 9)
    assert torch.equal(up.data[16:25, :22], t["l0.mlp.e1.up"].float()) and up.data[25:32].abs().max() == 0
    assert torch.equal(dw.data[48:70, :9], t["l0.mlp.e2.down"].float())
    assert L["router"].n == 4 and L["correction"].dtype == torch.float32 and isinstance(L["norm1"], float) and L["shift"].shape == (24,)
    G = w["layers"][1]
    assert G["zxg"].n == 48 and torch.equal(G["zxg"].data[16:29, :22], t["l1.mix.x"].float()) and G["zb"].shape == (16,) and len(w["step"]) == 2
    bad = dict(t)
    bad["l0.mix.uk"] = bad["l0.mix.uk"][:-1]
    with pytest.raises(ValueError, match="l0.mix.uk"):
        LW.place(cfg, RuntimeConfig(), bad, "cpu")


def test_checkpoint_folder_round_trip_and_registry(tmp_path):
    cfg = LC.tiny_rakelorn()
    t = LW.init_master(cfg, 2)
    p = str(tmp_path / "m")
    LW.save(p, cfg, t)
    fam = registry.family_at(p)
    assert fam.name == "layered" and "float32" in fam.dtypes and registry.family_of(cfg).name == "layered"
    cfg2, w = registry.open_model(p, RuntimeConfig(), "cpu")
    assert cfg2 == cfg and torch.equal(w["embed"][:, :192], t["embed"])
    assert {"Volonex", "Rakelorn"} <= set(registry.ARCHITECTURES)
    for name in ("rakelorn-16b", "rakelorn-2b"):
        c = registry.PRESETS[name]()
        size = sum(math.prod(s) for role, s in LW.tensor_shapes(c).values() if role == "matrix")
        assert c.weight_bytes() == 2 * size
    assert 14e9 < registry.PRESETS["rakelorn-16b"]().weight_bytes() / 2 < 18e9


def test_random_weights_have_the_checkpoint_layout():
    cfg = LC.tiny_rakelorn()
    a = LW.random_weights(cfg, RuntimeConfig(), "cpu", seed=3)
    b = LW.place(cfg, RuntimeConfig(), LW.init_master(cfg, 3), "cpu")
    for x, y in zip(a["layers"], b["layers"]):
        assert x.keys() == y.keys()
        assert all(x[k].data.shape == y[k].data.shape for k in x if isinstance(x[k], (D.DenseW, D.GroupedW)))


def test_states_beside_the_cache():
    cfg = LC.tiny_rakelorn()                           # attention, (recurrent, attention) x 3, recurrent
    rt = RuntimeConfig(kv_pool_tokens=64)
    kv = KVState(cfg, rt, "cpu", 3, 256)
    assert [l is not None for l in kv.layers] == [True] + [False, True] * 3 + [False]
    assert kv.layers[0].dk == 88 + 16 and kv.layers[0].dv == 0 and kv.layers[2].dk == 56 + 32
    assert [sorted(s) for s in kv.states] == [["shift"]] + [["recurrent", "shift"], ["shift"]] * 3 + [["recurrent", "shift"]]
    assert kv.states[1]["recurrent"].shape == (3, 200) and kv.states[7]["recurrent"].shape == (3, 168)
    seen = set()
    for run in kv.states:                              # every pass has its own
        for s in run.values():
            assert s.dtype == torch.float32 and s.data_ptr() % 16 == 0
            s.fill_(len(seen))
            seen.add(s.data_ptr())
    assert len(seen) == 12 and all((s == s[0, 0]).all() for run in kv.states for s in run.values())
    assert len({float(s[0, 0]) for run in kv.states for s in run.values()}) == 12
    assert KVState.nbytes(cfg, rt, 3, 256) > kv.storage.numel() * 2 + sum(s.numel() * 4 for run in kv.states for s in run.values())
    kv.admit(0, 100)
    kv.retire(0, 100)                                  # attention without a window keeps every page
    assert kv.pages_in_use() == 7
    # layers that keep nothing per token let every page go
    only = LC.LayeredConfig("Rakelorn", 9, 8, (LC.LayerSpec(LC.MinGRUSpec(8), None),))
    kv = KVState(only, RuntimeConfig(max_prefill_tokens=64), "cpu", 2, 1 << 16)
    assert kv.num_pages < 20 and kv.first_visible(70) == 70
    for pos in range(0, 1000, 50):
        kv.retire(0, pos)
        kv.admit(0, pos + 50)
    kv.release(0)
    assert kv.pages_in_use() == 0


def test_padded_sizes_and_split_choice():
    d = LT.dims(5, 90, 10)
    assert (d.heads, d.rank, d.rot, d.true_rank, d.true_rot) == (5, 96, 16, 90, 10)
    assert LT.pick_splits(32, 1, 1024, 148) == 4 and LT.pick_splits(1, 1, 1024, 148) == 8 and LT.pick_splits(1, 1, 200, 148) == 1
    assert LT.pick_splits(200, 1, 4096, 148) == 1


def test_designs_refuse_what_they_do_not_combine():
    from mojo_linuxperiments_b200.models.layered import LayeredDecoder
    from mojo_linuxperiments_b200.models.layered_config import AttentionSpec, LayerSpec
    cfg = LC.LayeredConfig("Volonex", 9, 16, (LayerSpec(AttentionSpec(1, 1, 8, 8, 1.0), LC.MoE(2, 1, 8)),))
    with pytest.raises(ValueError, match="whole rows"):
        LayeredDecoder(cfg, RuntimeConfig(), {"embed": torch.zeros(9, 16)})


def test_command_line_knows_the_design(capsys):
    from mojo_linuxperiments_b200 import cli
    assert cli.main(["models"]) == 0
    out = capsys.readouterr().out
    assert "Rakelorn" in out and "rakelorn-16b" in out and "tiny-rakelorn" in out
