"""Volonex without a GPU: the oracle's mechanisms against hand computation, the configuration, the weight layout, the cache's
bookkeeping, the registry and the command line."""
import json
import math

import pytest
import torch

from mojo_linuxperiments_b200.models import layered_config as LC
from mojo_linuxperiments_b200.models import layered_weights as LW
from mojo_linuxperiments_b200.models import registry
from mojo_linuxperiments_b200.models.config import ModelConfig, RuntimeConfig
from mojo_linuxperiments_b200.models.kvcache import KVState
from mojo_linuxperiments_b200.ops import attention as A
from mojo_linuxperiments_b200.oracle import volonex as V


def test_oracle_norm_and_glu_by_hand():
    x = torch.tensor([[0.5, -2.0, 30.0]], dtype=torch.float64)
    w, b = torch.tensor([1.0, 2.0, 3.0], dtype=torch.float64), torch.tensor([0.0, 1.0, -1.0], dtype=torch.float64)
    got = V.dynamic_tanh(x, torch.tensor(0.5, dtype=torch.float64), w, b)[0].tolist()
    assert got == pytest.approx([math.tanh(0.25), 2 * math.tanh(-1.0) + 1, 3 * math.tanh(15.0) - 1])
    one = torch.eye(1, dtype=torch.float64)
    for g, u in [(9.0, 9.0), (-9.0, -9.0), (0.3, -0.2)]:
        h = torch.ones((1, 1), dtype=torch.float64)
        y = V.clamped_glu(h, {"gate": one * g, "up": one * u, "down": one}, 2.5).item()
        gg, uu = min(g, 2.5), max(-2.5, min(u, 2.5))
        assert y == pytest.approx(gg / (1 + math.exp(-1.702 * gg)) * (uu + 1))


def test_oracle_chunks_and_sink_by_hand():
    vis = V.chunk_mask(11, 4)
    for i in range(11):
        assert [j for j in range(11) if vis[i, j]] == [j for j in range(i // 4 * 4, i + 1)]
    assert V.chunk_mask(5, None).sum().item() == 15
    s = torch.tensor([[[1.0, 2.0], [0.0, 1.0]]], dtype=torch.float64)
    w = V.sink_softmax(s, V.chunk_mask(2, None), torch.tensor([0.5], dtype=torch.float64))
    e = math.exp
    assert w[0, 0].tolist() == pytest.approx([e(1) / (e(1) + e(0.5)), 0.0])
    assert w[0, 1].tolist() == pytest.approx([1 / (1 + e(1) + e(0.5)), e(1) / (1 + e(1) + e(0.5))])


def test_oracle_rotation_by_hand():
    f, mag = V.yarn_frequencies(4, 100.0, None)
    assert f.tolist() == pytest.approx([1.0, 0.1]) and mag == 1.0
    x = torch.arange(1.0, 7.0, dtype=torch.float64).view(1, 1, 6)
    y = V.rotate_interleaved(x, torch.tensor([3]), f, 2.0)[0, 0].tolist()
    c, s = math.cos(3.0), math.sin(3.0)
    assert y[:2] == pytest.approx([2 * (1 * c - 2 * s), 2 * (2 * c + 1 * s)])
    c, s = math.cos(0.3), math.sin(0.3)
    assert y[2:4] == pytest.approx([2 * (3 * c - 4 * s), 2 * (4 * c + 3 * s)]) and y[4:] == [5.0, 6.0]


@pytest.mark.parametrize("dims,base,sc", [
    (64, 10000.0, dict(factor=8.0, original=4096, fast=32.0, slow=1.0)),
    (24, 500.0, dict(factor=1.0, original=100, fast=4.0, slow=2.0)),
    (16, 1e6, dict(factor=3.0, original=64, fast=2.0, slow=2.0)),          # an empty ramp
    (8, 20.0, dict(factor=40.0, original=1 << 20, fast=1.0, slow=0.5)),     # ends beyond the last pair
    (32, 10000.0, None)])
def test_rotation_frequencies_of_the_product_match_the_oracle(dims, base, sc):
    want, mag = V.yarn_frequencies(dims, base, sc)
    got, mag2 = A.rope_frequencies(dims, base, LC.Yarn(**sc) if sc else None)
    assert torch.allclose(got, want, rtol=1e-12, atol=0) and mag2 == pytest.approx(mag, rel=1e-12)
    cos, sin = A.rope_tables(50, base, "cpu", dims, LC.Yarn(**sc) if sc else None)
    assert torch.allclose(cos.double(), (torch.arange(50)[:, None] * want).cos() * mag, atol=1e-6) and sin.shape == (50, dims // 2)
    if sc and sc["factor"] > 1 and sc["fast"] > sc["slow"] and dims == 64:
        plain, _ = V.yarn_frequencies(dims, base, None)
        r = want / plain
        assert r[0] == 1.0 and r[-1].item() == pytest.approx(1 / sc["factor"]) and ((r[1:] - r[:-1]) <= 0).all()


def test_layer_schedule_and_runs_agree():
    for loop in (None, LC.Loop(0, 2, 3), LC.Loop(1, 2, 1), LC.Loop(2, 3, 4)):
        cfg = LC.LayeredConfig("Volonex", 10, 8, LC.tiny_volonex().layers, loop=loop)
        want = V.layer_schedule(cfg.to_dict())
        assert [(r.layer, r.add_embedding) for r in cfg.runs] == want
        n = 3 if loop is None else 3 + (loop.times - 1) * (loop.stop - loop.start)
        assert len(want) == n and len(cfg.cache_layout(RuntimeConfig())) == n
    assert sum(a for _, a in V.layer_schedule({"layers": [0] * 4, "loop": {"start": 1, "stop": 3, "times": 3}})) == 2


def test_config_round_trip_and_rejections(tmp_path):
    cfg = LC.tiny_volonex()
    assert LC.LayeredConfig.from_json(cfg.to_json()) == cfg
    d = cfg.to_dict()
    assert d["layers"][1]["mlp"] is None and d["layers"][0]["mixer"]["rot"]["scaling"]["factor"] == 2.0
    for path, value in [(("layers", 0, "type"), "recurrent"), (("layers", 0, "mlp", "kind"), "routed"),
                        (("layers", 0, "mixer", "kv_heads"), 3), (("loop", "stop"), 9), (("layers", 0, "mixer", "rot", "dims"), 66)]:
        bad = json.loads(json.dumps(d))
        at = bad
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(ValueError):
            LC.LayeredConfig.from_dict(bad)
    # constants that a model may leave out: no chunk, no scaling, no rotation, no loop
    d.pop("loop")
    m = d["layers"][0]["mixer"]
    m.pop("mask"), m["rot"].pop("scaling"), d["layers"][1]["mixer"].pop("rot")
    c = LC.LayeredConfig.from_dict(d)
    assert c.layers[0].mixer.chunk is None and c.layers[0].mixer.rot.scaling is None and c.layers[1].mixer.rot is None and c.loop is None


def test_weight_layout_pads_heads_and_interleaves():
    m = LC.AttentionSpec(3, 1, 20, 12, 0.3, LC.Rotary(100.0, 6), 5)
    cfg = LC.LayeredConfig("Volonex", 19, 22, (LC.LayerSpec(m, LC.GatedMLP(9, 1.0)),))
    t = LW.init_master(cfg, 1)
    w = LW.place(cfg, RuntimeConfig(dtype="float32"), t, "cpu")
    L = w["layers"][0]
    q = L["qkvg"]
    assert (m.dk, m.dv) == (24, 16) and q.n == 3 * 24 + 24 + 16 + 3 and q.data.shape == (q.n, 24) and q.k == 22
    for h in range(3):
        assert torch.equal(q.data[24 * h:24 * h + 20, :22], t["l0.mix.q"][20 * h:20 * h + 20].float())
        assert q.data[24 * h + 20:24 * h + 24].abs().max() == 0
    assert torch.equal(q.data[96:108, :22], t["l0.mix.v"].float()) and torch.equal(q.data[112:115, :22], t["l0.mix.g"].float())
    assert torch.equal(L["o"].data[:, 16:28], t["l0.mix.o"][:, 12:24].float()) and L["o"].data[:, 28:32].abs().max() == 0
    assert torch.equal(L["gate_up"].data[0::2, :22], t["l0.mlp.gate"].float()) and torch.equal(L["gate_up"].data[1::2, :22], t["l0.mlp.up"].float())
    assert L["norm1"].alpha == float(t["l0.norm1.alpha"]) and L["sink"].dtype == torch.float32
    bad = dict(t)
    bad["l0.mix.k"] = bad["l0.mix.k"][:-1]
    with pytest.raises(ValueError, match="l0.mix.k"):
        LW.place(cfg, RuntimeConfig(), bad, "cpu")


def test_checkpoint_folder_round_trip_and_registry(tmp_path):
    cfg = LC.tiny_volonex()
    t = LW.init_master(cfg, 2)
    p = str(tmp_path / "m")
    LW.save(p, cfg, t)
    fam = registry.family_at(p)
    assert fam.name == "layered" and "float32" in fam.dtypes and registry.family_of(cfg).name == "layered"
    cfg2, w = registry.open_model(p, RuntimeConfig(), "cpu")
    assert cfg2 == cfg and torch.equal(w["embed"][:, :256], t["embed"])
    assert registry.family_of(ModelConfig("x", 1, 128, 1, 1, 128, 128)).name == "w8a8"
    with open(tmp_path / "m" / "config.json", "w") as f:
        json.dump({"architecture": "Other"}, f)
    with pytest.raises(ValueError, match="Other"):
        registry.family_at(p)
    with pytest.raises(TypeError):
        registry.family_of(object())


def test_cache_gives_back_pages_no_layer_can_see():
    cfg = LC.tiny_volonex()                        # chunks of 40 and 24 positions, pages of 16
    kv = KVState(cfg, RuntimeConfig(max_prefill_tokens=32), "cpu", 2, 4096)
    assert kv.num_pages - 1 == 2 * ((40 + 32 + 15) // 16 + 2)      # not 2 x 256
    for pos in (0, 23, 24, 39, 40, 47, 48, 79, 80, 119, 120):
        assert kv.first_visible(pos) == min(pos // 40 * 40, pos // 24 * 24)
    owned = []
    for pos in range(500):
        kv.retire(0, pos)
        kv.admit(0, pos + 1)
        first = kv.first_visible(pos)
        row = kv.table_host[0]
        live = {int(row[i]) for i in range(first // 16, pos // 16 + 1)}
        assert kv.scratch_page not in live and len(live) == pos // 16 - first // 16 + 1      # all visible pages are there
        assert all(int(row[i]) == kv.scratch_page for i in range(first // 16))
        owned.append(kv.pages_in_use())
    assert max(owned) <= 40 // 16 + 2
    kv.admit(1, 30)
    kv.release(0)
    assert kv.pages_in_use() == 2
    kv.release(1)
    assert sorted(kv.free_pages) == list(range(kv.num_pages - 1))
    # a layer that sees everything keeps everything
    full = LC.LayeredConfig("Volonex", 9, 8, (LC.LayerSpec(LC.AttentionSpec(1, 1, 8, 8, 1.0), None), cfg.layers[0]))
    kv = KVState(full, RuntimeConfig(), "cpu", 1, 256)
    kv.admit(0, 200)
    kv.retire(0, 200)
    assert kv.pages_in_use() == 13 and kv.num_pages == 17
    # a shared pool smaller than slots x length
    kv = KVState(full, RuntimeConfig(kv_pool_tokens=64), "cpu", 3, 256)
    assert kv.num_pages - 1 == 4 + 6
    kv.admit(0, 100)
    with pytest.raises(RuntimeError, match="exhausted"):
        kv.admit(1, 100)


def test_command_line_refuses_what_a_family_cannot_do(tmp_path, capsys):
    from mojo_linuxperiments_b200 import cli
    assert cli.main(["models"]) == 0
    assert "volonex-8b" in capsys.readouterr().out
    rc = cli.trace_main(["--model", str(tmp_path / "w8a8.safetensors"), "--dtype", "float32", "--out", str(tmp_path)])
    assert rc == 3 and "float32" in capsys.readouterr().err
