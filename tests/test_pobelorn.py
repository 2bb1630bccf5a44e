"""CPU: the Pobelorn decoder's configuration, the model as data, its loader, the cache's kept first positions, and the plain
implementation's pieces on inputs whose answers are known."""
import json
import math

import numpy as np
import pytest
import torch

from mashbox_b200.cache.manager import CacheManager, CacheNeed
from mashbox_b200.config.pobelorn import PobelornConfig
from mashbox_b200.config.registry import read_config
from mashbox_b200.errors import CacheError, ConfigError, WeightError
from mashbox_b200.models.model import Model
from tests import pobelorn_helpers as S
from tests.plain import pobelorn as plain

F64 = torch.float64


@pytest.mark.parametrize("cfg", [c[0] for c in S.CONFIGS.values()] + [S.random_config(i) for i in range(12)])
def test_configuration_round_trip(cfg):
    entry, back = read_config(json.loads(json.dumps(cfg.to_hf())))
    assert entry.name == "Pobelorn" and back == cfg


def test_configuration_refusals():
    good = S.POB_P.to_hf()

    def broken(change):
        c = json.loads(json.dumps(good))
        change(c)
        return c
    for change, word in ((lambda c: c["layers"][0].update(type="other"), "type"),
                         (lambda c: c["layers"][1]["mixer"].update(decay=[0.5, 0.9]), "decay"),
                         (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "rot.dims"),
                         (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "rot.dims"),
                         (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
                         (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "kv_heads"),
                         (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
                         (lambda c: c["layers"][0]["mixer"]["mask"].pop("size"), "mask.size"),
                         (lambda c: c["layers"][0]["mixer"]["mask"].update(size=-1), "mask"),
                         (lambda c: c["layers"][2]["mixer"].update(vdim=20), "mixes 60 values"),
                         (lambda c: c["layers"][1]["mlp"]["router"].update(top=13), "router"),
                         (lambda c: c["layers"][0]["mlp"].update(kind="other"), "kind"),
                         (lambda c: c.pop("width"), "width"),
                         (lambda c: c.pop("norm"), "eps")):
        with pytest.raises(ConfigError, match=word):
            PobelornConfig.from_hf(broken(change))


def test_absent_keys_mean_absent_parts():
    c = S.POB_P.to_hf()
    assert "rot" not in c["layers"][3]["mixer"] and "mask" not in c["layers"][3]["mixer"] and c["layers"][3]["mlp"] is None
    names = read_config(c)[0].stored_tensors(PobelornConfig.from_hf(c))
    assert "l3.mlp.up" not in names and "l3.mix.vmix" not in names and names["l2.mix.vmix"][0] == ()
    assert "l2.mlp.shared.up" not in names and names["l1.mlp.shared.up"][0] == (40, 64) and "head" not in names
    assert names["l1.mix.norm"][0] == (72,) and "l0.norm2" not in names and names["l1.mlp.router.b"][0] == (12,)
    del c["embedding"], c["layers"][0]["mixer"]["mask"]["keep_first"], c["layers"][0]["mixer"]["v_mix"]
    del c["layers"][4]["mixer"]["kv_heads"], c["layers"][0]["mixer"]["rot"]["scaling"]
    cfg = PobelornConfig.from_hf(c)
    m = cfg.layers[0].mixer
    assert cfg.embedding_scale == 1.0 and m.keep_first == 0 and not m.v_mix and m.rot.scaling is None
    assert cfg.layers[4].mixer.kv_heads == 4


def test_model_as_data():
    cfg = S.POB_P
    entry, _ = read_config(cfg.to_hf())
    model = Model(entry.model_spec(cfg), cfg)
    assert [(r.layer, r.cache, r.write, r.state_id) for r in model.schedule] == [
        (0, 0, True, 0), (1, None, False, 1), (2, 2, True, 2), (3, 3, True, 3), (4, 4, True, 4)]
    needs, states = model.cache_needs()
    assert needs[0] == CacheNeed("window", ((2, 16), (2, 24)), 21, 5) and needs[3] == CacheNeed("full", ((1, 32), (1, 8)))
    assert sorted(states) == [1] and states[1].shape == (3 * 16 * 24,)
    assert model.graph_safe and model.portion_alignment() == 1
    # one norm a layer; the first layer that mixes keeps its values, the others read them; its own weight is not read
    assert all(b.norm2 is None for b in model.layers)
    assert [getattr(b.mixer, "value_mix", None) for b in model.layers] == ["keep", None, "mix", None, "mix"]
    wanted = {w.name for w in model.wants()}
    canon = entry.canonical_names(cfg)
    stored = {n: canon(n) for n in entry.stored_tensors(cfg)}
    assert [n for n, c in stored.items() if c is None] == ["l0.mix.vmix"]
    assert {c[0] for c in stored.values() if c is not None} == wanted
    with pytest.raises(KeyError):
        canon("l0.norm2")
    needs, states = Model(entry.model_spec(S.POB_S), S.POB_S).cache_needs()
    assert not needs and sorted(states) == [0, 1]


def test_loader_checks_shapes_and_names(tmp_path):
    from mashbox_b200.engine.loading import build_model
    from mashbox_b200.weights.safetensors_io import SafetensorsSource
    folder = S.make_folder(tmp_path, "P")
    c = json.load(open(folder + "/config.json"))
    src = SafetensorsSource(folder)
    model = build_model(c, src, "float32", "cpu")
    m = model.layers[2].mixer
    assert m.w_in.shape == (6 * 24 + 3 * 24 + 3 * 16, 64) and 0.0 < m.lam < 1.0 and m.qw is None
    assert model.layers[1].mixer.norm_w.shape == (72,) and model.layers[1].ffn.br.shape == (12,)
    assert model.head.weight is model.embedding.table and model.embedding.scale == 3.0
    c["layers"][1]["mixer"].update(heads=2, decay=[0.5, 0.6])
    with pytest.raises(WeightError, match="wrong shape"):
        build_model(c, src, "float32", "cpu")
    src.close()


# ------------------------------------------------------------------------------------------------ kept first positions
def manager(need, page=4, pages=40, requests=3):
    return CacheManager({0: need}, {}, page, pages, requests, 400)


def test_pages_behind_the_window_come_back_and_the_kept_ones_stay():
    m = manager(CacheNeed("window", ((1, 8), (1, 8)), 6, keep=5))
    r = m.admit("a")
    g = m.groups[0]
    first_page = None
    for n in range(1, 61):
        m.extend("a", 1)
        if first_page is None:
            first_page = int(g.table[r.row, 0])
        m.commit("a", 1)
        held = [b for b in range(g.table.shape[1]) if g.table[r.row, b] >= 0]
        # every key that the next query can read lies in a held page: the kept five, and the window's
        for p in [p for p in range(n) if p < 5 or n - p < 6]:
            assert p // 4 in held, (n, p)
        # nothing else is held: positions 0-7 are two pages; the window of the next query spans at most three
        assert all(b < 2 or (b + 1) * 4 > n - 5 for b in held), (n, held)
        m.check()
    assert int(g.table[r.row, 0]) == first_page and len(held) <= 5
    assert m.pages_to_hold(60, 1)[0] >= len(held)
    m.release("a")
    m.check()
    assert m.free_pages() == [40]


@pytest.mark.parametrize("portion", [1, 2, 3, 7, 16])
def test_pages_to_hold_bounds_what_a_request_holds(portion):
    for window, keep in ((6, 5), (1, 1), (16, 4), (5, 30), (9, 0)):
        m = manager(CacheNeed("window", ((1, 8),), window, keep=keep), pages=60)
        m.admit("a")
        most, total = 0, 100
        for at in range(0, total, portion):
            n = min(portion, total - at)
            m.extend("a", n)
            most = max(most, m.pages_held("a")[0])
            m.commit("a", n)
            m.check()
        assert most <= m.pages_to_hold(total, portion)[0], (window, keep, portion)


def test_groups_by_window_and_kept_positions():
    a, b = CacheNeed("window", ((1, 8),), 6, keep=5), CacheNeed("window", ((1, 8),), 6, keep=4)
    m = CacheManager({0: a, 1: b, 2: a}, {}, 4, 10, 2, 100)
    assert [g.cache_ids for g in m.groups] == [[0, 2], [1]]
    assert a.merged(b) == a and a.merged(CacheNeed("full", ((1, 8),))) == CacheNeed("full", ((1, 8),))
    with pytest.raises(CacheError):
        manager(CacheNeed("full", ((1, 8),), None, keep=3))


# ------------------------------------------------------------------------------------------------ the plain pieces
def test_plain_mask_on_its_edges():
    ok = plain.seen(12, dict(size=4, keep_first=2))
    row = lambda i: [j for j in range(12) if ok[i, j]]
    assert row(0) == [0] and row(1) == [0, 1] and row(3) == [0, 1, 2, 3] and row(5) == [0, 1, 2, 3, 4, 5]
    assert row(6) == [0, 1, 3, 4, 5, 6] and row(11) == [0, 1, 8, 9, 10, 11]
    assert plain.seen(5, None).sum() == 15 and plain.seen(5, dict(size=1)).sum() == 5


def test_plain_frequencies_and_rotation_on_known_cases():
    f, gain = plain.frequencies(dict(dims=8, base=100.0))
    assert gain == 1.0 and torch.allclose(f, torch.tensor([1.0, 100 ** -0.25, 0.1, 100 ** -0.75], dtype=F64))
    # pairs before lo keep their frequency, pairs from hi on are slowed by the whole factor, linear in between
    rot = dict(dims=16, base=1e4, scaling=dict(factor=4.0, original=512.0, fast=32.0, slow=1.0))
    b, gain = plain.frequencies(rot)
    lo = max(math.floor(16 * math.log(512 / (2 * math.pi * 32)) / (2 * math.log(1e4))), 0)
    hi = min(math.ceil(16 * math.log(512 / (2 * math.pi)) / (2 * math.log(1e4))), 15)
    assert (lo, hi) == (0, 4) and abs(gain - (0.1 * math.log(4.0) + 1.0)) < 1e-12
    base = torch.tensor([1e4 ** (-i / 8) for i in range(8)], dtype=F64)
    assert torch.allclose(b / base, torch.tensor([1.0, 1 - 0.75 / 4, 1 - 0.75 / 2, 1 - 0.75 * 3 / 4] + [0.25] * 4, dtype=F64))
    x = torch.zeros(2, 1, 6, dtype=F64)
    x[:, 0, 2], x[:, 0, 5] = 1.0, 7.0           # dim 2 turns with dim 3, dim 5 passes (dims = 4)
    y = plain.rotate(x, torch.tensor([0, 3]), dict(dims=4, base=100.0))
    assert abs(float(y[1, 0, 2]) - math.cos(0.3)) < 1e-12 and abs(float(y[1, 0, 3]) - math.sin(0.3)) < 1e-12
    assert float(y[1, 0, 5]) == 7.0 and float(y[1, 0, 0]) == 0.0


def test_engine_frequencies_are_the_plain_ones():
    from mashbox_b200.parts.position import RotaryEncoding
    for dims, base, sc in ((16, 1e4, (4.0, 512.0, 32.0, 1.0)), (8, 100.0, (2.0, 64.0, 8.0, 0.5)), (64, 5e5, None), (2, 50.0, (3.0, 32.0, 4.0, 1.0))):
        rot = dict(dims=dims, base=base, scaling=dict(zip(("factor", "original", "fast", "slow"), sc)) if sc else None)
        f, gain = plain.frequencies(rot)
        r = RotaryEncoding(dims, dims, base, ("yarn",) + sc + (0.1,) if sc else None, "adjacent")
        assert np.allclose(r.frequencies(), f.numpy(), rtol=1e-6) and abs(r.gain - gain) < 1e-12


def test_plain_norm_after_a_rotation_with_a_gain_takes_the_gain_back():
    """all dims rotated: a gain on cos and sin scales the whole head, and the norm after it removes it again; with half of
    the dims rotated it does not"""
    g = torch.Generator().manual_seed(0)
    x = torch.randn(5, 2, 8, generator=g, dtype=F64)
    pos = torch.arange(5)
    sc = dict(factor=1e6, original=1e-9, fast=1e-9, slow=1e-10)       # a gain of 2.4
    f, gain = plain.frequencies(dict(dims=8, base=100.0, scaling=sc))
    assert gain > 2.0
    whole = plain.rms(plain.rotate(x, pos, dict(dims=8, base=100.0, scaling=sc)), 1e-12)
    assert torch.allclose((whole ** 2).mean(-1), torch.ones(5, 2, dtype=F64))
    turned = plain.rotate(x, pos, dict(dims=8, base=100.0, scaling=sc)) / gain
    assert torch.allclose(whole, plain.rms(turned, 1e-12))
    part = plain.rotate(x, pos, dict(dims=4, base=100.0, scaling=sc))
    assert not torch.allclose(plain.rms(part, 1e-12)[..., 4:], plain.rms(x, 1e-12)[..., 4:], rtol=0.1)


def test_plain_value_mixing_uses_the_first_mixing_layers_own_values():
    v, v0 = torch.tensor([[1.0, 2.0]], dtype=F64), torch.tensor([[5.0, -2.0]], dtype=F64)
    assert torch.equal(plain.mixed_values(v, None, torch.tensor(0.7)), v)
    assert torch.allclose(plain.mixed_values(v, v0, torch.tensor(0.25, dtype=F64)), torch.tensor([[2.0, 1.0]], dtype=F64))


def test_plain_router_weights_are_a_softmax_over_the_chosen_logits():
    W = {"m.router": torch.eye(4, dtype=F64), "m.router.b": torch.tensor([0.0, 0.0, 5.0, -9.0], dtype=F64)}
    for e in range(4):                          # expert e returns silu(1) * 1 * (e + 1) in channel 0
        W[f"m.e{e}.gate"], W[f"m.e{e}.up"] = torch.ones(1, 4, dtype=F64), torch.ones(1, 4, dtype=F64)
        W[f"m.e{e}.down"] = torch.tensor([[e + 1.0], [0.0], [0.0], [0.0]], dtype=F64)
    h = torch.tensor([[1.0, 2.0, -2.0, 0.0]], dtype=F64)            # logits 1, 2, 3, -9: experts 2 and 1
    f = dict(router=dict(experts=4, top=2))
    s = 1.0 / (1.0 + math.exp(-1.0))
    p = 1.0 / (1.0 + math.exp(-1.0))                                 # softmax over (3, 2)
    assert abs(float(plain.routed(W, "m.", f, h)[0, 0]) - s * (3 * p + 2 * (1 - p))) < 1e-12


def test_plain_lightning_recurrence_on_known_cases():
    """one head, one key channel, one value channel: the state is a sum of decayed products, and the norm is over all heads"""
    W = {n: torch.tensor([[w]], dtype=F64) for n, w in (("q", 1.0), ("k", 1.0), ("v", 1.0), ("g", 0.0), ("o", 1.0))}
    W["norm"] = torch.tensor([3.0], dtype=F64)
    m = dict(heads=1, dim=1, vdim=1, decay=[0.5])
    h = torch.tensor([[2.0], [0.0], [1.0]], dtype=F64)
    st = torch.zeros(1, 1, 1, dtype=F64)
    out = plain.lightning(W, "", m, h, 1e-12, st)
    silu = lambda z: z / (1.0 + math.exp(-z))
    assert abs(float(st) - (0.25 * silu(2.0) ** 2 + silu(1.0) ** 2)) < 1e-12
    assert abs(float(out[0, 0]) - 3.0 * 0.5) < 1e-6 and float(out[1, 0]) == 0.0      # rms of one value is itself; sigmoid(0)


def test_plain_dense_unit_squares_the_positive_part():
    W = {"up": torch.tensor([[1.0], [-1.0]], dtype=F64), "down": torch.tensor([[1.0, 10.0]], dtype=F64)}
    assert torch.equal(plain.dense(W, "", torch.tensor([[3.0], [-2.0]], dtype=F64)), torch.tensor([[9.0], [40.0]], dtype=F64))
