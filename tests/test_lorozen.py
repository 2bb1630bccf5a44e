"""CPU: the Lorozen decoder's configuration, the model as data, its loader, and the plain implementation's pieces on inputs
whose answers are known."""
import json
import math

import numpy as np
import pytest
import torch

from mashbox_b200.cache.manager import CacheNeed
from mashbox_b200.config.lorozen import LorozenConfig
from mashbox_b200.config.registry import read_config
from mashbox_b200.errors import ConfigError, WeightError
from mashbox_b200.models.model import Model
from tests import lorozen_helpers as S
from tests.plain import lorozen as plain

F64 = torch.float64


@pytest.mark.parametrize("cfg", [c[0] for c in S.CONFIGS.values()] + [S.random_config(i) for i in range(12)])
def test_configuration_round_trip(cfg):
    entry, back = read_config(json.loads(json.dumps(cfg.to_hf())))
    assert entry.name == "Lorozen" and back == cfg


def test_configuration_refusals():
    good = S.LOR_P.to_hf()

    def broken(change):
        c = json.loads(json.dumps(good))
        change(c)
        return c
    for change, word in ((lambda c: c["layers"][0].update(type="other"), "type"),
                         (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "rot.dims"),
                         (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "rot.dims"),
                         (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=10), "rot.dims"),
                         (lambda c: c["layers"][2]["mixer"]["rot"].update(scaling={"factor": 2}), "scaling"),
                         (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("low"), "low"),
                         (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "kv_heads"),
                         (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
                         (lambda c: c["layers"][2]["mixer"].pop("kv_rank"), "kv_rank"),
                         (lambda c: c["layers"][0]["mixer"]["mask"].pop("size"), "mask.size"),
                         (lambda c: c["layers"][2]["mixer"]["mask"].update(size=-1), "mask"),
                         (lambda c: c["layers"][1]["mlp"]["router"].update(top=13), "router"),
                         (lambda c: c["layers"][0]["mlp"].update(kind="other"), "kind"),
                         (lambda c: c["loop"].update(stop=6), "loop"),
                         (lambda c: c["loop"].update(start=4), "loop"),
                         (lambda c: c["loop"].update(times=0), "loop"),
                         (lambda c: c["loop"].pop("times"), "loop.times"),
                         (lambda c: c.pop("width"), "width"),
                         (lambda c: c.pop("norm"), "eps")):
        with pytest.raises(ConfigError, match=word):
            LorozenConfig.from_hf(broken(change))


def test_absent_keys_mean_absent_parts():
    c = S.LOR_P.to_hf()
    assert "rot" not in c["layers"][3]["mixer"] and "mask" not in c["layers"][3]["mixer"] and c["layers"][3]["mlp"] is None
    names = read_config(c)[0].stored_tensors(LorozenConfig.from_hf(c))
    assert "l3.norm2" not in names and "l3.norm2b" not in names and "l3.norm1b" in names and "l3.mlp.up" not in names
    assert "l2.mlp.shared.up" not in names and names["l1.mlp.shared.up"][0] == (40, 64) and names["head"][0] == (131, 64)
    assert names["l1.mix.norm"][0] == (48,) and names["l1.mix.u"][0] == (3, 16) and names["l1.mix.w2"][0] == (48, 12)
    assert names["l0.mix.v.b"][0] == (48,) and names["l0.mix.sink"][0] == (4,) and names["l2.mix.dkv"][0] == (40, 64)
    assert names["l2.mix.g"][0] == (6, 64) and "l2.mix.q.b" not in names and "l0.mix.o.b" not in names
    del c["loop"], c["logit_softcap"], c["layers"][0]["mixer"]["rot"]["scaling"], c["layers"][4]["mixer"]["kv_heads"]
    cfg = LorozenConfig.from_hf(c)
    assert cfg.loop is None and cfg.logit_softcap is None and cfg.layers[0].mixer.rot.scaling is None
    assert cfg.layers[4].mixer.kv_heads == 4 and cfg.order() == [(i, False) for i in range(5)]


def test_model_as_data():
    cfg = S.LOR_P
    entry, _ = read_config(cfg.to_hf())
    model = Model(entry.model_spec(cfg), cfg)
    # layers 1 to 3 run three times; every run has a cache or a state of its own; the embedding joins before runs 4 and 7
    assert [r.layer for r in model.schedule] == [0, 1, 2, 3, 1, 2, 3, 1, 2, 3, 4]
    assert [r.cache for r in model.schedule] == [0, None, 2, 3, None, 5, 6, None, 8, 9, 10]
    assert [i for i, r in enumerate(model.schedule) if r.rejoin] == [4, 7]
    assert len(model.layers) == 5 and plain.order_of_layers(cfg.to_hf()) == cfg.order()
    needs, states = model.cache_needs()
    assert needs[0] == CacheNeed("window", ((2, 16), (2, 24)), 21) and needs[3] == needs[9] == CacheNeed("full", ((1, 32), (1, 8)))
    assert needs[2] == needs[5] == CacheNeed("window", ((1, 40),), 18)
    assert sorted(states) == [1, 4, 7] and states[1].shape == (64 + 3 * 16 * 16,)
    assert model.graph_safe and model.portion_alignment() == 1
    wanted = {w.name for w in model.wants()}
    canon = entry.canonical_names(cfg)
    assert {canon(n)[0] for n in entry.stored_tensors(cfg)} == wanted
    with pytest.raises(KeyError):
        canon("l0.mix.g")
    needs, states = Model(entry.model_spec(S.LOR_S), S.LOR_S).cache_needs()
    assert not needs and sorted(states) == [0, 1, 2, 3, 4]
    once = Model(entry.model_spec(S.LOR_T), S.LOR_T)
    assert [(r.layer, r.rejoin) for r in once.schedule] == [(0, False), (1, False)]


def test_loader_checks_shapes_and_reads_the_inner_rank(tmp_path):
    from mashbox_b200.engine.loading import build_model
    from mashbox_b200.weights.safetensors_io import SafetensorsSource
    folder = S.make_folder(tmp_path, "P")
    c = json.load(open(folder + "/config.json"))
    src = SafetensorsSource(folder)
    del c["layers"][1]["mixer"]["decay_rank"]               # only random-weights mode writes it
    model = build_model(c, src, "float32", "cpu")
    a, w, m = model.layers[0].mixer, model.layers[1].mixer, model.layers[2].mixer
    assert a.w_in.shape == (4 * 16 + 2 * 16 + 2 * 24, 64) and a.bias.shape == (144,) and a.sinks.shape == (4,)
    assert w.w1.shape == (12, 64) and w.w_in.shape == (4 * 48, 64) and w.mu.shape == (5, 64) and w.norm_w.shape == (3, 16)
    assert m.w_in.shape == (240, 64) and m.window == 18        # 6 x 32 query rows, 40 kept, 6 gates, 2 rows of zeros
    assert float(m.w_in[238:].abs().max()) == 0.0
    assert model.head.softcap == 8.0 and model.head.weight is not model.embedding.table
    c["layers"][1]["mixer"].update(heads=2)
    with pytest.raises(WeightError, match="wrong shape"):
        build_model(c, src, "float32", "cpu")
    src.close()


# ------------------------------------------------------------------------------------------------ the plain pieces
def test_plain_mask_on_its_edges():
    ok = plain.visible(9, dict(size=4))
    row = lambda i: [j for j in range(9) if ok[i, j]]
    assert row(0) == [0] and row(3) == [0, 1, 2, 3] and row(4) == [1, 2, 3, 4] and row(8) == [5, 6, 7, 8]
    assert plain.visible(5, None).sum() == 15 and plain.visible(5, dict(size=1)).sum() == 5


def test_plain_frequencies_and_rotation_on_known_cases():
    assert torch.allclose(plain.frequencies(dict(dims=8, base=100.0)),
                          torch.tensor([1.0, 100 ** -0.25, 0.1, 100 ** -0.75], dtype=F64))
    # wavelengths 6.3, 63 and 628 and 6,283 against original / high = 50 and original / low = 200
    sc = dict(factor=8.0, low=1.0, high=4.0, original=200.0)
    f = plain.frequencies(dict(dims=8, base=1e4, scaling=sc))
    s = (200 / (20 * math.pi) - 1) / 3
    assert torch.allclose(f, torch.tensor([1.0, 0.1 * (s + (1 - s) / 8), 0.01 / 8, 0.001 / 8], dtype=F64))
    x = torch.zeros(2, 1, 6, dtype=F64)
    x[:, 0, 1], x[:, 0, 5] = 1.0, 7.0           # dims = 4: dim 1 turns with dim 3 (halves) or dim 0 (adjacent), dim 5 passes
    pos = torch.tensor([0, 3])
    y = plain.rotate(x, pos, dict(dims=4, base=100.0), "halves")
    assert abs(float(y[1, 0, 1]) - math.cos(0.3)) < 1e-12 and abs(float(y[1, 0, 3]) - math.sin(0.3)) < 1e-12
    z = plain.rotate(x, pos, dict(dims=4, base=100.0), "adjacent")
    assert abs(float(z[1, 0, 0]) + math.sin(3.0)) < 1e-12 and abs(float(z[1, 0, 1]) - math.cos(3.0)) < 1e-12
    assert float(y[1, 0, 5]) == float(z[1, 0, 5]) == 7.0


def test_engine_frequencies_are_the_plain_ones():
    from mashbox_b200.parts.position import RotaryEncoding
    for dims, base, sc in ((16, 1e4, (4.0, 1.0, 4.0, 512.0)), (8, 100.0, (2.0, 0.5, 8.0, 64.0)), (64, 5e5, None),
                           (2, 50.0, (3.0, 1.0, 3.0, 32.0))):
        rot = dict(dims=dims, base=base, scaling=dict(zip(("factor", "low", "high", "original"), sc)) if sc else None)
        r = RotaryEncoding(dims, dims, base, ("llama3",) + sc if sc else None, "halves")
        assert np.allclose(r.frequencies(), plain.frequencies(rot).numpy(), rtol=2e-6)


def test_plain_sink_takes_its_share_of_the_weight():
    s = torch.tensor([[[0.0, -math.inf], [1.0, 2.0]]], dtype=F64)
    w = plain.softmax_with_sink(s, torch.tensor([0.5], dtype=F64))
    assert abs(float(w[0, 0, 0]) - 1 / (1 + math.exp(0.5))) < 1e-12 and float(w[0, 0, 1]) == 0.0
    d = math.exp(1) + math.exp(2) + math.exp(0.5)
    assert abs(float(w[0, 1, 1]) - math.exp(2) / d) < 1e-12


def test_plain_wkv_on_known_cases():
    """one head, one channel, every projection one: a mix of one half, a decay of exp(-1), the current token counted u times"""
    one = torch.ones(1, 1, dtype=F64)
    W = {k: one for k in ("r", "k", "v", "o", "w1", "u")}
    W.update({"g": one * 0.0, "w2": one * 0.0, "w0": torch.zeros(1, dtype=F64), "norm": torch.tensor([3.0], dtype=F64),
              "u": torch.tensor([[2.0]], dtype=F64)})
    W.update({"mu." + s: torch.tensor([0.5], dtype=F64) for s in "rkvgw"})
    m = dict(heads=1, dim=1)
    assert torch.equal(plain.wkv(W, "", m, torch.ones(3, 1, dtype=F64), 1e-9), torch.zeros(3, 1, dtype=F64))    # silu(0)
    W["g"] = one
    h = torch.tensor([[2.0], [4.0]], dtype=F64)
    y = plain.wkv(W, "", m, h, 1e-12)
    silu = lambda z: z / (1 + math.exp(-z))
    # mixes 1 and 3; o is positive, so its rms-normed value is 1
    assert abs(float(y[0]) - 3.0 * silu(1.0)) < 1e-9 and abs(float(y[1]) - 3.0 * silu(3.0)) < 1e-9
    # under a large eps o itself shows.  The third token's mix is 1; the second token's product has not decayed when it reads
    # it, the first one's has once
    y = plain.wkv(W, "", m, torch.tensor([[2.0], [4.0], [-2.0]], dtype=F64), 1e14) * 1e7
    o = [1 * (2 * 1), 3 * (1 + 2 * 9), 1 * (math.exp(-1.0) + 9 + 2 * 1)]
    want = [a * 3 * silu(b) for a, b in zip(o, (1.0, 3.0, 1.0))]
    assert torch.allclose(y[:, 0], torch.tensor(want, dtype=F64), rtol=1e-9)


def test_plain_router_weights_meet_the_experts_inputs():
    W = {"m.router": torch.eye(3, 2, dtype=F64)}
    for e in range(3):                          # expert e: silu(x0) * x0 * (e + 1) in channel 0
        W[f"m.e{e}.gate"] = W[f"m.e{e}.up"] = torch.tensor([[1.0, 0.0]], dtype=F64)
        W[f"m.e{e}.down"] = torch.tensor([[e + 1.0], [0.0]], dtype=F64)
    h = torch.tensor([[2.0, -3.0]], dtype=F64)                       # logits 2, -3, 0: experts 0 and 2
    sig = lambda z: 1 / (1 + math.exp(-z))
    unit = lambda x: x * x * sig(x)
    want = unit(2 * sig(2.0)) + 3 * unit(2 * sig(0.0))
    assert abs(float(plain.experts(W, "m.", dict(router=dict(top=2)), h)[0, 0]) - want) < 1e-12


def test_plain_dense_unit_is_gated_by_gelu():
    W = {"gate": torch.tensor([[1.0]], dtype=F64), "up": torch.tensor([[3.0]], dtype=F64), "down": torch.tensor([[2.0]], dtype=F64)}
    x = torch.tensor([[0.7], [-2.0]], dtype=F64)
    want = torch.nn.functional.gelu(x, approximate="tanh") * 3 * x * 2
    assert torch.allclose(plain.gated_unit(W, "", x, plain.gelu_tanh), want)


def test_plain_loop_adds_the_embedding_before_every_pass_but_the_first(tmp_path):
    """three passes over layers whose norms after the sublayers are zero: the stream is one, two, three embeddings"""
    cfg, W = S._model(S.make_folder(tmp_path, "S"))
    W = {k: torch.zeros_like(v) if k.endswith(("norm1b", "norm2b")) else v for k, v in W.items()}
    after = []
    plain.forward(cfg, W, [5, 9], after)
    e = W["embed"][[5, 9]].double()
    assert [round(float((x / e).mean()), 9) for x in after] == [1.0, 1.0, 2.0, 3.0, 4.0]
