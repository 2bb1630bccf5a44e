"""Small Lorozen configurations with random weights, and the plain implementation's logits for them."""
import functools
import os

import numpy as np
import torch

from mashbox_b200.config.lorozen import (AttentionMixer, DenseFF, ExpertsFF, LatentMixer, Loop, LorozenConfig, LorozenLayer,
                                         Rotation, WkvMixer)
from tests.plain import lorozen as plain
from tests.plain.llama import read_model


def att(heads, kv, dim, vdim, scale, rot=0, base=10000.0, scaling=None, window=None):
    return AttentionMixer(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale,
                          rot=Rotation(rot, base, scaling) if rot else None, window=window)


def lat(heads, dim, vdim, rank, scale, rot=0, base=10000.0, window=None):
    return LatentMixer(heads=heads, dim=dim, vdim=vdim, kv_rank=rank, scale=scale, rot_dim=rot,
                       rot=Rotation(rot, base) if rot else None, window=window)


def wkv(heads, dim, rank=None):
    return WkvMixer(heads=heads, dim=dim, decay_rank=rank)


TYPES = {AttentionMixer: "attention", LatentMixer: "latent_attention", WkvMixer: "wkv"}


def model(width, vocab, eps, cap, loop, *layers):
    return LorozenConfig("Lorozen", width=width, vocab=vocab, norm_eps=eps, logit_softcap=cap,
                         loop=Loop(*loop) if loop else None,
                         layers=tuple(LorozenLayer(TYPES[type(m)], m, f) for m, f in layers))


# P: every size differs from layer to layer where it may: windows of 21, 18 and 1 position and none, rotations in part, whole
#    and none, frequencies slowed in part; queries wider than values and narrower; experts with and without a shared one, one
#    chosen and all chosen; a dense unit; no feed-forward; the loop in the middle, three passes, over one layer of each kind
LOR_P = model(64, 131, 1e-2, 8.0, (1, 4, 3),
              (att(4, 2, 16, 24, 0.3, 8, 100.0, (4.0, 1.0, 4.0, 64.0), 21), DenseFF(96)),
              (wkv(3, 16, 12), ExpertsFF(32, 12, 3, 40)),
              (lat(6, 24, 16, 32, 0.2, 8, 500.0, 18), ExpertsFF(24, 6, 1, None)),
              (att(2, 1, 32, 8, 0.25), None),
              (att(4, 4, 8, 12, 0.4, 2, 50.0, (2.0, 1.0, 3.0, 32.0), 1), ExpertsFF(16, 4, 4, 16)))
# Q: the loop over the whole model; a wkv layer first and two in a row, one without a feed-forward; more query heads on one
#    kv head and on one latent than a decode tile has rows; a window of exactly two pages; no cap on the logits
LOR_Q = model(96, 89, 3e-2, None, (0, 4, 2),
              (wkv(1, 40, 5), DenseFF(40)),
              (att(20, 1, 16, 16, 0.35, 16, 1e6, (8.0, 1.0, 4.0, 4096.0), 32), ExpertsFF(40, 5, 2, 64)),
              (wkv(5, 8, 24), None),
              (lat(18, 8, 40, 48, 0.3, 16, 1e4), ExpertsFF(24, 8, 2, None)))
# R: sizes the tensor-core kernels take: heads of 64 x 64 and 128 x 128 (the TMA and tcgen05 kernels with sinks, windows of
#    100 and 64 and none), 32 x 64 (the general one), latent rows of 112 and 64, wkv heads of 32 with products that group
LOR_R = model(128, 301, 1e-2, 20.0, (2, 5, 2),
              (att(8, 2, 64, 64, 0.15, 32, 1e5, (2.0, 1.0, 8.0, 256.0), 100), ExpertsFF(64, 16, 4, 96)),
              (wkv(4, 32, 16), DenseFF(256)),
              (att(4, 1, 128, 128, 0.1, 128, 1e4, None, 64), ExpertsFF(32, 4, 2, 32)),
              (lat(8, 32, 64, 96, 0.15, 16, 1e4, 70), DenseFF(128)),
              (att(6, 2, 32, 64, 0.2, 16, 1e4, None, 70), DenseFF(128)),
              (att(16, 2, 64, 64, 0.15, 64, 1e4), ExpertsFF(64, 8, 2, None)))
# S: wkv layers only -- the model keeps nothing per position, the cache manager has no group and takes no page; one head; a
#    loop of one layer, which ends the model
LOR_S = model(48, 61, 2e-2, 5.0, (1, 2, 4),
              (wkv(2, 16, 3), ExpertsFF(16, 4, 2, 8)),
              (wkv(1, 32, 8), None))
# Z: sizes that are multiples of neither 8 nor 16, so that no 16-byte form of any kernel applies, a page of 5 positions; no
#    loop
LOR_Z = model(100, 53, 5e-2, 3.0, None,
              (att(3, 3, 10, 6, 0.3, 6, 300.0, (3.0, 0.5, 2.0, 32.0), 18), DenseFF(28)),
              (wkv(3, 10, 7), ExpertsFF(12, 6, 2, 20)),
              (lat(3, 6, 9, 22, 0.4, 4, 70.0, 11), None),
              (wkv(1, 6, 1), ExpertsFF(20, 3, 1, None)),
              (att(5, 1, 14, 10, 0.25, 2, 70.0, None, 40), ExpertsFF(28, 5, 3, 44)))
# T: a loop that runs once (the embedding joins nowhere), latent attention without a rotated part and over every earlier key
LOR_T = model(64, 71, 1e-5, 12.0, (0, 2, 1),
              (lat(4, 16, 16, 32, 0.3), DenseFF(48)),
              (att(2, 2, 16, 16, 0.3, 16, 1e3, None, 33), ExpertsFF(16, 8, 2, 16)))
CONFIGS = {"P": (LOR_P, 51, 8), "Q": (LOR_Q, 52, 16), "R": (LOR_R, 53, 16), "S": (LOR_S, 54, 32),
           "Z": (LOR_Z, 55, 5), "T": (LOR_T, 56, 16)}       # config, seed, page size

# Readers near 1/sqrt(fan in), writers into the stream moderate; the router wide enough that the chosen experts are seldom a
# close call; biases, sinks and bonuses of order 1 so that they matter; decays from quick to slow.  The weights of the norms
# after the sublayers are scaled by POST (whatever a sublayer's size, its normed output has this one), so that a token whose
# expert is a close call differs, and does not become another; and eps is not small beside the mean square of a recurrence's
# output, which at a token where r, u and k cancel (at the first one it is nothing but their product times v) would otherwise
# be rounding noise brought to full scale.
STD_BY_NAME = (("mlp.router", 0.4), (".down", 0.15), ("mix.o", 0.15), ("embed", 1.2), ("mix.w0", 1.5), ("mix.u", 0.7),
               ("mix.sink", 1.5), ("mix.q.b", 0.5), ("mix.k.b", 0.5), ("mix.v.b", 0.5))
POST = 0.4


def random_config(seed):
    """a configuration drawn at random: 2 to 5 layers of any kind in any order, a loop over any run of them or none, sizes
    from small sets that include 1, odd sizes, multiples of 16 (which the tensor-core kernels take) and keys wider and
    narrower than values"""
    rng = np.random.default_rng(3000 + seed)
    pick = lambda *xs: xs[int(rng.integers(len(xs)))]
    layers = []
    for _ in range(int(rng.integers(2, 6))):
        kind, window = pick(0, 1, 2), pick(None, 1, 7, 16, 40)
        if kind == 0:
            m = wkv(pick(1, 2, 3, 4), pick(8, 10, 16, 20, 32, 64), pick(1, 4, 8, 20))
        elif kind == 1:
            kv, dim, vdim = pick(1, 2, 3), pick(8, 10, 16, 32, 64), pick(8, 12, 16, 32, 64)
            rot = pick(0, 2, dim // 2 - (dim // 2) % 2, dim)
            m = att(kv * pick(1, 2, 4), kv, dim, vdim, pick(0.1, 0.2, 0.4), rot, pick(100.0, 1e4, 5e5),
                    pick(None, (2.0, 1.0, 4.0, 2048.0), (4.0, 0.5, 4.0, 64.0)), window)
        else:
            m = lat(pick(1, 2, 3, 8), pick(8, 10, 32), pick(8, 12, 32), pick(16, 24, 48, 64), pick(0.1, 0.2, 0.4),
                    pick(2, 4, 16), pick(100.0, 1e4), window)
        experts = pick(1, 4, 6, 16)
        f = pick(None, DenseFF(pick(16, 24, 40, 64)), ExpertsFF(pick(8, 24, 32), experts, min(experts, pick(1, 2, 4)),
                                                               pick(None, 16, 28)))
        layers.append((m, f))
    a = int(rng.integers(0, len(layers)))
    loop = pick(None, (a, int(rng.integers(a + 1, len(layers) + 1)), pick(1, 2, 3)))
    return model(pick(32, 48, 64, 96, 100), pick(50, 97, 128), pick(1e-2, 5e-2), pick(None, 4.0, 20.0), loop, *layers)


def write_folder(d, cfg, seed, dtype):
    import json
    from mashbox_b200.config.registry import architecture
    from mashbox_b200.weights.random_init import random_tensors
    from mashbox_b200.weights.safetensors_io import write_safetensors
    os.makedirs(d, exist_ok=True)
    with open(os.path.join(d, "config.json"), "w") as fh:
        json.dump(cfg.to_hf(), fh)
    t = random_tensors(architecture("Lorozen").stored_tensors(cfg), seed, std=cfg.width ** -0.5, norm_std=0.1,
                       std_by_name=STD_BY_NAME)
    write_safetensors(os.path.join(d, "model.safetensors"),
                      {k: (v * POST if k.endswith(("norm1b", "norm2b")) else v).to(dtype) for k, v in t.items()})
    return d


def make_folder(tmp, name, store="float32"):
    cfg, seed, _ = CONFIGS[name]
    d = os.path.join(str(tmp), f"lor_{name}_{store}")
    return d if os.path.isdir(d) else write_folder(d, cfg, seed, getattr(torch, store))


@functools.lru_cache(maxsize=None)
def _model(folder):
    return read_model(folder)


@functools.lru_cache(maxsize=64)
def _logits(folder, tokens):
    cfg, W = _model(folder)
    return plain.forward(cfg, W, list(tokens)).numpy()


def plain_logits(folder, tokens):
    """float64 logits (T, V) of the plain implementation for one whole sequence"""
    return _logits(folder, tuple(int(t) for t in tokens))


def prompts_for(name, lengths, seed=0):
    rng = np.random.default_rng(seed)
    return [rng.integers(0, CONFIGS[name][0].vocab, n).tolist() for n in lengths]


def row_nmse(got, want):
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    return ((got - want) ** 2).sum(-1) / np.maximum((want ** 2).sum(-1), 1e-300)


# float32 against the float64 plain model: every product and sum is float32.  bfloat16 against the exact model: a row may
# reach the bar, a tenth of the rows more than that (a token whose last chosen expert is a close call gets another
# expert than the exact model gives it, and the rows that see it inherit the difference), and the median over the rows a
# tenth of the bar.
BAR = {"float32": 1e-9, "bfloat16": 1e-2}
BAR_SAME = {"float32": 1e-10, "bfloat16": 1e-2}


def assert_close(got, want, dtype, what, bar=None):
    got = np.asarray(got, np.float64)
    assert got.shape == np.asarray(want).shape, (what, got.shape, np.asarray(want).shape)
    assert np.isfinite(got).all(), f"{what}: non-finite logits"
    e = row_nmse(got, want)
    limit = (bar or BAR)[dtype]
    if dtype == "float32":
        assert e.max() <= limit, f"{what}: float32 NMSE {e.max():.3e} at row {int(e.argmax())}"
    else:
        over = int((e > limit).sum())
        assert over <= len(e) // 10 and np.median(e) <= limit / 10, \
            f"{what}: bfloat16: {over} of {len(e)} rows over {limit:.0e}, worst {e.max():.3e} at row {int(e.argmax())}, " \
            f"median {np.median(e):.3e}"
    return float(e.max())
