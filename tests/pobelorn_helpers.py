"""Small Pobelorn configurations with random weights, and the plain implementation's logits for them."""
import functools
import os

import numpy as np
import torch

from mashbox_b200.config.pobelorn import (AttentionMixer, DenseFF, ExpertsFF, LightningMixer, PobelornConfig, PobelornLayer,
                                          Rotation)
from tests.plain import pobelorn as plain
from tests.plain.llama import read_model


def att(heads, kv, dim, vdim, scale, rot=0, base=10000.0, scaling=None, window=None, keep=0, mix=False):
    return AttentionMixer(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale,
                          rot=Rotation(rot, base, scaling) if rot else None, window=window, keep_first=keep, v_mix=mix)


def light(heads, dim, vdim, decay):
    return LightningMixer(heads=heads, dim=dim, vdim=vdim, decay=tuple(decay))


def model(width, vocab, eps, scale, *layers):
    return PobelornConfig("Pobelorn", width=width, vocab=vocab, norm_eps=eps, embedding_scale=scale, layers=tuple(
        PobelornLayer("lightning" if isinstance(m, LightningMixer) else "attention", m, f) for m, f in layers))


# P: every size differs from layer to layer where it may: windows of 21, 33 and 1 position and none, kept tokens that are
#    no multiple of a page, none of them, more than the window holds; layers that mix values with the first (48 values a
#    token in heads of 24, 16 and 12) and one between that does not; a rotation bent in part, a whole one, none; experts
#    with and without a shared one, one chosen and all chosen; a dense unit; no feed-forward
POB_P = model(64, 131, 1e-5, 3.0,
              (att(4, 2, 16, 24, 0.3, 8, 100.0, (4.0, 64.0, 8.0, 0.5), 21, 5, True), DenseFF(96)),
              (light(3, 16, 24, (0.5, 0.9, 0.995)), ExpertsFF(32, 12, 3, 40)),
              (att(6, 3, 24, 16, 0.2, 24, 500.0, None, 33, 0, True), ExpertsFF(24, 6, 1, None)),
              (att(2, 1, 32, 8, 0.25), None),
              (att(4, 4, 8, 12, 0.4, 2, 50.0, (2.0, 32.0, 4.0, 1.0), 1, 3, True), ExpertsFF(16, 4, 4, 16)))
# Q: a lightning layer first and two in a row; more query heads on one kv head than a decode tile has rows; kept tokens and
#    windows that are multiples of the page; no mixing; a head rotated whole with every frequency bent; embedding scale 1
POB_Q = model(96, 89, 1e-6, 1.0,
              (light(1, 40, 24, (0.98,)), DenseFF(40)),
              (att(20, 1, 16, 16, 0.35, 16, 1e6, (8.0, 4096.0, 2.0, 1.0), 32, 16), ExpertsFF(40, 5, 2, 64)),
              (light(5, 8, 8, (0.6, 0.8, 0.9, 0.95, 0.9999)), None),
              (light(2, 24, 40, (0.9, 1.0)), ExpertsFF(24, 8, 2, None)))
# R: sizes the tensor-core kernels take: heads of 64 x 64 and 128 x 128 (the TMA and tcgen05 kernels, windows of 100 and 64
#    with 24 and 130 kept tokens, no window), 32 x 64 (the general one), lightning heads of 64 x 32
POB_R = model(128, 301, 2e-6, 2.0,
              (att(8, 2, 64, 64, 0.15, 32, 1e5, (2.0, 256.0, 16.0, 1.0), 100, 24, True), ExpertsFF(64, 16, 4, 96)),
              (light(4, 64, 32, (0.9, 0.99, 0.995, 0.999)), DenseFF(256)),
              (att(4, 1, 128, 128, 0.1, 128, 1e4, None, 64, 130, True), ExpertsFF(32, 4, 2, 32)),
              (att(6, 2, 32, 64, 0.2, 16, 1e4, None, 70, 9, True), DenseFF(128)),
              (att(16, 2, 64, 64, 0.15, 64, 1e4), ExpertsFF(64, 8, 2, None)))
# S: lightning layers only -- the model keeps nothing per position, the cache manager has no group and takes no page
POB_S = model(48, 61, 1e-5, 2.5,
              (light(2, 16, 8, (0.9, 0.99)), ExpertsFF(16, 4, 2, 8)),
              (light(1, 32, 48, (0.97,)), None))
# Z: sizes that are multiples of neither 8 nor 16, so that no 16-byte form of any kernel applies, a page of 5 positions
POB_Z = model(100, 53, 1e-5, 1.5,
              (att(3, 3, 10, 6, 0.3, 6, 300.0, (3.0, 32.0, 2.0, 0.25), 18, 7, True), DenseFF(28)),
              (light(3, 10, 6, (0.8, 0.9, 0.99)), ExpertsFF(12, 6, 2, 20)),
              (att(2, 2, 6, 9, 0.4, 4, 70.0, None, 11, 2, True), None),
              (att(5, 1, 14, 10, 0.25, 2, 70.0, None, 40, 13), ExpertsFF(28, 5, 3, 44)))
CONFIGS = {"P": (POB_P, 41, 8), "Q": (POB_Q, 42, 16), "R": (POB_R, 43, 16), "S": (POB_S, 44, 32),
           "Z": (POB_Z, 45, 5)}       # config, seed, page size

# Readers near 1/sqrt(fan in), writers into the stream moderate; the router wide enough that the chosen experts are seldom a
# close call, its bias of order 1 so that it matters
STD_BY_NAME = (("router.b", 0.7), ("mlp.router", 0.6), (".down", 0.15), ("mix.o", 0.15), ("embed", 0.4))


def random_config(seed):
    """a configuration drawn at random: 2 to 5 layers of any kind in any order, sizes from small sets that include 1, odd
    sizes, multiples of 16 (which the tensor-core kernels take) and keys wider and narrower than values"""
    rng = np.random.default_rng(2000 + seed)
    pick = lambda *xs: xs[int(rng.integers(len(xs)))]
    layers, mixed = [], None
    for _ in range(int(rng.integers(2, 6))):
        if pick(0, 0, 1):
            heads = pick(1, 2, 3)
            m = light(heads, pick(8, 16, 20, 40, 64), pick(8, 10, 16, 48), [pick(0.3, 0.9, 0.99, 0.999, 1.0) for _ in range(heads)])
        else:
            kv, dim, vdim = pick(1, 2, 3), pick(8, 10, 16, 32, 64), pick(8, 12, 16, 32, 64)
            mix = bool(pick(0, 1, 1))
            if mix and mixed is None:
                mixed = kv * vdim
            elif mix:
                kv = next(g for g in (kv, 2, 1) if mixed % g == 0)
                vdim = mixed // kv
            rot = pick(0, 2, dim // 2 - (dim // 2) % 2, dim)
            window = pick(None, 1, 7, 16, 40)
            m = att(kv * pick(1, 2, 4), kv, dim, vdim, pick(0.1, 0.2, 0.4), rot, pick(100.0, 1e4, 5e5),
                    pick(None, (2.0, 2048.0, 32.0, 1.0), (4.0, 64.0, 4.0, 0.5)), window, pick(0, 1, 4, 16, 23) if window else 0, mix)
        experts = pick(1, 4, 6, 16)
        f = pick(None, DenseFF(pick(16, 24, 40, 64)), ExpertsFF(pick(8, 24, 32), experts, min(experts, pick(1, 2, 4)),
                                                               pick(None, 16, 28)))
        layers.append((m, f))
    return model(pick(32, 48, 64, 96, 100), pick(50, 97, 128), pick(1e-5, 1e-6), pick(1.0, 2.5, 5.0), *layers)


def make_folder(tmp, name, store="float32"):
    from mashbox_b200.weights.random_init import write_model_folder
    cfg, seed, _ = CONFIGS[name]
    d = os.path.join(str(tmp), f"pob_{name}_{store}")
    if not os.path.isdir(d):
        write_model_folder(d, cfg, seed, dtype=getattr(torch, store), std=cfg.width ** -0.5, norm_std=0.1,
                           std_by_name=STD_BY_NAME)
    return d


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
# reach the bar, a twentieth of the rows more than that (a token whose last chosen expert is a close call gets another
# expert than the exact model gives it, and the rows that see it inherit the difference), and the median over the rows a
# fifth of the bar.
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
        assert over <= len(e) // 20 and np.median(e) <= limit / 5, \
            f"{what}: bfloat16: {over} of {len(e)} rows over {limit:.0e}, worst {e.max():.3e} at row {int(e.argmax())}, " \
            f"median {np.median(e):.3e}"
    return float(e.max())
