"""-m gpu: the Lorozen decoder in the engine against the plain implementation (tests/plain/lorozen.py), in float32 and
bfloat16.  Single kernels on inputs built so that a fault shows: attention with a sink over a window, every kernel form, with
ONE loud key just inside and just outside the window, at a page's border, at the query's own position and after it, in
prompts and decoded, and with loud and quiet sinks, while the pages behind the window are given back and hold loud garbage;
latent attention with a window and a gate per head alike; the mix with the token before, the decays, the recurrence and its
norm across cuts and slots; experts weighted at their input; the gelu-gated unit; capped logits.  Then the model layer by
layer, whole prompts, prefill against token-by-token decoding, portions down to two tokens, batches of unequal requests
against each alone, pages and state slots used again, long decoding, and greedy generation through the engine's own entry
point."""
import math

import numpy as np
import pytest
import torch

from tests import lorozen_helpers as S
from tests.gpu_harness import DEV, i32
from tests.plain import lorozen as plain

pytestmark = pytest.mark.gpu
DTYPES = ("float32", "bfloat16")
TD = {"float32": torch.float32, "bfloat16": torch.bfloat16}
KERNEL_BAR = {"float32": 2e-5, "bfloat16": 2e-2}          # of the largest value
F64 = torch.float64


def kernel_close(got, want, dtype, what, bar=None):
    got, want = np.asarray(got.detach().float().cpu(), np.float64), np.asarray(want, np.float64)
    assert got.shape == want.shape, (what, got.shape, want.shape)
    err = np.abs(got - want).max() / max(np.abs(want).max(), 1e-30)
    assert np.isfinite(got).all() and err <= (bar or KERNEL_BAR[dtype]), \
        f"{what}: {dtype} worst error {err:.3e} of the largest value"


def rnd(g, *shape, dtype="float32", scale=1.0):
    """random values that the storage dtype holds exactly, as float64"""
    return (torch.randn(*shape, generator=g) * scale).to(TD[dtype]).double()


def dev(t, dtype="float32"):
    return t.to(DEV, TD[dtype]).contiguous()


# ------------------------------------------------------------------------------------------------ attention
class Step:
    """what the attention's plan and kernels read of a step"""

    def __init__(self, dtype, lengths, q_lens, page, pages, options):
        from mashbox_b200 import ops
        from mashbox_b200.parts.base import StepInputs, Workspace
        n = len(lengths)
        self.ops, self.device, self.dtype, self.options, self.memo = ops, DEV, TD[dtype], dict(options), {}
        self.err = torch.zeros(1, dtype=torch.int32, device=DEV)
        self.N, self.S, self.q_len = sum(q_lens), n, list(q_lens)
        self.pos0 = [a - b for a, b in zip(lengths, q_lens)]
        self.q_start = [int(v) for v in np.concatenate([[0], np.cumsum(q_lens)[:-1]])]
        self.ws, self.inputs = Workspace(DEV, self.N), StepInputs(DEV)
        for name, v in (("q_start", self.q_start), ("q_len", q_lens), ("pos0", self.pos0), ("seq_row", range(n)),
                        ("positions", np.concatenate([p + np.arange(k) for p, k in zip(self.pos0, q_lens)])),
                        ("tok_row", np.repeat(np.arange(n), q_lens))):
            self.inputs.add(name, np.asarray(list(v), np.int32))

        class Cache:
            page_size, pool_pages = page, pages
        self.cache = Cache()

    def dev(self, name):
        return self.inputs.get(name)


class WindowCase:
    """S sequences in shuffled pages, the last q_len positions of each the step's queries.  Pages behind the window of every
    query are given back (-1 in the table); every slot that holds no key is loud garbage.  latent: one row per position that
    is key and, in its first DV values, value.  sinks: a score per head, or None; gated: a gate per token and head."""

    def __init__(self, dtype, H, KV, DK, DV, window, lengths, q_lens, page, loud=(), seed=0, amount=4.0, sinks=None, gated=False,
                 latent=False):
        g = torch.Generator().manual_seed(seed)
        self.__dict__.update(dtype=dtype, H=H, KV=KV, DK=DK, DV=DV, window=window, lengths=lengths, q_lens=q_lens, page=page,
                             latent=latent)
        self.q = [rnd(g, n, H, DK, dtype=dtype) for n in lengths]
        self.k = [rnd(g, n, KV, DK, dtype=dtype) for n in lengths]
        self.v = [k[..., :DV].clone() if latent else rnd(g, n, KV, DV, dtype=dtype, scale=0.25) for k, n in zip(self.k, lengths)]
        for (s, qpos, kpos) in loud:            # one score that stands out, its value loud in the first channel
            d = torch.zeros(DK, dtype=F64)
            d[DK - 1] = amount
            self.q[s][qpos], self.k[s][kpos] = d, d
            if latent:
                self.k[s][kpos, :, 0] = 8.0
                self.v[s][kpos] = self.k[s][kpos][..., :DV]
            else:
                self.v[s][kpos] = 0.0
                self.v[s][kpos, :, 0] = 8.0
        self.sinks = None if sinks is None else torch.tensor([sinks + 0.3 * h for h in range(H)], dtype=torch.float32).double()
        self.gate = rnd(g, sum(q_lens), H, dtype=dtype) if gated else None
        total = sum(-(-n // page) for n in lengths) + 2
        perm = torch.randperm(total, generator=g).tolist()
        table = np.full((len(lengths), max(-(-n // page) for n in lengths) + 1), -1, np.int32)
        kpool = torch.full((total, KV, page, DK), 30.0, dtype=F64)
        vpool = torch.full((total, KV, page, DV), 30.0, dtype=F64)
        self.given_back = 0
        for s, (n, ql) in enumerate(zip(lengths, q_lens)):
            lo = max(0, n - ql - window + 1) if window else 0
            for b in range(-(-n // page)):
                if (b + 1) * page <= lo:
                    self.given_back += 1
                    continue
                pg = table[s, b] = perm.pop()
                for p in range(max(lo, b * page), min(n, (b + 1) * page)):
                    kpool[pg, :, p % page], vpool[pg, :, p % page] = self.k[s][p], self.v[s][p]
        self.table, self.pages = i32(table), total
        self.kpool = dev(kpool, dtype)
        self.vpool = self.kpool if latent else dev(vpool, dtype)

    def want(self, scale):
        out, at = [], 0
        for q, k, v, n, ql in zip(self.q, self.k, self.v, self.lengths, self.q_lens):
            ok = plain.visible(n, dict(size=self.window) if self.window else None)[n - ql:]
            G = self.H // self.KV
            s = torch.einsum("ihd,jhd->hij", q[n - ql:], k.repeat_interleave(G, 1)) * scale
            s = s.masked_fill(~ok[None], -math.inf)
            w = torch.softmax(s, -1) if self.sinks is None else plain.softmax_with_sink(s, self.sinks)
            o = torch.einsum("hij,jhd->ihd", w, v.repeat_interleave(G, 1))
            if self.gate is not None:
                o = o * torch.sigmoid(self.gate[at:at + ql])[:, :, None]
            at += ql
            out.append(o.reshape(ql, -1))
        return torch.cat(out)

    def run(self, scale, **options):
        from mashbox_b200.parts.attention import PagedAttention
        core = PagedAttention(self.H, self.KV, self.DK, self.window, scale, vdim=self.DV, sinks=self.sinks is not None,
                              gated=self.gate is not None)
        core.general = core.general or self.latent
        step = Step(self.dtype, self.lengths, self.q_lens, self.page, self.pages, options)
        core.prepare(step)
        step.inputs.upload()
        rows = torch.cat([q[n - ql:].reshape(ql, -1) for q, n, ql in zip(self.q, self.lengths, self.q_lens)])
        rows = dev(torch.cat([rows, torch.full((rows.shape[0], 8), 30.0, dtype=F64)], 1), self.dtype)
        out = torch.full((step.N, self.H * self.DV), float("nan"), device=DEV, dtype=TD[self.dtype])
        core.attend(step, rows, rows.stride(0), out, self.table, self.kpool, self.vpool,
                    sinks=dev(self.sinks) if self.sinks is not None else None,
                    gate=dev(self.gate, self.dtype) if self.gate is not None else None)
        assert int(step.err.item()) == 0
        return out


# (kernel form, heads, kv heads, key width, value width, page, options): the plain kernel in both types; the general
# tensor-core kernel whole and cut along the keys; the TMA kernel (decode form alone, cut, in clusters; prompt form) and the
# tcgen05 kernel (prompt form), at both head sizes, with 1 to 20 query heads a kv head
FORMS = [("plain", 4, 2, 16, 24, 8, {}), ("plain", 3, 1, 12, 20, 5, {}), ("plain", 2, 2, 64, 64, 16, {}),
         ("general", 8, 2, 32, 64, 16, {}), ("general", 4, 1, 128, 48, 8, {}), ("general", 20, 1, 48, 64, 16, {}),
         ("general", 4, 2, 64, 64, 16, dict(attention_kernel="mma")),
         ("fast", 8, 2, 64, 64, 16, {}), ("fast", 4, 1, 128, 128, 32, {}), ("fast", 2, 2, 128, 128, 8, {}),
         ("fast", 16, 1, 64, 64, 64, {}), ("fast", 8, 2, 64, 64, 16, dict(attention_clusters=False)),
         ("fast", 8, 2, 128, 128, 16, dict(attention_target_blocks=1)), ("fast", 20, 1, 64, 64, 16, {}),
         ("fast", 4, 2, 64, 64, 16, dict(attention_prefill_kernel="mma"))]


def edges(window, page, n):
    """keys that the last of n tokens asks for: around the window's edge, pages' borders and its own position"""
    q = n - 1
    border = (q - window // 2) // page * page
    ks = {q, q - 1, q - window + 1, q - window, border, border - 1, 0}
    return [k for k in sorted(ks) if 0 <= k <= q]


@pytest.mark.parametrize("form,H,KV,DK,DV,page,options", FORMS)
def test_windows_with_sinks_on_their_edges(form, H, KV, DK, DV, page, options):
    amount = 4.5 if DK <= 32 else 7.0           # the loud score stands well above sqrt(DK) times a unit normal
    for dtype in (DTYPES if form == "plain" else ("bfloat16",)):
        for window, n, sinks in ((70, 300, 2.0), (128, 513, -40.0), (1, 90, 1.0), (64, 2 * page + 70, 0.0), (200, 190, 3.0)):
            q = n - 1
            for kpos in edges(window, page, n):
                seen = q - kpos < window
                # the query decoded alone; at the end of a portion that starts inside a page; and among whole prompts
                for ql in (1, 37 if kpos % 2 else 2, n if n < 300 else 131):
                    if ql > n:
                        continue
                    case = WindowCase(dtype, H, KV, DK, DV, window, [n, 40], [ql, 1], page, [(0, q, kpos)], seed=kpos,
                                      amount=amount, sinks=sinks)
                    got, want = case.run(1.0, **options), case.want(1.0)
                    what = f"{form} window {window} n {n} key {kpos} {'seen' if seen else 'not seen'}, {ql} queries, sink {sinks}"
                    kernel_close(got, want, dtype, what, 3e-2 if dtype == "bfloat16" else None)
                    loud = float(want[ql - 1].view(H, DV)[:, 0].abs().min())
                    assert (loud > 2.0) == seen, (what, loud)


@pytest.mark.parametrize("form,H,KV,DK,DV,page,options", FORMS)
def test_sinks_from_silent_to_deafening(form, H, KV, DK, DV, page, options):
    """a sink far below the scores changes nothing, one far above them takes everything; between the two the weight of a
    single key shows it; one key or many, decoded and in portions; every head its own sink"""
    for dtype in (DTYPES if form == "plain" else ("bfloat16",)):
        for sinks in (-300.0, -3.0, 0.0, 4.0, 12.0, 90.0):
            for lengths, q_lens in (([1, 3], [1, 3]), ([200, 2], [1, 1]), ([150, 700], [150, 300])):
                case = WindowCase(dtype, H, KV, DK, DV, 300, lengths, q_lens, page, seed=int(sinks) + 400, sinks=sinks)
                got, want = case.run(DK ** -0.5, **options), case.want(DK ** -0.5)
                assert (float(want.abs().max()) < 1e-20) == (sinks == 90.0)
                if sinks == 90.0:
                    assert float(got.float().abs().max()) < 1e-20
                else:
                    kernel_close(got, want, dtype, f"{form} sinks {sinks}, {lengths} {q_lens}", 3e-2 if dtype == "bfloat16" else None)


@pytest.mark.parametrize("splits", [1, 2, 5, 16])
@pytest.mark.parametrize("H,KV,DK,DV", [(8, 2, 64, 64), (4, 1, 128, 128), (8, 2, 32, 64), (4, 4, 48, 16)])
def test_decode_form_cut_along_the_keys_counts_the_sink_once(H, KV, DK, DV, splits):
    for window in (300, 640, 100, None):
        case = WindowCase("bfloat16", H, KV, DK, DV, window, [1000, 130, 17, 720], [1, 1, 1, 1], 16,
                          [(3, 719, 719 - (window or 400) + 1)], seed=splits, amount=7.0, sinks=3.5)
        kernel_close(case.run(0.5, attention_splits=splits, attention_clusters=False), case.want(0.5), "bfloat16",
                     f"{splits} splits, window {window}", 3e-2)
    case = WindowCase("bfloat16", H, KV, DK, DV, 300, [1000, 700], [1, 1], 16, seed=splits, sinks=3.5)
    if DK == DV and splits > 1:
        kernel_close(case.run(0.2, attention_cluster_size=min(splits, 8)), case.want(0.2), "bfloat16", f"a cluster of {splits}", 3e-2)


@pytest.mark.parametrize("H,KV,DK,DV,window", [(8, 2, 64, 64, 96), (2, 1, 128, 128, 700), (8, 1, 64, 64, 31), (4, 2, 32, 64, 96),
                                               (3, 3, 24, 40, 96), (20, 1, 128, 128, None)])
def test_long_prompts_and_portions_with_sinks(H, KV, DK, DV, window):
    """hundreds of queries per sequence in one step, from the start and far from it, beside a decoded one"""
    for lengths, q_lens in (([600, 333], [600, 1]), ([1500, 900], [700, 257]), ([1030], [300])):
        case = WindowCase("bfloat16", H, KV, DK, DV, window, lengths, q_lens, 16, seed=window or 1, sinks=1.0)
        kernel_close(case.run(DK ** -0.5), case.want(DK ** -0.5), "bfloat16", f"{lengths} {q_lens}", 3e-2)


@pytest.mark.parametrize("H,DK,DV,page", [(8, 112, 96, 16), (18, 64, 48, 8), (3, 26, 22, 5), (4, 40, 32, 32)])
def test_latent_rows_with_windows_and_gates(H, DK, DV, page):
    """one row per position that is key and value at once, a window over it, a gate per token and head"""
    for dtype in DTYPES:
        for window, n in ((70, 300), (1, 90), (64, 2 * page + 70), (None, 150)):
            q = n - 1
            for kpos in edges(window or n + 3, page, n):
                seen = q - kpos < (window or n + 1)
                for ql in (1, 37, n):
                    case = WindowCase(dtype, H, 1, DK, DV, window, [n, 40], [min(ql, n), 1], page, [(0, q, kpos)], seed=kpos,
                                      amount=7.0, gated=True, latent=True)
                    got, want = case.run(1.0), case.want(1.0)
                    what = f"window {window} n {n} key {kpos} {'seen' if seen else 'not seen'}, {ql} queries"
                    kernel_close(got, want, dtype, what, 3e-2 if dtype == "bfloat16" else None)
        case = WindowCase(dtype, H, 1, DK, DV, 128, [900, 400], [260, 1], page, seed=3, gated=True, latent=True)
        kernel_close(case.run(DK ** -0.5), case.want(DK ** -0.5), dtype, "a long portion", 3e-2 if dtype == "bfloat16" else None)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,KV,DK,DV,RD,pairing,pad", [(4, 2, 16, 24, 8, 1, 0), (3, 1, 12, 20, 12, 0, 4), (2, 2, 64, 64, 32, 1, 0),
                                                       (5, 1, 10, 6, 6, 1, 3), (6, 3, 32, 8, 0, 0, 8)])
def test_biases_before_the_rotation(dtype, H, KV, DK, DV, RD, pairing, pad):
    from mashbox_b200 import ops
    gen = torch.Generator().manual_seed(DK + RD)
    page, lengths = 4, [11, 70]
    blocks = [-(-n // page) for n in lengths]
    pages = sum(blocks) + 2
    perm = torch.randperm(pages, generator=gen).tolist()
    table = np.full((2, max(blocks)), -1, np.int32)
    for s, nb in enumerate(blocks):
        for b in range(nb):
            table[s, b] = perm.pop()
    positions, tok_row = np.concatenate([np.arange(n) for n in lengths]), np.repeat([0, 1], lengths)
    N, width = len(positions), (H + KV) * DK + KV * DV
    rows, bias = rnd(gen, N, width + pad, dtype=dtype), rnd(gen, width)
    rot = dict(dims=RD, base=100.0)
    freqs = torch.tensor([100.0 ** (-2 * i / max(RD, 1)) for i in range(RD // 2)], dtype=torch.float32)
    r = dev(rows, dtype)
    kpool = torch.zeros(pages, KV, page, DK, device=DEV, dtype=TD[dtype])
    vpool = torch.zeros(pages, KV, page, DV, device=DEV, dtype=TD[dtype])
    err = torch.zeros(1, dtype=torch.int32, device=DEV)
    ops.norm_rope_kv_write(r, None, None, 1e-6, dev(freqs) if RD else None, RD, pairing, 1.0, i32(positions), i32(tok_row),
                           i32(table), kpool, vpool, H, KV, DK, DV, page, pages, err, norm=None, bias=dev(bias))
    assert int(err.item()) == 0
    b = rows[:, :width] + bias
    turned = lambda x: plain.rotate(x, torch.as_tensor(positions), rot, "halves" if pairing else "adjacent")
    kernel_close(r[:, :H * DK], turned(b[:, :H * DK].view(N, H, DK)).reshape(N, -1), dtype, "q in place")
    at = torch.as_tensor(table[tok_row, positions // page]).long().to(DEV), torch.as_tensor(positions % page).to(DEV)
    kernel_close(kpool[at[0], :, at[1]], turned(b[:, H * DK:(H + KV) * DK].view(N, KV, DK)), dtype, "keys in their pages")
    kernel_close(vpool[at[0], :, at[1]], b[:, (H + KV) * DK:].view(N, KV, DV), dtype, "values in their pages")
    kernel_close(r[:, (H + KV) * DK:], rows[:, (H + KV) * DK:], dtype, "what lies behind the keys is left alone", 1e-9)


# ------------------------------------------------------------------------------------------------ wkv
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D", [64, 100, 37, 1024])
def test_mix_with_the_token_before_across_cuts_and_slots(dtype, D):
    """three sequences in slots out of order, in portions of their own sizes (a portion of one token reads the kept row and
    replaces it), the kept rows in a wider state whose other values stay"""
    from mashbox_b200 import ops
    gen = torch.Generator().manual_seed(D)
    mu = torch.rand(5, D, generator=gen).float().double()
    lens, cuts, slots = [13, 5, 9], [[1, 2, 9, 1], [2, 1, 1, 1], [3, 1, 2, 3]], [2, 0, 3]
    hs = [rnd(gen, n, D, dtype=dtype) for n in lens]
    state = torch.full((5, D + 12), 3.0, device=DEV)
    state[:, :D] = 0.0
    at = [0, 0, 0]
    for step in range(4):
        q_len = [cuts[s][step] for s in range(3)]
        q_start = np.concatenate([[0], np.cumsum(q_len)[:-1]])
        N = sum(q_len)
        out = torch.full((5, N, D), float("nan"), device=DEV, dtype=TD[dtype])
        ops.token_mix(dev(torch.cat([hs[s][at[s]:at[s] + q_len[s]] for s in range(3)]), dtype), dev(mu), state[:, :D],
                      (i32(np.repeat([0, 1, 2], q_len)), i32(q_start), i32(q_len), i32(slots)), out)
        want = []
        for s in range(3):
            before = torch.cat([torch.zeros(1, D, dtype=F64), hs[s]])[at[s]:at[s] + q_len[s]]
            x = hs[s][at[s]:at[s] + q_len[s]]
            want.append(x[None] + (before - x)[None] * mu[:, None, :])
            at[s] += q_len[s]
        kernel_close(out, torch.cat(want, 1), dtype, f"step {step}", 1e-2 if dtype == "bfloat16" else 1e-6)
        for s in range(3):
            kernel_close(state[slots[s], :D], hs[s][at[s] - 1], "float32", f"kept row {s}", 1e-7)
    assert float(state[[1, 4], :D].abs().max()) == 0.0 and float((state[:, D:] - 3.0).abs().max()) == 0.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,dim,R", [(3, 16, 12), (1, 40, 1), (4, 64, 32), (2, 10, 7), (2, 128, 64), (5, 8, 16)])
def test_decays_and_the_current_tokens_share(dtype, H, dim, R):
    from mashbox_b200 import ops
    gen = torch.Generator().manual_seed(R)
    N, C = 9, H * dim
    rows = rnd(gen, N, 4 * C, dtype=dtype)
    low, w2, w0, u = rnd(gen, N, R, scale=2.0), rnd(gen, C, R, dtype=dtype, scale=R ** -0.5), rnd(gen, C, scale=3.0), rnd(gen, C)
    w0[0], w0[1] = 30.0, -30.0                  # a channel that forgets at once, one that never does
    z = torch.tanh(low) @ w2.T
    bent = torch.empty(N, R, device=DEV, dtype=TD[dtype])
    ops.tanh_rows(dev(low), bent)
    kernel_close(bent, torch.tanh(low), dtype, "tanh")
    r, k, v = (rows[:, i * C:(i + 1) * C] for i in range(3))
    for kw in (dict(z=dev(z)), dict(low=dev(low), w2=dev(w2, dtype))):
        o = [torch.full((N, C), float("nan"), device=DEV) for _ in range(4)]
        share = torch.full((N, H), float("nan"), device=DEV)
        ops.wkv_gates(dev(rows, dtype), dev(w0), dev(u), *o, share, H, dim, **kw)
        for got, want, what in zip(o, (r, k, v, torch.exp(-torch.exp(z + w0))), ("r", "k", "v", "decay")):
            kernel_close(got, want, "float32", what)
        kernel_close(share, (r * u * k).view(N, H, dim).sum(-1), "float32", "share")


@pytest.mark.parametrize("H,dim", [(3, 16), (1, 40), (2, 64), (2, 128), (2, 6), (1, 20), (1, 256), (9, 10)])
def test_recurrence_reads_before_it_writes_and_carries_its_state(H, dim):
    """three sequences side by side in portions of their own sizes, in slots out of order; decays of one and of zero among
    the others; a first token's output is its own share alone"""
    from mashbox_b200 import ops
    gen = torch.Generator().manual_seed(dim)
    lens, cuts, slots = [337, 5, 190], [[1, 2, 330, 4], [2, 1, 1, 1], [33, 1, 2, 154]], [2, 0, 3]
    state = torch.zeros(5, H * dim * dim + 4, device=DEV)
    view = state[:, 4:]
    rs, ks, vs = ([rnd(gen, n, H, dim) for n in lens] for _ in range(3))
    ds = [torch.exp(-torch.exp(rnd(gen, n, H, dim) * 2 - 2)).float().double() for n in lens]
    ds[0][:, :, 0], ds[2][:, :, -1] = 1.0, 0.0
    bs = [rnd(gen, n, H) for n in lens]
    at, got = [0, 0, 0], [[], [], []]
    for step in range(4):
        q_len = [cuts[s][step] for s in range(3)]
        q_start = np.concatenate([[0], np.cumsum(q_len)[:-1]])
        cat = lambda xs: dev(torch.cat([xs[s][at[s]:at[s] + q_len[s]].reshape(q_len[s], -1) for s in range(3)]))
        o = torch.full((sum(q_len), H * dim), float("nan"), device=DEV)
        ops.gated_scan(cat(rs), cat(ks), cat(vs), cat(ds), o, view, (i32(q_start), i32(q_len), i32(slots)), H, H, dim, dim,
                       per_head=False, bonus=cat(bs))
        for s in range(3):
            got[s].append(o[q_start[s]:q_start[s] + q_len[s]].cpu())
            at[s] += q_len[s]
    for s in range(3):
        S_ = torch.zeros(H, dim, dim, dtype=F64)
        want = torch.zeros(lens[s], H, dim, dtype=F64)
        for t in range(lens[s]):
            want[t] = (S_ * rs[s][t][:, :, None]).sum(1) + bs[s][t][:, None] * vs[s][t]
            S_ = ds[s][t][:, :, None] * S_ + ks[s][t][:, :, None] * vs[s][t][:, None, :]
        kernel_close(torch.cat(got[s]), want.view(lens[s], -1), "float32", f"sequence {s}", 5e-5)
        kernel_close(view[slots[s]].view(H, dim, dim), S_, "float32", f"state {s}", 5e-5)
        kernel_close(got[s][0][0], (bs[s][0][:, None] * vs[s][0]).reshape(-1), "float32", "the first token")
    assert float(state[[1, 4]].abs().max()) == 0.0 and float(state[:, :4].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", DTYPES)
def test_norm_per_head_with_a_weight_per_head(dtype):
    from mashbox_b200 import ops
    gen = torch.Generator().manual_seed(5)
    for H, dim, pad in ((3, 10, 5), (4, 64, 8), (2, 300, 0), (3, 512, 8)):
        N = 7
        o, w, gate = rnd(gen, N, H * dim), rnd(gen, H, dim) + 1, rnd(gen, N, H * dim + pad, dtype=dtype, scale=2.0)
        o[1] *= 1e-4                            # a row whose mean square is below eps
        out = torch.empty(N, H * dim, device=DEV, dtype=TD[dtype])
        ops.gated_rms(dev(o), dev(gate, dtype), dev(w), out, H, dim, 1e-5, silu=True)
        want = (plain.rms(o.view(N, H, dim), 1e-5) * w).reshape(N, -1) * plain.silu(gate[:, :H * dim])
        kernel_close(out, want, dtype, f"{H} heads of {dim}")
        kernel_close(out[1], want[1], dtype, "the quiet row")


@pytest.mark.parametrize("dtype", DTYPES)
def test_products_of_several_inputs_side_by_side(dtype):
    from mashbox_b200 import ops
    ops.configure({})
    gen = torch.Generator().manual_seed(6)
    for G, N, M, K in ((4, 1, 128, 64), (4, 2, 256, 320), (4, 16, 1024, 1000), (3, 7, 384, 72), (4, 5, 48, 64), (4, 40, 128, 64),
                       (2, 200, 136, 72), (4, 3, 30, 37), (4, 9, 2048, 2048)):
        a, w = rnd(gen, G, N, K, dtype=dtype), rnd(gen, G * M, K, dtype=dtype, scale=K ** -0.5)
        out = torch.full((N, G * M), float("nan"), device=DEV, dtype=TD[dtype])
        ops.linear_groups(dev(a, dtype), dev(w, dtype), out)
        want = torch.cat([a[g] @ w[g * M:(g + 1) * M].T for g in range(G)], 1)
        kernel_close(out, want, dtype, f"{G} products {N} x {M} x {K}")


# ------------------------------------------------------------------------------------------------ feed-forward, logits, stream
@pytest.mark.parametrize("D,F,E,top", [(64, 32, 8, 2), (64, 40, 5, 5), (100, 28, 3, 1), (256, 128, 16, 4), (48, 24, 1, 1)])
def test_experts_weighted_at_their_input(D, F, E, top):
    """a step of few tokens, of some and of many (three kernel forms in bfloat16); the weights far from one, so that weighing
    the outputs would show"""
    from mashbox_b200.parts.base import Env, PartSpec, Workspace, make
    from mashbox_b200 import ops
    gen = torch.Generator().manual_seed(E)
    for dtype in DTYPES:
        W = {f"mlp.e{e}.{r}": rnd(gen, *((D, F) if r == "down" else (F, D)), dtype=dtype, scale=(F if r == "down" else D) ** -0.5)
             for e in range(E) for r in ("gate", "up", "down")}
        W["mlp.router"] = rnd(gen, E, D, dtype=dtype, scale=0.7 * D ** -0.5)
        W.update({"mlp.shared." + r: rnd(gen, *((D, 24) if r == "down" else (24, D)), dtype=dtype, scale=0.2)
                  for r in ("gate", "up", "down")})
        shared = PartSpec("swiglu", hidden=D, intermediate=24, names=dict(gate="gate", up="up", down="down"))
        part = make("feed_forward", PartSpec("routed_experts", hidden=D, intermediate=F, experts=E, top=top, limit=None, alpha=1.0,
                                             shift=0.0, correction=False, weigh="input", shared=shared))
        part.bind({k + (".weight" if ".shared." in k else ""): dev(v, dtype) for k, v in W.items()},
                  Env(TD[dtype], torch.device(DEV), ops))
        for N in (1, 5, 40, 300):
            class Ctx:
                pass
            ctx = Ctx()
            ctx.ops, ctx.N, ctx.dtype, ctx.options, ctx.ws = ops, N, TD[dtype], {}, Workspace(DEV, 320)
            h = rnd(gen, N, D, dtype=dtype, scale=2.0)
            got, _ = part.forward(ctx, dev(h, dtype))
            # the plain choice, made on the logits as the product's float32 result has them
            want = plain.experts(W, "mlp.", dict(router=dict(top=top), shared=dict(ff=24)), h)
            kernel_close(got, want, dtype, f"{N} tokens, {top} of {E} experts")
            late = plain.experts(W, "mlp.", dict(router=dict(top=top)), h * 0)        # nothing without the shared expert
            assert float(late.abs().max()) == 0.0


@pytest.mark.parametrize("dtype", DTYPES)
def test_gelu_gate_alone_and_in_the_products_epilogue(dtype):
    from mashbox_b200 import ops
    ops.configure({})
    gen = torch.Generator().manual_seed(1)
    for N, F in ((6, 37), (5, 64)):
        gu = rnd(gen, N, 2 * F, dtype=dtype, scale=3.0)
        gu[0, 0], gu[0, 1] = -60.0, 60.0
        out = torch.empty(N, F, device=DEV, dtype=TD[dtype])
        ops.geglu(dev(gu, dtype), out)
        kernel_close(out, plain.gelu_tanh(gu[:, :F]) * gu[:, F:], dtype, "gelu(gate) up", 1e-2 if dtype == "bfloat16" else None)
    if dtype == "bfloat16":
        # one token (matrix-vector, short and long rows), a decode batch (weight-streaming), prompt portions (tcgen05)
        for N, F, K in ((1, 264, 64), (1, 72, 8448), (1, 40, 2568), (2, 96, 1024), (5, 136, 4096), (16, 1032, 328), (9, 24, 72),
                        (128, 256, 64), (200, 264, 328), (515, 1032, 128)):
            a, w = rnd(gen, N, K, dtype=dtype), rnd(gen, 2 * F, K, dtype=dtype, scale=2 * K ** -0.5)
            out = torch.full((N, F), float("nan"), device=DEV, dtype=torch.bfloat16)
            assert ops.fused_swiglu_supports(N, F, K)
            ops.linear_swiglu(dev(a, dtype), dev(w, dtype), out, "geglu")
            kernel_close(out, plain.gelu_tanh(a @ w[:F].T) * (a @ w[F:].T), dtype, f"product {N} x {F} x {K}")


def test_capped_logits():
    from mashbox_b200 import ops
    gen = torch.Generator().manual_seed(2)
    y = rnd(gen, 5, 301, scale=20.0)
    y[0, 0], y[0, 1] = 1e4, -1e4
    for cap in (15.0, 0.5):
        got = dev(y)
        ops.softcap_rows(got, cap)
        kernel_close(got, cap * torch.tanh(y / cap), "float32", f"cap {cap}", 1e-6)


@pytest.mark.parametrize("dtype", DTYPES)
def test_normed_output_and_a_row_that_joins_the_stream(dtype):
    from mashbox_b200 import ops
    gen = torch.Generator().manual_seed(4)
    for N, D in ((3, 64), (2, 37), (4, 2048)):
        x, y, again, w, nw = rnd(gen, N, D), rnd(gen, N, D, dtype=dtype), rnd(gen, N, D), rnd(gen, D), rnd(gen, D)
        for joins in (False, True):
            xs = dev(x)
            normed = torch.empty(N, D, device=DEV, dtype=TD[dtype])
            ops.post_norm_add(xs, dev(y, dtype), dev(w), 1e-5, dev(nw), 1e-6, normed, again=dev(again) if joins else None)
            want = x + plain.rms(y, 1e-5, w) + (again if joins else 0.0)
            kernel_close(xs, want, "float32", f"stream of {D}, joins {joins}")
            kernel_close(normed, plain.rms(want, 1e-6, nw), dtype, "the next norm")


# ------------------------------------------------------------------------------------------------ the model in the engine
def runner_for(tmp, name, dtype, max_tokens, options=None, max_requests=4):
    from mashbox_b200.engine.replay import make_runner
    folder = S.make_folder(tmp, name, "float32" if dtype == "float32" else "bfloat16")
    return folder, make_runner(folder, dtype, max_tokens, page_size=S.CONFIGS[name][2], options=options,
                               max_requests=max_requests)


def replay(runner, steps):
    from mashbox_b200.engine.replay import run_step
    out = {}
    for i, s in enumerate(steps):
        r = run_step(runner, dict(s, step=i))
        if r is not None:
            out[i] = r.numpy()
    return out


def cut_steps(rid, tokens, cuts, end=True):
    """the steps that feed `tokens` in portions of the given sizes, asking for every position's logits"""
    steps, at = [], 0
    for n in cuts:
        steps.append(dict(entries=[dict(id=rid, tokens=tokens[at:at + n], want=list(range(n)))], end=[]))
        at += n
    assert at == len(tokens)
    if end:
        steps[-1]["end"] = [rid]
    return steps


def joined(out):
    return np.concatenate([out[i] for i in sorted(out)])


CASES = [(n, d) for n in S.CONFIGS for d in DTYPES]


@pytest.mark.parametrize("name", ["P", "Q", "Z"])
def test_layer_by_layer(tmp_path_factory, name):
    """float32: the model cut after its first, second, ... layer (a tensor's values depend on its name and the seed alone,
    so the shorter models are the longer one's beginnings) against the plain implementation cut alike"""
    import dataclasses
    import os
    from mashbox_b200.engine.replay import make_runner
    from tests.plain.llama import read_model
    cfg, seed, page = S.CONFIGS[name]
    tmp = tmp_path_factory.mktemp("layers")
    (p,) = S.prompts_for(name, (75,))
    for n in range(1, len(cfg.layers) + 1):
        lp = cfg.loop
        if lp and n < lp.stop:                  # the loop ends with the model, or is not reached
            lp = dataclasses.replace(lp, stop=n) if n > lp.start else None
        d = S.write_folder(os.path.join(str(tmp), f"first{n}"), dataclasses.replace(cfg, layers=cfg.layers[:n], loop=lp), seed,
                           torch.float32)
        c, W = read_model(d)
        got = joined(replay(make_runner(d, "float32", 128, page_size=page), cut_steps("a", p, [len(p)])))
        S.assert_close(got, plain.forward(c, W, p).numpy(), "float32", f"{name}: the first {n} layers ({cfg.layers[n - 1].type} last)")


@pytest.mark.parametrize("seed", range(12))
def test_configurations_drawn_at_random(tmp_path_factory, seed):
    """2 to 5 layers of any kind in any order, looped or not, with sizes drawn from small sets: a whole prompt, then the same prompt in
    portions and single tokens"""
    import os
    from mashbox_b200.engine.replay import make_runner
    from tests.plain.llama import read_model
    cfg = S.random_config(seed)
    page = (4, 8, 16, 5)[seed % 4]
    tmp = tmp_path_factory.mktemp("r")
    p = np.random.default_rng(seed).integers(0, cfg.vocab, 75).tolist()
    for dtype in DTYPES:
        d = S.write_folder(os.path.join(str(tmp), dtype), cfg, 700 + seed, TD[dtype])
        c, W = read_model(d)
        want = plain.forward(c, W, p).numpy()
        runner = make_runner(d, dtype, 128, page_size=page)
        what = f"random configuration {seed}: {[x.type for x in cfg.layers]}"
        S.assert_close(joined(replay(runner, cut_steps("a", p, [len(p)]))), want, dtype, what + ", whole")
        S.assert_close(joined(replay(runner, cut_steps("b", p, [33, 2, 1, 17, 1, 1, 20]))), want, dtype, what + ", in portions")
        runner.cache.check()


@pytest.mark.parametrize("name,dtype", CASES)
def test_whole_prompts_and_first_tokens(tmp_path_factory, name, dtype):
    folder, runner = runner_for(tmp_path_factory.mktemp("m"), name, dtype, 320)
    for p in S.prompts_for(name, (1, 2, 3, 5, 21, 64, 65, 150, 300)):
        S.assert_close(joined(replay(runner, cut_steps("a", p, [len(p)]))), S.plain_logits(folder, p), dtype,
                       f"{name}: whole prompt of {len(p)}")
    runner.cache.check()
    assert runner.cache.free_pages() == [runner.cache.num_pages] * len(runner.cache.groups)


@pytest.mark.parametrize("name,dtype", CASES)
def test_prefill_against_token_by_token(tmp_path_factory, name, dtype):
    """every token alone from the first one, over many pages, against the whole prompt in one step and against the
    plain implementation; a second request in the same state slot and pages right after starts from nothing"""
    folder, runner = runner_for(tmp_path_factory.mktemp("m"), name, dtype, 192, max_requests=1)
    p, p2 = S.prompts_for(name, (170, 30), seed=1)
    whole = joined(replay(runner, cut_steps("a", p, [len(p)])))
    single = joined(replay(runner, cut_steps("b", p, [1] * len(p))))
    S.assert_close(single, S.plain_logits(folder, p), dtype, f"{name}: 170 tokens one by one")
    S.assert_close(single, whole, dtype, f"{name}: one by one against one step", S.BAR_SAME)
    again = joined(replay(runner, cut_steps("c", p2, [len(p2)])))
    S.assert_close(again, S.plain_logits(folder, p2), dtype, f"{name}: a request in a slot that was used before")
    runner.cache.check()


@pytest.mark.parametrize("name,dtype", CASES)
def test_portions_of_every_size(tmp_path_factory, name, dtype):
    folder, runner = runner_for(tmp_path_factory.mktemp("m"), name, dtype, 256)
    (p,) = S.prompts_for(name, (230,), seed=2)
    want = S.plain_logits(folder, p)
    whole = joined(replay(runner, cut_steps("w", p, [len(p)])))
    for cuts in ([2] * 115, [3, 37, 1, 2, 64, 17, 2, 2, 1, 50, 33, 5, 7, 6], [7, 8, 9, 1, 15, 16, 17, 157],
                 [63, 1, 1, 63, 2, 62, 38], [128, 2, 100]):
        got = joined(replay(runner, cut_steps("a", p, cuts)))
        S.assert_close(got, want, dtype, f"{name}: portions {cuts[:6]}...")
        S.assert_close(got, whole, dtype, f"{name}: portions {cuts[:6]}... against one step", S.BAR_SAME)
    runner.cache.check()


@pytest.mark.parametrize("name,dtype", CASES)
def test_unequal_requests_side_by_side_with_pages_and_slots_used_again(tmp_path_factory, name, dtype):
    """Two requests at most are live, portions of some beside single tokens of others; the pool holds less than all
    requests together, and two state slots only, so pages and slots come back and are taken again.  Every request's
    logits must be those it has alone."""
    from mashbox_b200.engine.replay import run_step
    folder, runner = runner_for(tmp_path_factory.mktemp("m"), name, dtype, 224, max_requests=2)
    prompts = dict(zip("abcdef", S.prompts_for(name, (90, 47, 3, 110, 66, 21), seed=3)))
    plans = dict(a=[30, 1, 1, 2, 50, 1, 1, 1, 1, 1, 1], b=[1, 1, 20, 2, 23], c=[1, 2], d=[64, 1, 40, 2, 1, 1, 1],
                 e=[2, 62, 1, 1], f=[21])
    order = list("abcdef")
    at, turn, got = {r: 0 for r in order}, {r: 0 for r in order}, {r: [] for r in order}
    waiting, live, step = list(order), [], 0
    while waiting or live:
        while waiting and len(live) < 2:
            live.append(waiting.pop(0))
        entries, end = [], []
        for r in live:
            n = plans[r][turn[r]]
            entries.append(dict(id=r, tokens=prompts[r][at[r]:at[r] + n], want=list(range(n))))
            at[r] += n
            turn[r] += 1
            if turn[r] == len(plans[r]):
                assert at[r] == len(prompts[r])
                end.append(r)
        out = run_step(runner, dict(step=step, entries=entries, end=end)).numpy()
        o = 0
        for e in entries:
            got[e["id"]].append(out[o:o + len(e["tokens"])])
            o += len(e["tokens"])
        live = [r for r in live if r not in end]
        runner.cache.check()
        step += 1
    for r in order:
        S.assert_close(np.concatenate(got[r]), S.plain_logits(folder, prompts[r]), dtype, f"{name}: request {r} in a batch")
    assert runner.cache.free_pages() == [runner.cache.num_pages] * len(runner.cache.groups)


@pytest.mark.parametrize("options", [dict(plain_attention=True), dict(attention_splits=4), dict(attention_target_blocks=1),
                                     dict(attention_kernel="mma"), dict(attention_prefill_kernel="mma"),
                                     dict(plain_experts=True), dict(attention_folds_rotation=False)])
def test_every_kernel_form_gives_the_same_model(tmp_path_factory, options):
    """the forms the engine chooses between, forced"""
    folder, runner = runner_for(tmp_path_factory.mktemp("m"), "R", "bfloat16", 512, options=options)
    (p,) = S.prompts_for("R", (300,), seed=7)
    got = joined(replay(runner, cut_steps("a", p, [200, 70] + [1] * 30)))
    S.assert_close(got, S.plain_logits(folder, p), "bfloat16", f"R with {options}")


def test_tensor_core_attention_is_what_bfloat16_runs(tmp_path_factory):
    from mashbox_b200 import ops
    folder, runner = runner_for(tmp_path_factory.mktemp("m"), "R", "bfloat16", 192)
    (p,) = S.prompts_for("R", (150,), seed=8)
    replay(runner, cut_steps("a", p, [149, 1]))
    loaded = [k[0] for k in ops._fn_cache]
    for name in ("attention_tc5", "attention_tma", "attention_general_mma_32_64", "attention_general_mma_112_96", "gemm_tc5", "wkv"):
        assert name in loaded, (name, loaded)


@pytest.mark.parametrize("name,dtype", [("P", "float32"), ("P", "bfloat16"), ("R", "bfloat16"), ("S", "float32"),
                                        ("Z", "bfloat16")])
def test_long_decoding(tmp_path_factory, name, dtype):
    """a short prompt and 368 tokens one by one (graphs replayed), two requests side by side"""
    folder, runner = runner_for(tmp_path_factory.mktemp("m"), name, dtype, 896)
    a, b = S.prompts_for(name, (412, 380), seed=4)
    steps = [dict(entries=[dict(id="a", tokens=a[:12], want=[11])], end=[]),
             dict(entries=[dict(id="a", tokens=a[12:44], want=[31]), dict(id="b", tokens=b[:3], want=[2])], end=[])]
    for i in range(400 - 32):
        e = [dict(id="a", tokens=[a[44 + i]], want=[0])]
        if 3 + i < len(b):
            e.append(dict(id="b", tokens=[b[3 + i]], want=[0]))
        steps.append(dict(entries=e, end=[]))
    out = replay(runner, steps)
    wa, wb = S.plain_logits(folder, a), S.plain_logits(folder, b)
    ga = np.stack([out[0][0], out[1][0]] + [out[2 + i][0] for i in range(368)])
    gb = np.stack([out[1][1]] + [out[2 + i][1] for i in range(368)])
    S.assert_close(ga, wa[[11, 43] + list(range(44, 412))], dtype, f"{name}: 368 tokens decoded, request a")
    S.assert_close(gb, wb[[2] + list(range(3, 371))], dtype, f"{name}: 368 tokens decoded, request b")
    assert runner.stats["graph_replays"] > 300
    runner.cache.check()


def test_windows_free_pages_for_a_pool_smaller_than_the_sequence(tmp_path_factory):
    """400 tokens decoded in a pool of 96: it holds them only because pages behind the windows come back, in every pass of
    the loop"""
    import dataclasses
    import os
    from mashbox_b200.config.engine import EngineConfig
    from mashbox_b200.engine.loading import load_model
    from mashbox_b200.engine.runner import ModelRunner
    from tests.plain.llama import read_model
    cfg = dataclasses.replace(S.LOR_P, layers=S.LOR_P.layers[:3], loop=S.Loop(0, 3, 2))
    d = S.write_folder(os.path.join(str(tmp_path_factory.mktemp("w")), "m"), cfg, 9, torch.float32)
    runner = ModelRunner(load_model(d, dtype="float32", device=DEV),
                         EngineConfig(dtype="float32", page_size=8, max_tokens=96, max_requests=2, max_tokens_per_step=64,
                                      max_context=448, chunk=64, device=DEV))
    p = np.random.default_rng(1).integers(0, cfg.vocab, 400).tolist()
    got = joined(replay(runner, cut_steps("a", p, [20, 30] + [1] * 350)))
    c, W = read_model(d)
    S.assert_close(got, plain.forward(c, W, p).numpy(), "float32", "400 tokens in a pool of 96")
    runner.cache.check()


@pytest.mark.parametrize("name", ["P", "S"])
def test_the_embedding_joins_behind_a_block_that_does_not_take_it_in(tmp_path_factory, monkeypatch, name):
    """a block that leaves what joins the stream to the model, after it has made the next norm's output already"""
    from mashbox_b200.parts.block import SandwichBlock
    own = SandwichBlock.forward

    def forward(self, ctx, x, pending, run):
        rows = ctx.take_joining()
        pending = own(self, ctx, x, pending, run)
        ctx.joining = rows
        return pending
    monkeypatch.setattr(SandwichBlock, "forward", forward)
    for dtype in DTYPES:
        folder, runner = runner_for(tmp_path_factory.mktemp("m"), name, dtype, 128)
        (p,) = S.prompts_for(name, (60,), seed=9)
        got = joined(replay(runner, cut_steps("a", p, [30, 2] + [1] * 28)))
        S.assert_close(got, S.plain_logits(folder, p), dtype, f"{name}: joined by the model")


@pytest.mark.parametrize("name,dtype", [("P", "float32"), ("Q", "float32"), ("R", "bfloat16"), ("S", "float32")])
def test_greedy_generation_through_the_engine(tmp_path_factory, name, dtype):
    """Engine.generate with its scheduler, graphs and sampler: three prompts of unequal length in portions of at most
    32 tokens; in float32 the ids are the plain implementation's greedy ids."""
    from mashbox_b200.engine.engine import Engine
    folder = S.make_folder(tmp_path_factory.mktemp("m"), name, "float32" if dtype == "float32" else "bfloat16")
    eng = Engine.from_folder(folder, dtype=dtype, page_size=S.CONFIGS[name][2], max_tokens=512, max_requests=3, chunk=32,
                             max_tokens_per_step=40)
    prompts = S.prompts_for(name, (70, 5, 33), seed=5)
    new = 40
    r = eng.generate(prompts, max_new=new)
    assert r["finish"] == ["length"] * 3 and all(len(ids) == new for ids in r["ids"])
    again = eng.generate(prompts, max_new=new)                            # captured graphs now
    assert again["ids"] == r["ids"]
    assert eng.runner.stats["graph_replays"] > 0
    for p, ids in zip(prompts, r["ids"]):
        lg = S.plain_logits(folder, p + ids)
        for t, tok in enumerate(ids):
            row = lg[len(p) + t - 1]
            best = int(row.argmax())
            if dtype == "float32":
                assert tok == best or row[best] - row[tok] < 1e-4, f"{name}: token {t} is {tok}, plain says {best}"
            else:                                                          # bf16 may pick another of two near-equal ids
                assert row[best] - row[tok] < 0.05 * (row.max() - row.min()), f"{name}: token {t} = {tok} is far from the best"
    eng.cache.check()
