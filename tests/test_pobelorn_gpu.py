"""-m gpu: the Pobelorn decoder in the engine against the plain implementation (tests/plain/pobelorn.py), in float32 and
bfloat16.  Single kernels on inputs built so that a fault shows: attention over a window with kept first positions, every
kernel form, with ONE loud key just inside and just outside the window, the last kept and the first one that is not, at a
page's border, at the query's own position and after it, in prompts and decoded, while the pages between are given back
and hold loud garbage; head norms after the rotation with mixed values; activated projections; the choice of experts by
biased logits; the squared ReLU.  Then the model layer by layer, whole prompts, prefill against token-by-token decoding,
portions down to two tokens, batches of unequal requests against each alone, pages and state slots used again, long
decoding, and greedy generation through the engine's own entry point."""
import math

import numpy as np
import pytest
import torch

from tests import pobelorn_helpers as S
from tests.gpu_harness import DEV, i32
from tests.plain import pobelorn as plain

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


# ------------------------------------------------------------------------------------------------ windows with kept tokens
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
    """S sequences in shuffled pages, the last q_len positions of each the step's queries.  Pages that no query of the step
    can see are given back (-1 in the table); every slot that holds no key and every key outside the step's reach is
    loud garbage."""

    def __init__(self, dtype, H, KV, DK, DV, window, keep, lengths, q_lens, page, loud=(), seed=0, amount=4.0):
        g = torch.Generator().manual_seed(seed)
        self.__dict__.update(dtype=dtype, H=H, KV=KV, DK=DK, DV=DV, window=window, keep=keep, lengths=lengths, q_lens=q_lens,
                             page=page)
        self.q = [rnd(g, n, H, DK, dtype=dtype) for n in lengths]
        self.k = [rnd(g, n, KV, DK, dtype=dtype) for n in lengths]
        self.v = [rnd(g, n, KV, DV, dtype=dtype, scale=0.25) for n in lengths]
        for (s, qpos, kpos) in loud:            # one score that stands out, its value loud in the first channel
            d = torch.zeros(DK, dtype=F64)
            d[DK - 1] = amount
            self.q[s][qpos], self.k[s][kpos], self.v[s][kpos] = d, d, 0.0
            self.v[s][kpos, :, 0] = 8.0
        total = sum(-(-n // page) for n in lengths) + 2
        perm = torch.randperm(total, generator=g).tolist()
        table = np.full((len(lengths), max(-(-n // page) for n in lengths) + 1), -1, np.int32)
        kpool = torch.full((total, KV, page, DK), 30.0, dtype=F64)
        vpool = torch.full((total, KV, page, DV), 30.0, dtype=F64)
        self.given_back = 0
        for s, (n, ql) in enumerate(zip(lengths, q_lens)):
            lo = max(0, n - ql - window + 1) if window else 0
            for b in range(-(-n // page)):
                if window and b * page >= keep and (b + 1) * page <= lo:
                    self.given_back += 1
                    continue
                pg = table[s, b] = perm.pop()
                for p in range(b * page, min(n, (b + 1) * page)):
                    if not window or p >= lo or p < keep:
                        kpool[pg, :, p % page], vpool[pg, :, p % page] = self.k[s][p], self.v[s][p]
        self.table, self.pages = i32(table), total
        self.kpool, self.vpool = dev(kpool, dtype), dev(vpool, dtype)

    def want(self, scale):
        out = []
        for q, k, v, n, ql in zip(self.q, self.k, self.v, self.lengths, self.q_lens):
            ok = plain.seen(n, dict(size=self.window, keep_first=self.keep) if self.window else None)[n - ql:]
            G = self.H // self.KV
            s = torch.einsum("ihd,jhd->hij", q[n - ql:], k.repeat_interleave(G, 1)) * scale
            w = torch.softmax(s.masked_fill(~ok[None], -math.inf), -1)
            out.append(torch.einsum("hij,jhd->ihd", w, v.repeat_interleave(G, 1)).reshape(ql, -1))
        return torch.cat(out)

    def run(self, scale, **options):
        from mashbox_b200.parts.attention import PagedAttention
        core = PagedAttention(self.H, self.KV, self.DK, self.window, scale, vdim=self.DV, keep_first=self.keep)
        step = Step(self.dtype, self.lengths, self.q_lens, self.page, self.pages, options)
        core.prepare(step)
        step.inputs.upload()
        rows = torch.cat([q[n - ql:].reshape(ql, -1) for q, n, ql in zip(self.q, self.lengths, self.q_lens)])
        rows = dev(torch.cat([rows, torch.full((rows.shape[0], 8), 30.0, dtype=F64)], 1), self.dtype)
        out = torch.full((step.N, self.H * self.DV), float("nan"), device=DEV, dtype=TD[self.dtype])
        core.attend(step, rows, rows.stride(0), out, self.table, self.kpool, self.vpool)
        assert int(step.err.item()) == 0
        return out


# (kernel form, heads, kv heads, key width, value width, page, options): the plain kernel in both types; the general
# tensor-core kernel whole and cut along the keys; the TMA kernel (decode form alone, cut, in clusters; prompt form) and the
# tcgen05 kernel (prompt form), at both head sizes, with 1 to 16 query heads a kv head
FORMS = [("plain", 4, 2, 16, 24, 8, {}), ("plain", 3, 1, 12, 20, 5, {}), ("plain", 2, 2, 64, 64, 16, {}),
         ("general", 8, 2, 32, 64, 16, {}), ("general", 4, 1, 128, 48, 8, {}), ("general", 6, 2, 16, 16, 5, {}),
         ("general", 20, 1, 48, 64, 16, {}), ("general", 4, 2, 64, 64, 16, dict(attention_kernel="mma")),
         ("fast", 8, 2, 64, 64, 16, {}), ("fast", 4, 1, 128, 128, 32, {}), ("fast", 2, 2, 128, 128, 8, {}),
         ("fast", 16, 1, 64, 64, 64, {}), ("fast", 8, 2, 64, 64, 16, dict(attention_clusters=False)),
         ("fast", 8, 2, 128, 128, 16, dict(attention_target_blocks=1)), ("fast", 20, 1, 64, 64, 16, {}),
         ("fast", 4, 2, 64, 64, 16, dict(attention_prefill_kernel="mma"))]


def edges(window, keep, n):
    """(query, key) pairs of a sequence of n tokens whose last token asks, around everything the mask does"""
    q = n - 1
    ks = {q, q - window + 1, q - window, keep - 1, keep, 0, q - 1}
    return [(q, k) for k in sorted(ks) if 0 <= k <= q]


@pytest.mark.parametrize("form,H,KV,DK,DV,page,options", FORMS)
def test_windows_with_kept_tokens_on_their_edges(form, H, KV, DK, DV, page, options):
    scale = 1.0
    amount = 4.5 if DK <= 32 else 7.0           # the loud score stands well above sqrt(DK) times a unit normal
    for dtype in (DTYPES if form == "plain" else ("bfloat16",)):
        for window, keep, n in ((70, 9, 300), (33, 64, 700), (128, 130, 513), (1, 3, 90), (64, 64, 2 * page + 70), (200, 1, 190),
                                (50, 0, 260)):
            for qpos, kpos in edges(window, keep, n):
                seen = kpos < keep or qpos - kpos < window
                # the query decoded alone; at the end of a portion that starts inside a page; and among whole prompts
                for ql in (1, 37 if kpos % 2 else 2, n if n < 300 else 131):
                    if ql > n:
                        continue
                    case = WindowCase(dtype, H, KV, DK, DV, window, keep, [n, 40], [ql, 1], page, [(0, qpos, kpos)], seed=kpos,
                                      amount=amount)
                    got, want = case.run(scale, **options), case.want(scale)
                    what = f"{form} window {window} keep {keep} n {n} key {kpos} {'seen' if seen else 'not seen'}, {ql} queries"
                    kernel_close(got, want, dtype, what, 3e-2 if dtype == "bfloat16" else None)
                    loud = float(want[ql - 1].view(H, DV)[:, 0].abs().min())
                    assert (loud > 2.0) == seen, (what, loud)
    assert case.given_back > 0 or keep == 0 or n < 200


@pytest.mark.parametrize("form,H,KV,DK,DV,page,options", FORMS)
def test_kept_tokens_after_the_query_do_not_count(form, H, KV, DK, DV, page, options):
    """the first tokens of a sequence: a kept position that lies after the query is not seen"""
    for dtype in (DTYPES if form == "plain" else ("bfloat16",)):
        for ql, qpos, kpos in ((9, 4, 5), (30, 0, 1), (8, 6, 7)):
            case = WindowCase(dtype, H, KV, DK, DV, 4, 20, [ql, 3], [ql, 1], page, [(0, qpos, kpos)], seed=ql, amount=6.0)
            kernel_close(case.run(0.7, **options), case.want(0.7), dtype, f"{form} query {qpos} key {kpos}",
                         3e-2 if dtype == "bfloat16" else None)


@pytest.mark.parametrize("splits", [1, 2, 5, 16])
@pytest.mark.parametrize("H,KV,DK,DV", [(8, 2, 64, 64), (4, 1, 128, 128), (8, 2, 32, 64), (4, 4, 48, 16)])
def test_decode_form_cut_along_the_keys(H, KV, DK, DV, splits):
    """the cuts fall among the kept tiles, in the gap and in the window; sequences shorter than the window beside long ones"""
    for window, keep in ((300, 150), (640, 10), (100, 400)):
        case = WindowCase("bfloat16", H, KV, DK, DV, window, keep, [1000, 130, 17, 720], [1, 1, 1, 1], 16,
                          [(0, 999, keep - 1), (3, 719, 719 - window + 1)], seed=splits, amount=7.0)
        kernel_close(case.run(0.5, attention_splits=splits, attention_clusters=False), case.want(0.5), "bfloat16",
                     f"{splits} splits, window {window}, keep {keep}", 3e-2)


@pytest.mark.parametrize("H,KV,DK,DV,window,keep", [(8, 2, 64, 64, 96, 40), (2, 1, 128, 128, 700, 5), (8, 1, 64, 64, 31, 128),
                                                    (4, 2, 32, 64, 96, 40), (3, 3, 24, 40, 96, 40)])
def test_long_prompts_and_portions(H, KV, DK, DV, window, keep):
    """hundreds of queries per sequence in one step, from the start and far from it, beside a decoded one"""
    for lengths, q_lens in (([600, 333], [600, 1]), ([1500, 900], [700, 257]), ([1030], [300])):
        case = WindowCase("bfloat16", H, KV, DK, DV, window, keep, lengths, q_lens, 16, seed=window)
        kernel_close(case.run(DK ** -0.5), case.want(DK ** -0.5), "bfloat16", f"{lengths} {q_lens}", 3e-2)


# ------------------------------------------------------------------------------------------------ the other kernels alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,KV,DK,DV,RD,pairing,gain,pad", [
    (4, 2, 16, 24, 8, 0, 1.0, 0), (3, 1, 12, 20, 12, 0, 1.3, 4), (2, 2, 64, 32, 0, 0, 1.0, 8), (6, 3, 32, 8, 6, 0, 1.3, 8),
    (5, 1, 10, 6, 6, 0, 1.2, 3), (4, 2, 128, 128, 64, 0, 1.1, 0), (3, 1, 256, 64, 256, 0, 1.1, 0), (20, 4, 8, 16, 2, 0, 1.5, 0),
    (2, 1, 384, 16, 100, 0, 1.1, 8), (2, 2, 32, 16, 16, 1, 1.3, 0)])
def test_head_norms_after_the_rotation_and_mixed_values(dtype, H, KV, DK, DV, RD, pairing, gain, pad):
    from mashbox_b200 import ops
    gen = torch.Generator().manual_seed(DK + RD)
    for lengths in ([11, 4], [700, 40]):
        page = 4
        blocks = [-(-n // page) for n in lengths]
        perm = torch.randperm(sum(blocks) + 2, generator=gen).tolist()
        table = np.full((2, max(blocks)), -1, np.int32)
        for s, nb in enumerate(blocks):
            for b in range(nb):
                table[s, b] = perm.pop()
        pages = sum(blocks) + 2
        positions, tok_row = np.concatenate([np.arange(n) for n in lengths]), np.repeat([0, 1], lengths)
        N, C = len(positions), (H + KV) * DK + KV * DV + pad
        rows, first, lam = rnd(gen, N, C, dtype=dtype), rnd(gen, N, KV * DV, dtype=dtype), 0.3
        freqs = torch.tensor([100.0 ** (-2 * i / max(RD, 1)) for i in range(RD // 2)], dtype=torch.float32)
        a = torch.as_tensor(positions, dtype=F64)[:, None] * freqs.double()[None, :]
        c, s = (torch.cos(a) * gain)[:, None, :], (torch.sin(a) * gain)[:, None, :]

        def turned(x):
            if not RD:
                return x
            u, v = (x[..., :RD // 2], x[..., RD // 2:RD]) if pairing else (x[..., 0:RD:2], x[..., 1:RD:2])
            r = torch.cat([u * c - v * s, v * c + u * s], -1) if pairing else torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2)
            return torch.cat([r, x[..., RD:]], -1)
        q3, k3 = rows[:, :H * DK].view(N, H, DK), rows[:, H * DK:(H + KV) * DK].view(N, KV, DK)
        own = rows[:, (H + KV) * DK:(H + KV) * DK + KV * DV]
        for norm, mixing in (("after", "mix"), ("after", "keep"), (None, None), ("before", "mix")):
            r = dev(rows, dtype)
            kpool = torch.zeros(pages, KV, page, DK, device=DEV, dtype=TD[dtype])
            vpool = torch.zeros(pages, KV, page, DV, device=DEV, dtype=TD[dtype])
            kept = torch.full((N, KV * DV), float("nan"), device=DEV, dtype=TD[dtype])
            err = torch.zeros(1, dtype=torch.int32, device=DEV)
            ops.norm_rope_kv_write(r, None, None, 1e-6, dev(freqs) if RD else None, RD, pairing, gain, i32(positions), i32(tok_row),
                                   i32(table), kpool, vpool, H, KV, DK, DV, page, pages, err, norm=norm,
                                   v_keep=kept if mixing == "keep" else None,
                                   v_first=dev(first, dtype) if mixing == "mix" else None, lam=lam)
            assert int(err.item()) == 0
            heads = lambda x: {"after": lambda: plain.rms(turned(x), 1e-6), "before": lambda: turned(plain.rms(x, 1e-6)),
                               None: lambda: turned(x)}[norm]()
            bar = 1e-4 if dtype == "float32" else None      # position * frequency is one float32 product: 4e-5 at 700
            kernel_close(r[:, :H * DK], heads(q3).reshape(N, -1), dtype, f"q in place, norm {norm}", bar)
            kernel_close(r[:, (H + KV) * DK:], rows[:, (H + KV) * DK:], dtype, "what lies behind the keys is left alone", 1e-9)
            at = torch.as_tensor(table[tok_row, positions // page]).long().to(DEV), torch.as_tensor(positions % page).to(DEV)
            kernel_close(kpool[at[0], :, at[1]], heads(k3), dtype, f"keys in their pages, norm {norm}", bar)
            v = plain.mixed_values(own, first if mixing == "mix" else None, lam).view(N, KV, DV)
            kernel_close(vpool[at[0], :, at[1]], v, dtype, f"values in their pages, {mixing}", None if mixing == "mix" else 1e-9)
            if mixing == "keep":
                kernel_close(kept, own, dtype, "values kept for other layers", 1e-9)


@pytest.mark.parametrize("dtype", DTYPES)
def test_activated_projections_and_the_norm_over_all_heads(dtype):
    from mashbox_b200 import ops
    gen = torch.Generator().manual_seed(3)
    for H, dim, vdim, pad in ((3, 10, 6, 5), (2, 16, 24, 0), (4, 64, 32, 8), (32, 128, 128, 0)):
        N, C1, C2 = 9, H * dim, H * vdim
        rows = rnd(gen, N, 2 * C1 + 2 * C2 + pad, dtype=dtype, scale=3.0)
        rows[0, 0], rows[0, 1] = -60.0, 60.0
        q, k, v = torch.empty(N, C1, device=DEV), torch.empty(N, C1, device=DEV), torch.empty(N, C2, device=DEV)
        r = dev(rows, dtype)
        ops.silu_rows(r, q, k, v)
        for got, a, b in ((q, 0, C1), (k, C1, 2 * C1), (v, 2 * C1, 2 * C1 + C2)):
            kernel_close(got, plain.silu(rows[:, a:b]), "float32", f"silu of columns {a} to {b}")
        o, w = rnd(gen, N, C2), rnd(gen, C2) + 1
        o[1] *= 1e-4                            # a row whose mean square is below eps
        out = torch.empty(N, C2, device=DEV, dtype=TD[dtype])
        ops.gated_rms(dev(o), r[:, 2 * C1 + C2:], dev(w), out, 1, C2, 1e-5, silu=False)
        want = plain.rms(o, 1e-5, w) * torch.sigmoid(rows[:, 2 * C1 + C2:2 * C1 + 2 * C2])
        kernel_close(out, want, dtype, "normed over all heads, gated")
        kernel_close(out[1], want[1], dtype, "the quiet row")


@pytest.mark.parametrize("chunked", [False, True])
@pytest.mark.parametrize("H,dim,vdim", [(3, 16, 24), (1, 40, 20), (2, 64, 32), (2, 128, 128), (2, 6, 10)])
def test_recurrence_carries_its_state_across_cuts_and_slots(H, dim, vdim, chunked):
    """three sequences side by side in portions of their own sizes, in slots out of order; a decay of one, and one so quick
    that its powers leave float32"""
    from mashbox_b200 import ops
    gen = torch.Generator().manual_seed(dim)
    decay = torch.tensor([1.0, 0.3, 0.995][:H], dtype=torch.float32).double()
    lens, cuts, slots = [337, 5, 190], [[1, 2, 330, 4], [2, 1, 1, 1], [33, 1, 2, 154]], [2, 0, 3]
    state = torch.zeros(5, H * vdim * dim, device=DEV)
    qs, ks, vs = ([plain.silu(rnd(gen, n, H, w)).float().double() for n in lens] for w in (dim, dim, vdim))
    at, got = [0, 0, 0], [[], [], []]
    for step in range(4):
        q_len = [cuts[s][step] for s in range(3)]
        q_start = np.concatenate([[0], np.cumsum(q_len)[:-1]])
        cat = lambda xs: dev(torch.cat([xs[s][at[s]:at[s] + q_len[s]].reshape(q_len[s], -1) for s in range(3)]))
        o = torch.full((sum(q_len), H * vdim), float("nan"), device=DEV)
        ops.retention(cat(qs), cat(ks), cat(vs), dev(decay), o, state, (i32(q_start), i32(q_len), i32(slots)), H, dim, vdim,
                      chunked=chunked, segment=48 if chunked else None)
        for s in range(3):
            got[s].append(o[q_start[s]:q_start[s] + q_len[s]].cpu())
            at[s] += q_len[s]
    for s in range(3):
        S_ = torch.zeros(H, dim, vdim, dtype=F64)
        want = torch.zeros(lens[s], H, vdim, dtype=F64)
        for t in range(lens[s]):
            S_ = decay[:, None, None] * S_ + ks[s][t][:, :, None] * vs[s][t][:, None, :]
            want[t] = (S_ * qs[s][t][:, :, None]).sum(1)
        kernel_close(torch.cat(got[s]), want.view(lens[s], -1), "float32", f"sequence {s}")
        kernel_close(state[slots[s]].view(H, vdim, dim), S_.transpose(1, 2), "float32", f"state {s}")
    assert float(state[1].abs().max()) == 0.0 and float(state[4].abs().max()) == 0.0


@pytest.mark.parametrize("E,top", [(12, 2), (5, 5), (1, 1), (64, 6), (40, 33), (256, 8)])
def test_choice_by_biased_logits_weighted_by_the_softmax_over_the_chosen(E, top):
    from mashbox_b200 import ops
    gen = torch.Generator().manual_seed(E)
    N = 33
    z, b = rnd(gen, N, E + 3, scale=2.0), rnd(gen, E, scale=3.0)
    z[0] = 80.0                                     # far from zero: no overflow, the bias decides alone
    z[1, :E] = -b                                   # every biased logit zero: the first `top` experts, equal weights
    ids, wts = torch.empty(N, top, dtype=torch.int32, device=DEV), torch.empty(N, top, device=DEV)
    for bias in (b, None):
        ops.moe_select(dev(z), None, ids, wts, experts=E, score="softmax_chosen", bias=dev(bias) if bias is not None else None)
        zb = z[:, :E] + (bias if bias is not None else 0.0)
        want = plain.choose(zb, top)
        assert torch.equal(ids.cpu().long(), want)
        kernel_close(wts, torch.softmax(torch.gather(zb, 1, want), -1), "float32", "weights")


@pytest.mark.parametrize("dtype", DTYPES)
def test_squared_relu_alone_and_in_the_products_epilogue(dtype):
    from mashbox_b200 import ops
    gen = torch.Generator().manual_seed(1)
    for shape in ((6, 37), (5, 64)):
        z = rnd(gen, *shape, dtype=dtype, scale=3.0)
        out = torch.empty(*shape, device=DEV, dtype=TD[dtype])
        ops.relu2(dev(z, dtype), out)
        kernel_close(out, torch.clamp(z, min=0) ** 2, dtype, "max(z, 0)^2", 1e-2 if dtype == "bfloat16" else None)
    if dtype == "bfloat16":
        # one token (matrix-vector, short and long rows), a decode batch (weight-streaming), prompt portions (tcgen05)
        ops.configure({})
        for N, F, K in ((1, 264, 64), (1, 72, 8448), (1, 40, 2568), (2, 96, 1024), (5, 136, 4096), (16, 4104, 328), (9, 24, 72),
                        (128, 256, 64), (200, 264, 328), (515, 1032, 128)):
            a, w = rnd(gen, N, K, dtype=dtype), rnd(gen, F, K, dtype=dtype, scale=K ** -0.5)
            out = torch.full((N, F), float("nan"), device=DEV, dtype=torch.bfloat16)
            assert ops.fused_relu2_supports(N, F, K, torch.bfloat16)
            ops.linear_relu2(dev(a, dtype), dev(w, dtype), out)
            kernel_close(out, torch.clamp(a @ w.T, min=0) ** 2, dtype, f"product {N} x {F} x {K}")
        assert not ops.fused_relu2_supports(64, 256, 64, torch.bfloat16) and not ops.fused_relu2_supports(5, 100, 64, torch.bfloat16)


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
    from mashbox_b200.weights.random_init import write_model_folder
    from tests.plain.llama import read_model
    cfg, seed, page = S.CONFIGS[name]
    tmp = tmp_path_factory.mktemp("layers")
    (p,) = S.prompts_for(name, (75,))
    for n in range(1, len(cfg.layers) + 1):
        d = os.path.join(str(tmp), f"first{n}")
        write_model_folder(d, dataclasses.replace(cfg, layers=cfg.layers[:n]), seed, dtype=torch.float32, std=cfg.width ** -0.5,
                           norm_std=0.1, std_by_name=S.STD_BY_NAME)
        c, W = read_model(d)
        got = joined(replay(make_runner(d, "float32", 128, page_size=page), cut_steps("a", p, [len(p)])))
        S.assert_close(got, plain.forward(c, W, p).numpy(), "float32", f"{name}: the first {n} layers ({cfg.layers[n - 1].type} last)")


@pytest.mark.parametrize("seed", range(12))
def test_configurations_drawn_at_random(tmp_path_factory, seed):
    """2 to 5 layers of any kind in any order with sizes drawn from small sets: a whole prompt, then the same prompt in
    portions and single tokens"""
    import os
    from mashbox_b200.engine.replay import make_runner
    from mashbox_b200.weights.random_init import write_model_folder
    from tests.plain.llama import read_model
    cfg = S.random_config(seed)
    page = (4, 8, 16, 5)[seed % 4]
    tmp = tmp_path_factory.mktemp("r")
    p = np.random.default_rng(seed).integers(0, cfg.vocab, 75).tolist()
    for dtype in DTYPES:
        d = os.path.join(str(tmp), dtype)
        write_model_folder(d, cfg, 500 + seed, dtype=TD[dtype], std=cfg.width ** -0.5, norm_std=0.1, std_by_name=S.STD_BY_NAME)
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
                                     dict(plain_experts=True), dict(retention_scan_only=True)])
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
    for name in ("attention_tc5", "attention_tma", "attention_general_mma_32_64", "gemm_tc5"):
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


def test_a_window_frees_pages_for_a_pool_smaller_than_the_sequence(tmp_path_factory):
    """400 tokens decoded in a pool of 96: it holds them only because pages behind the window come back while those of the
    kept tokens stay"""
    import dataclasses
    import os
    from mashbox_b200.config.engine import EngineConfig
    from mashbox_b200.engine.loading import load_model
    from mashbox_b200.engine.runner import ModelRunner
    from mashbox_b200.weights.random_init import write_model_folder
    from tests.plain.llama import read_model
    cfg = dataclasses.replace(S.POB_P, layers=S.POB_P.layers[:3])
    d = os.path.join(str(tmp_path_factory.mktemp("w")), "m")
    write_model_folder(d, cfg, 9, dtype=torch.float32, std=cfg.width ** -0.5, norm_std=0.1, std_by_name=S.STD_BY_NAME)
    runner = ModelRunner(load_model(d, dtype="float32", device=DEV),
                         EngineConfig(dtype="float32", page_size=8, max_tokens=96, max_requests=2, max_tokens_per_step=64,
                                      max_context=448, chunk=64, device=DEV))
    p = np.random.default_rng(1).integers(0, cfg.vocab, 400).tolist()
    got = joined(replay(runner, cut_steps("a", p, [20, 30] + [1] * 350)))
    c, W = read_model(d)
    S.assert_close(got, plain.forward(c, W, p).numpy(), "float32", "400 tokens in a pool of 96")
    runner.cache.check()


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
