"""The attention mixer: grouped-query attention over the paged cache.

q = h Wq^T (+bq), k, v likewise from one fused product (the three weights are concatenated at load); q and k are
rotated, k and v written to the layer's pages, then every query attends to the cached keys of its own sequence up to
its own position -- the step's own tokens are read from the cache like the older ones, so a portion of a prompt, a
single decoded token and a whole prompt all take the same path.  Query head h reads kv head h // (H / KV); scores are
scaled by head_dim^-0.5 (or `scale`), softmax and the weighted sum are float32; `window` w limits a query to the last w
positions.  Formulas: src/mashbox/gguf/archs/dense.py:339-348, src/mashbox/runtime/attention.py:54-93.

Kernels: the float32 path, and head sizes the tensor-core kernel does not take, use the plain paged kernel (one warp
per token and head, fixed order).  The bf16 path packs the G query heads of a kv head into the rows of an MMA tile and
runs the flash kernel: row tiles of 64 for prompt portions, tiles of 16 with the keys split over warps (and over
blocks, merged by a second kernel) for decode tokens.  `prepare` builds that work list on the host.
"""
import numpy as np

from ..cache.manager import CacheNeed
from ..errors import ConfigError
from ..weights.loader import Want
from .base import PartSpec, make, register

DECODE_ROWS, PREFILL_ROWS, KEY_TILE = 16, 64, 64


def many_splits(blocks, work, slots, head_dim, most=4):
    """Into how many splits (1 to `most`) to cut each of `blocks` decode-form tiles of the TMA attention kernel, `work`
    key tiles in all, when there are more of them than half the `slots` the device has for such blocks.  The model: the
    blocks run in rounds of `slots`; a round of n blocks of w key tiles takes the longer of what the memory needs for
    them (n w tiles at 6.5 TB/s, but never less than `enough` blocks' worth: that many blocks, with three or four
    stages of 64 keys in flight each, about 19 MB, keep the memory busy) and what one block needs for itself (7 us to
    start, meet and finish, half a microsecond a tile); splits cost 4 us and 0.15 us each on top (their partial
    results meet through global memory).  The fewest splits within 1 % of the best."""
    tile_bytes = 2 * 64 * head_dim * 2
    enough = max(1, int(19.2e6 // ((3 if head_dim > 64 else 4) * tile_bytes)))
    tile_us = tile_bytes / 6.5e6                                 # a tile's share of the memory's time
    costs = []
    for ns in range(1, max(1, most) + 1):
        n, w = blocks * ns, work / (blocks * ns)
        full, rest = divmod(n, slots)
        alone = 7.0 + 0.5 * w                                     # a block by itself
        t = full * max(slots * w * tile_us, alone)
        if rest:
            t += max(max(rest, enough) * w * tile_us, alone)
        costs.append(t + (4.0 + 0.15 * ns if ns > 1 else 0.0))
    best = min(costs)
    return 1 + next(i for i, c in enumerate(costs) if c <= 1.01 * best)


class PagedAttention:
    """Attention of a step's queries over rows kept per position in pages: the work lists (`prepare`, on the host) and
    the choice of kernel (`attend`).  `heads` query heads read `kv_heads` rows of `head_dim` values per position;
    whoever keeps other things per position than keys and values of its own (one latent vector that is key and value at
    once, say) hands its pools in."""

    def __init__(self, heads, kv_heads, head_dim, window=None, scale=None, vdim=None, softcap=None, sinks=False,
                 gated=False, keep_first=0):
        """vdim: the width of a value when it is not the key's (the result is heads * vdim wide); softcap: scores become
        softcap tanh(s / softcap); sinks: attend() is handed one number per query head that joins the softmax's
        denominator without a value; gated: attend() is handed a gate per token and query head (the head's result
        times its sigmoid).  Other value widths, a cap, gates, or pools whose rows are wider than what is read of them,
        make the attention *general*: it runs on the kernels that take all of that.  keep_first: behind the window the
        first `keep_first` positions stay visible.  That and sinks the TMA and tcgen05 kernels take, and the general ones;
        where a step would run another kernel the attention is general too (`is_general`)."""
        self.H, self.KV, self.HD = int(heads), int(kv_heads), int(head_dim)
        if self.H % self.KV:
            raise ConfigError(f"{heads} heads do not divide into {kv_heads} kv heads")
        self.window = int(window) if window else None
        self.scale = float(scale) if scale else self.HD ** -0.5
        self.VD = int(vdim) if vdim else self.HD
        self.softcap = float(softcap) if softcap else None
        self.keep = int(keep_first) if self.window else 0       # without a window every position is visible anyway
        self.sunk = bool(sinks)
        self.general = self.VD != self.HD or self.softcap is not None or bool(gated)

    # ------------------------------------------------------------------------------------------ planning
    def is_general(self, ctx):
        """whether this step runs the general kernels"""
        import torch
        if self.general or not (self.keep or self.sunk):
            return self.general
        page = ctx.cache.page_size
        return not (ctx.dtype == torch.bfloat16 and ctx.options.get("attention_kernel", "tma") == "tma"
                    and ctx.ops.attention_tma_supports(self.HD, page) and not ctx.options.get("plain_attention", False))

    def uses_mma(self, ctx):
        import torch
        if self.is_general(ctx):        # keys and values of their own widths, caps, sinks, gates: the general tensor-core form
            return (ctx.dtype == torch.bfloat16 and ctx.ops.attention_general_mma_supports(self.HD, self.VD)
                    and not ctx.options.get("plain_attention", False))
        return ctx.dtype == torch.bfloat16 and ctx.ops.attention_mma_supports(self.HD) and not ctx.options.get(
            "plain_attention", False)

    def uses_tc5(self, ctx):
        """prompt-form tiles go to the tcgen05 kernel (its own number of packed rows per block, no splits) when it takes
        the sizes"""
        return (not self.is_general(ctx) and ctx.options.get("attention_prefill_kernel", "tc5") == "tc5"
                and ctx.ops.attention_tc5_supports(self.HD, ctx.cache.page_size))

    def _tma(self, ctx):
        """decode-form sequences go to the TMA kernel (whose splits may meet in a cluster)"""
        return (not self.is_general(ctx) and ctx.options.get("attention_kernel", "tma") == "tma"
                and ctx.ops.attention_tma_supports(self.HD, ctx.cache.page_size))

    def plan_key(self):
        # everything the work list depends on: the head size decides the kernel and its rows per tile
        return ("attention", self.H // self.KV, self.KV, self.HD, self.window, self.keep, self.general, self.sunk)

    def prepare(self, ctx):
        """Work list of the flash kernel for this step: (sequence, row tile, split, splits) per block, decode-form
        sequences (at most 16 packed rows) and prompt-form ones apart; sequences cut into splits get a place in the
        partial buffers."""
        if not self.uses_mma(ctx):
            return
        key = self.plan_key()
        if key in ctx.memo:
            return
        G, KV = self.H // self.KV, self.KV
        target = int(ctx.options.get("attention_target_blocks", 296))
        max_splits = int(ctx.options.get("attention_max_splits", 32))
        S = ctx.S
        tc5 = self.uses_tc5(ctx)
        pre_rows = ctx.ops.attention_tc5_rows() if tc5 else PREFILL_ROWS
        decode_form = [ctx.q_len[s] * G <= DECODE_ROWS for s in range(S)]
        tiles = [1 if decode_form[s] else -(-ctx.q_len[s] * G // pre_rows) for s in range(S)]
        # the two forms are two launches: each is cut into splits by its own number of blocks
        base = {f: max(1, sum(t for t, d in zip(tiles, decode_form) if d == f) * KV) for f in (True, False)}
        dec, pre, mid, part_base, part_tok = [], [], [], [-1] * S, []
        # More query heads per kv head than a decode tile has rows (every head reads one row per position, say): a single
        # token is already a prompt-form tile, which the tcgen05 kernel does not cut along the keys.  Such stretches of
        # at most DECODE_ROWS tokens go to the TMA/mma prompt form with splits, in a list of their own.
        wide = tc5 and G > DECODE_ROWS

        def key_tiles(s):
            hi = ctx.pos0[s] + ctx.q_len[s]
            lo = max(0, ctx.pos0[s] - self.window + 1) if self.window else 0
            front = min(-(-self.keep // KEY_TILE), lo // KEY_TILE)          # tiles of kept positions before the window's
            return front + -(-(hi - lo // KEY_TILE * KEY_TILE) // KEY_TILE)

        # Decode-form sequences on the TMA kernel: when they can all be cut into the same number of splits (set by the
        # longest of them; a shorter one leaves some of its splits empty) the blocks of a sequence and kv head are
        # launched as one thread-block cluster and their results meet in shared memory.
        cluster = 0
        page = ctx.cache.page_size
        if (any(decode_form) and base[True] < target and self._tma(ctx) and ctx.options.get("attention_clusters", True)):
            raw = min(max_splits, -(-target // base[True]), max(key_tiles(s) for s in range(S) if decode_form[s]) // 2)
            want = 1 << (max(1, raw).bit_length() - 1)
            # only when the cluster holds all the splits the launch wants anyway: at one or two sequences (32 and 16
            # splits) more, smaller blocks that meet through global memory are faster than clusters of 8
            most = ctx.ops.attention_tma_max_cluster(self.HD)
            longest = max(key_tiles(s) for s in range(S) if decode_form[s])
            if want > most and longest <= 6 * most:
                # ... unless the sequences are short: up to six key tiles per block, the cheaper meeting of a cluster
                # outweighs the longer blocks (one sequence of 2,048 keys: 9.2 us in a cluster of 8, 10.4 as 16 splits)
                raw = want = most
            if 2 <= want <= most:
                # the largest cluster, of any size, that leaves all clusters of the launch on the device at once with
                # room to spare: the kernel before this one still holds SMs when the first clusters are placed
                room = float(ctx.options.get("attention_cluster_room", 0.91))
                fits = [c for c in range(2, min(raw, most) + 1)
                        if base[True] <= room * ctx.ops.attention_tma_active_clusters(self.HD, c)]
                cluster = max(fits) if fits else 0
        if ctx.options.get("attention_cluster_size") is not None and any(decode_form):
            cluster = int(ctx.options["attention_cluster_size"])
        # More decode-form tiles than half the blocks the device holds: cutting them to fill `target` blocks would mean
        # one or two splits, and what then decides is the last, partly filled round of blocks: too few blocks to keep
        # the memory busy (8 kv heads, 8,192 keys: 20 sequences as 320 blocks take 8.2 ms a step, as 480 blocks 6.9; 40
        # as 320 blocks 12.4, as 1,280 10.6).  many_splits() picks the number of splits by a model of that.
        crowd = 0
        if (not cluster and any(decode_form) and self._tma(ctx) and ctx.options.get("attention_splits") is None):
            slots = 2 * ctx.ops.attention_tma_active_clusters(self.HD, 2)
            if slots and 2 * base[True] > slots:
                work = sum(key_tiles(s) for s in range(S) if decode_form[s]) * KV
                crowd = many_splits(base[True], work, slots, self.HD, min(4, max_splits))
        for s in range(S):
            kv_tiles = key_tiles(s)
            ns = 1
            if cluster and decode_form[s]:
                for sp in range(cluster):
                    dec.append((0, s, 0, sp, cluster))
                continue
            short = wide and not decode_form[s] and ctx.q_len[s] <= DECODE_ROWS
            if ctx.q_len[s] <= DECODE_ROWS and base[decode_form[s]] < target and (decode_form[s] or not tc5 or short):
                ns = max(1, min(max_splits, -(-target // base[decode_form[s]]), kv_tiles // 2))
                ns = 1 << (ns.bit_length() - 1)                    # a power of two: few distinct work-list shapes
            if decode_form[s] and (crowd or ctx.options.get("attention_splits") is not None):
                ns = max(1, min(crowd or int(ctx.options["attention_splits"]), kv_tiles // 2))
            if ns > 1:
                part_base[s] = len(part_tok) // 2
                for t in range(ctx.q_len[s]):
                    part_tok += [ctx.q_start[s] + t, ns]
            dst = dec if decode_form[s] else (mid if short else pre)
            rows = PREFILL_ROWS if short else pre_rows
            for m in range(-(-ctx.q_len[s] * G // rows) if short else tiles[s]):
                for sp in range(ns):
                    dst.append((-(ctx.pos0[s] + (m + 1) * rows // G), s, m, sp, ns))
        pre.sort()                                                  # the tiles with the most keys first
        name = "attn%d_" % len([k for k in ctx.memo if k[0] == "attention"])
        flat = lambda items: np.asarray([i[1:] for i in items], np.int32).reshape(-1)
        ctx.inputs.add(name + "dec", flat(dec))
        ctx.inputs.add(name + "pre", flat(pre))
        ctx.inputs.add(name + "mid", flat(mid))
        ctx.inputs.add(name + "part_base", np.asarray(part_base, np.int32))
        ctx.inputs.add(name + "part_tok", np.asarray(part_tok, np.int32))
        ctx.memo[key] = dict(name=name, n_dec=len(dec), n_pre=len(pre), n_mid=len(mid), n_part=len(part_tok) // 2,
                             max_splits=max_splits, tc5=tc5, cluster=cluster)

    # ------------------------------------------------------------------------------------------ kernels
    def attend(self, ctx, qkv, width, out, table, kpool, vpool, rope=None, sinks=None, gate=None):
        """The step's queries -- rows of qkv, `width` values apart, head h at column h * head_dim -- attend to the rows
        of their sequences' pages; out (N, heads * vdim).  rope = (bias, freqs, rotary dims, pairing): the decode
        form of the TMA kernel rotates and stores the step's own keys and values from qkv itself.  sinks (heads,)
        float32 and gate (a view (N, heads) of the gates' logits): see the constructor."""
        import torch
        ops = ctx.ops
        H, KV, HD = self.H, self.KV, self.HD
        page, pages = ctx.cache.page_size, ctx.cache.pool_pages
        if self.is_general(ctx):
            self.attend_general(ctx, qkv, width, out, table, kpool, vpool, sinks, gate)
            return
        if self.uses_mma(ctx):
            plan = ctx.memo[self.plan_key()]
            nm = plan["name"]
            n_part, ms = plan["n_part"], plan["max_splits"]
            part_o = part_ml = None
            if n_part:
                part_o = ctx.ws.get("attn_part_o", n_part * H * ms, (HD,), torch.float32, reserve=0)
                part_ml = ctx.ws.get("attn_part_ml", n_part * H * ms, (2,), torch.float32, reserve=0)
            kind = ctx.options.get("attention_kernel", "tma")
            tma = kind == "tma" and ops.attention_tma_supports(HD, page)
            flash = ops.attention_tma if tma else ops.attention_mma
            # the TMA kernel merges the splits itself (the last block of a group does it); the other needs the merge kernel
            fused = (tma and n_part > 0 and ctx.options.get("attention_fused_merge", True)
                     and ops.attention_tma_merges(max(plan["n_pre"], plan["n_mid"], plan["n_dec"]), KV))
            extra = dict(merge=True) if fused else {}
            if self.keep:
                extra["keep"] = self.keep
            if self.sunk:
                extra["sinks"] = sinks
            if rope is not None:
                extra["rope"] = rope
            if plan["tc5"] and plan["n_pre"]:
                ops.attention_tc5(qkv, width, out, kpool, vpool, ctx.dev(nm + "pre"), plan["n_pre"], ctx.dev("q_start"),
                                  ctx.dev("q_len"), ctx.dev("pos0"), ctx.dev("seq_row"), table, H, KV, HD, page, pages,
                                  self.window, self.scale, ctx.err, keep=self.keep, sinks=sinks if self.sunk else None)
            for form, n_items, decode in ((nm + "pre", 0 if plan["tc5"] else plan["n_pre"], False),
                                          (nm + "mid", plan["n_mid"], False), (nm + "dec", plan["n_dec"], True)):
                if n_items and decode and plan["cluster"]:
                    ops.attention_tma(qkv, width, out, kpool, vpool, ctx.dev(form), n_items, True, ctx.dev("q_start"),
                                      ctx.dev("q_len"), ctx.dev("pos0"), None, ctx.dev("seq_row"), table, None, None, 1,
                                      H, KV, HD, page, pages, self.window, self.scale, ctx.err,
                                      rope=extra.get("rope"), cluster=plan["cluster"], keep=self.keep,
                                      sinks=extra.get("sinks"))
                elif n_items:
                    flash(qkv, width, out, kpool, vpool, ctx.dev(form), n_items, decode, ctx.dev("q_start"),
                          ctx.dev("q_len"), ctx.dev("pos0"), ctx.dev(nm + "part_base"), ctx.dev("seq_row"),
                          table, part_o, part_ml, ms, H, KV, HD, page, pages, self.window, self.scale, ctx.err, **extra)
            if n_part and not fused:
                ops.attention_merge(part_o, part_ml, ctx.dev(nm + "part_tok"), n_part, out, H, HD, ms)
        else:
            ops.attention_simple(qkv, width, out, ctx.dev("positions"), ctx.dev("tok_row"), table, kpool, vpool, H, KV,
                                 HD, page, pages, self.window, self.scale, ctx.err)


    def attend_general(self, ctx, q, width, out, table, kpool, vpool, sinks, gate):
        import torch
        ops, H, KV = ctx.ops, self.H, self.KV
        page, pages = ctx.cache.page_size, ctx.cache.pool_pages
        if self.uses_mma(ctx) and width % 8 == 0 and kpool.shape[-1] % 8 == 0 and vpool.shape[-1] % 8 == 0:
            plan = ctx.memo[self.plan_key()]
            nm, n_part, ms = plan["name"], plan["n_part"], plan["max_splits"]
            part_o = part_ml = None
            if n_part:
                part_o = ctx.ws.get("attn_part_o", n_part * H * ms, (self.VD,), torch.float32, reserve=0)
                part_ml = ctx.ws.get("attn_part_ml", n_part * H * ms, (2,), torch.float32, reserve=0)
            for form, n_items, decode in ((nm + "pre", plan["n_pre"], False), (nm + "mid", plan["n_mid"], False),
                                          (nm + "dec", plan["n_dec"], True)):
                if n_items:
                    ops.attention_general_mma(q, width, out, kpool, vpool, ctx.dev(form), n_items, decode,
                                              ctx.dev("q_start"), ctx.dev("q_len"), ctx.dev("pos0"),
                                              ctx.dev(nm + "part_base"), ctx.dev("seq_row"), table, part_o, part_ml, ms, H,
                                              KV, self.HD, self.VD, page, pages, self.window, self.scale, ctx.err,
                                              self.softcap, sinks, gate, keep=self.keep)
            if n_part:
                ops.attention_general_merge(part_o, part_ml, ctx.dev(nm + "part_tok"), n_part, out, H, self.HD, self.VD, ms,
                                            sinks, gate)
            return
        ctx.ops.attention_general(q, width, out, ctx.dev("positions"), ctx.dev("tok_row"), table, kpool, vpool, self.H,
                                  self.KV, self.HD, self.VD, ctx.cache.page_size, ctx.cache.pool_pages, self.window,
                                  self.scale, ctx.err, self.softcap, sinks, gate, keep=self.keep)


class Attention(PagedAttention):
    @property
    def graph_safe(self):
        """forward() depends on the batch only through the lengths of the step's arrays; so must the position encoding"""
        return self.position is None or bool(getattr(self.position, "graph_safe", False))

    def __init__(self, hidden, heads, kv_heads, head_dim, bias=False, position=None, window=None, scale=None,
                 prefix="", names=None):
        super().__init__(heads, kv_heads, head_dim, window, scale)
        self.D, self.bias = int(hidden), bool(bias)
        self.prefix = prefix
        n = dict(q="attn_q", k="attn_k", v="attn_v", o="attn_output")
        n.update(names or {})
        self.names = {k: prefix + v for k, v in n.items()}
        self.position = make("position", position) if isinstance(position, PartSpec) else position
        self.wqkv = self.bqkv = self.wo = self.bo = None

    # ------------------------------------------------------------------------------------------ weights
    def wants(self):
        H, KV, HD, D = self.H, self.KV, self.HD, self.D
        shapes = dict(q=(H * HD, D), k=(KV * HD, D), v=(KV * HD, D), o=(D, H * HD))
        w = [Want(self.names[r] + ".weight", shapes[r], "matrix") for r in "qkvo"]
        if self.bias:
            w += [Want(self.names[r] + ".bias", (shapes[r][0],), "vector") for r in "qkvo"]
        return w + (self.position.wants() if self.position is not None else [])

    def bind(self, tensors, env):
        import torch
        t = lambda r, s: tensors[self.names[r] + s]
        self.wqkv = torch.cat([t("q", ".weight"), t("k", ".weight"), t("v", ".weight")], 0).contiguous()
        self.wo = t("o", ".weight")
        if self.bias:
            self.bqkv = torch.cat([t("q", ".bias"), t("k", ".bias"), t("v", ".bias")], 0).contiguous()
            self.bo = t("o", ".bias")
        if self.position is not None:
            self.position.bind(tensors, env)

    def cache_need(self):
        return CacheNeed.keys_and_values(self.KV, self.HD, self.window)

    def state_need(self):
        return None

    # ------------------------------------------------------------------------------------------ forward
    fuses_small = True      # forward() takes normed= and residual= (see PreNormBlock)

    def forward(self, ctx, h, run, normed=None, residual=None):
        import torch
        ops, N = ctx.ops, ctx.N
        H, KV, HD = self.H, self.KV, self.HD
        width = (H + 2 * KV) * HD
        qkv = ctx.ws.get("qkv", N, (width,), ctx.dtype)
        group, kpool, vpool = ctx.cache.layer_cache(run.cache)
        table = group.device_table
        page, pages = ctx.cache.page_size, ctx.cache.pool_pages
        rot = self.position.rotation() if self.position is not None else (None, HD, 0)
        # A step in which every sequence brings one token (N == S: that follows from the lengths of the step's arrays):
        # the decode form of the TMA attention kernel rotates, stores and attends in one launch.
        folded = (rot is not None and run.write and N == ctx.S and self.uses_mma(ctx)
                  and ctx.options.get("attention_kernel", "tma") == "tma" and ops.attention_tma_supports(HD, page)
                  and ops.attention_tma_folds_rotation(H // KV) and ctx.options.get("attention_folds_rotation", True)
                  and not (normed is not None and ops.small_qkv_supports(N, self.D)
                           and ctx.options.get("qkv_rope_epilogue", False)))
        if (normed is not None and rot is not None and ops.small_qkv_supports(N, self.D)
                and (ctx.options.get("qkv_rope_epilogue", False) or not folded)):
            # a step of very few tokens: norm, product, rotation and the cache write in one kernel -- where the attention
            # kernel cannot take the rotation in (when it can, it also fetches the cached keys before this product has
            # ended: a one-token step of the 8B shape 3.31 against 3.35 ms)
            x, norm = normed
            w, eps = norm.fusable()
            freqs, rd, pairing = rot
            ops.linear_small_normed_qkv(x, w, eps, self.wqkv, qkv, self.bqkv, ctx.dev("positions"), ctx.dev("tok_row"),
                                        table, kpool if run.write else None, vpool if run.write else None, freqs, H, KV,
                                        HD, rd, pairing, page, pages, ctx.err)
        else:
            if normed is not None:
                x, norm = normed
                w, eps = norm.fusable()
                ops.linear_small_normed(x, w, eps, self.wqkv, qkv, held=ctx.take_held(x, norm))
            else:
                ops.linear(h, self.wqkv, out=qkv)
            freqs, rd, pairing = (None, HD, 0)
            if rot is None:
                if self.bias:
                    raise ConfigError("a position encoding with its own kernel cannot be combined with q/k/v biases")
                self.position.apply(ctx, qkv, H, KV, HD)
            else:
                freqs, rd, pairing = rot
            if not folded:
                ops.rope_kv_write(qkv, self.bqkv, ctx.dev("positions"), ctx.dev("tok_row"), table,
                                  kpool if run.write else None, vpool if run.write else None, freqs, H, KV, HD, rd,
                                  pairing, page, pages, ctx.err)
        out = ctx.ws.get("attn_out", N, (H * HD,), ctx.dtype)
        self.attend(ctx, qkv, width, out, table, kpool, vpool,
                    rope=(self.bqkv, freqs, rd, pairing) if folded else None)
        if residual is not None:
            ctx.add_into_stream(out, self.wo, residual, self.bo)
            return None
        y = ctx.ws.get("delta", N, (self.D,), ctx.dtype)
        ops.linear(out, self.wo, out=y)
        return y, self.bo


register("mixer", "attention", Attention)


class GatedAttention(PagedAttention):
    """Grouped-query attention whose keys and values may differ in width, with, each optional: an RMS norm of every q
    and k head before the rotation (`qk_norm` True: weights `<q>.norm` and `<k>.norm` of head_dim values, shared by the
    heads) or after it (`qk_norm` "after": no weights), a sliding window (`window`) behind which the first `keep_first`
    positions stay visible, values mixed with those of another layer of the same step (`value_mix`: "keep" leaves this
    layer's values for the others, "mix" caches (1 - lam) v + lam v_kept, lam stored as `<vmix>`), a rotation of the first dims of a head (`position`, any rope spec), capped scores (`softcap`), a sink in
    the softmax's denominator (`sink`: "unit" -- a sink of score zero, so one is added to the denominator -- or the name
    of a tensor with one number per query head, or None) and a gate per token and query head (`gate`: head h's result
    times sigmoid(Wg h)_h, Wg stored as `<g>`).  `bias`: q, k and v have biases (the tensor's name with `.b`), added before anything
    else happens to them.

        q = Wq h (heads x dim), k = Wk h (kv_heads x dim), v = Wv h (kv_heads x vdim)
        q, k <- rms(.) n per head;  rotated;  s = scale q . k, s <- cap tanh(s / cap)
        p_j = e^s_j / (e^sink + sum_j e^s_j);  out = Wo concat_h(sigmoid(g_h) sum_j p_j v_j)

    One product makes q, k, v and the gates' logits; one kernel adds the biases, norms, rotates and writes k and v to
    their pages (without norms and with equal widths a decode step leaves that to the attention kernel); the attention
    kernel takes cap, sink and gate in.  Norms, angles, scores and the softmax are float32."""

    def __init__(self, hidden, heads, kv_heads, head_dim, vdim=None, scale=None, softcap=None, qk_norm=False, eps=1e-6,
                 sink=None, gate=False, position=None, window=None, keep_first=0, value_mix=None, bias=False, prefix="", names=None):
        super().__init__(heads, kv_heads, head_dim, window, scale, vdim=vdim, softcap=softcap, sinks=sink is not None,
                         gated=gate, keep_first=keep_first)
        self.D, self.eps, self.sink, self.gate = int(hidden), float(eps), sink, bool(gate)
        self.has_bias, self.bias = bool(bias), None
        if qk_norm not in (True, False, None, "after") or value_mix not in (None, "keep", "mix"):
            raise ConfigError(f"this attention has no q/k norm {qk_norm!r} or value mixing {value_mix!r}")
        self.norm_at = "after" if qk_norm == "after" else ("before" if qk_norm else None)
        self.value_mix, self.lam = value_mix, 0.0
        n = dict(q="q", k="k", v="v", g="g", o="o", q_norm="q.norm", k_norm="k.norm", vmix="vmix")
        n.update(names or {})
        self.n = {k: prefix + v for k, v in n.items()}
        self.sink_name = prefix + sink if sink not in (None, "unit") else None
        self.position = make("position", position) if isinstance(position, PartSpec) else position
        self.w_in = self.wo = self.qw = self.kw = self.sinks = None

    @property
    def graph_safe(self):
        return self.position is None or bool(getattr(self.position, "graph_safe", False))

    def wants(self):
        H, KV, HD, VD, D = self.H, self.KV, self.HD, self.VD, self.D
        out = [Want(self.n["q"], (H * HD, D), "matrix"), Want(self.n["k"], (KV * HD, D), "matrix"),
               Want(self.n["v"], (KV * VD, D), "matrix"), Want(self.n["o"], (D, H * VD), "matrix")]
        if self.has_bias:
            out += [Want(self.n[r] + ".b", (n,), "vector") for r, n in (("q", H * HD), ("k", KV * HD), ("v", KV * VD))]
        if self.value_mix == "mix":
            out.append(Want(self.n["vmix"], (), "vector"))
        if self.norm_at == "before":
            out += [Want(self.n["q_norm"], (HD,), "vector"), Want(self.n["k_norm"], (HD,), "vector")]
        if self.gate:
            out.append(Want(self.n["g"], (H, D), "matrix"))
        if self.sink_name:
            out.append(Want(self.sink_name, (H,), "vector"))
        return out + (self.position.wants() if self.position is not None else [])

    def bind(self, tensors, env):
        import torch
        t = lambda k: tensors[self.n[k]]
        parts = [t("q"), t("k"), t("v")] + ([t("g")] if self.gate else [])
        rows = sum(p.shape[0] for p in parts)
        if rows % 8:        # rows of the product start on 16-byte boundaries in bfloat16: zero rows behind the gates
            parts.append(torch.zeros((8 - rows % 8, self.D), dtype=parts[0].dtype, device=parts[0].device))
        self.w_in = torch.cat(parts, 0).contiguous()
        if self.has_bias:
            self.bias = torch.cat([tensors[self.n[r] + ".b"] for r in "qkv"], 0).contiguous()
        self.wo = t("o")
        self.qw, self.kw = (t("q_norm"), t("k_norm")) if self.norm_at == "before" else (None, None)
        if self.value_mix == "mix":
            self.lam = float(t("vmix").float().cpu())
        if self.sink == "unit":
            self.sinks = torch.zeros(self.H, dtype=torch.float32, device=env.device)
        elif self.sink_name:
            self.sinks = tensors[self.sink_name]
        if self.position is not None:
            self.position.bind(tensors, env)
            if self.position.rotation() is None:
                raise ConfigError("this attention rotates in its own kernel; its position part must hand it frequencies")

    def cache_need(self):
        return CacheNeed("window" if self.window else "full", ((self.KV, self.HD), (self.KV, self.VD)), self.window,
                         self.keep)

    def state_need(self):
        return None

    def forward(self, ctx, h, run, out="delta"):
        ops, N = ctx.ops, ctx.N
        H, KV, HD, VD = self.H, self.KV, self.HD, self.VD
        rows = ctx.ws.get("gattn_in", N, (self.w_in.shape[0],), ctx.dtype)
        ops.linear(h, self.w_in, out=rows)
        group, kpool, vpool = ctx.cache.layer_cache(run.cache)
        table, page, pages = group.device_table, ctx.cache.page_size, ctx.cache.pool_pages
        freqs, rd, pairing, gain = None, 0, 0, 1.0
        if self.position is not None:
            freqs, rd, pairing = self.position.rotation()
            gain = getattr(self.position, "gain", 1.0)
        plain = self.norm_at is None and self.value_mix is None and HD == VD and not self.gate and gain == 1.0
        # A step in which every sequence brings one token (N == S: that follows from the lengths of the step's arrays):
        # the decode form of the TMA attention kernel adds the biases, rotates, stores and attends in one launch.
        folded = (plain and run.write and N == ctx.S and not self.is_general(ctx) and self.uses_mma(ctx)
                  and ctx.options.get("attention_kernel", "tma") == "tma" and ops.attention_tma_supports(HD, page)
                  and ops.attention_tma_folds_rotation(H // KV) and ctx.options.get("attention_folds_rotation", True))
        if folded:
            pass
        elif plain and rows.shape[1] == (H + 2 * KV) * HD and freqs is not None:
            ops.rope_kv_write(rows, self.bias, ctx.dev("positions"), ctx.dev("tok_row"), table, kpool if run.write else None,
                              vpool if run.write else None, freqs, H, KV, HD, rd, pairing, page, pages, ctx.err)
        else:
            # the layer whose values others mix in runs first in the step and leaves them in a buffer of the step's tokens
            kept = ctx.ws.get("values_kept", N, (KV * VD,), ctx.dtype) if self.value_mix else None
            ops.norm_rope_kv_write(rows, self.qw, self.kw, self.eps, freqs, rd, pairing, gain, ctx.dev("positions"),
                                   ctx.dev("tok_row"), table, kpool if run.write else None, vpool if run.write else None, H,
                                   KV, HD, VD, page, pages, ctx.err, norm=self.norm_at,
                                   v_keep=kept if self.value_mix == "keep" else None,
                                   v_first=kept if self.value_mix == "mix" else None, lam=self.lam, bias=self.bias)
        o = ctx.ws.get("gattn_out", N, (H * VD,), ctx.dtype)
        off = (H + KV) * HD + KV * VD
        gate = rows[:, off:off + H] if self.gate else None
        self.attend(ctx, rows, rows.stride(0), o, table, kpool, vpool, sinks=self.sinks, gate=gate,
                    rope=(self.bias, freqs, rd, pairing) if folded else None)
        y = ctx.ws.get(out, N, (self.D,), ctx.dtype)
        ops.linear(o, self.wo, out=y)
        return y, None


register("mixer", "gated_attention", GatedAttention)
