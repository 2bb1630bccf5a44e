"""RWKV-style time mixing: a recurrent layer whose projections read a mix of a token's input and that of the token before,
with a matrix state per head that decays per key channel and an extra weight for the current token.

    h' = the input of the token before (zeros before the first);  mix_s = h + (h' - h) mu_s   for s in r, k, v, g, w
    r, k, v = W_s mix_s   (heads x dim);   d = exp(-exp(W2 tanh(W1 mix_w) + w0))   (heads x dim)
    per head and token:  o = (S + diag(u) k v^T)^T r = S^T r + (sum_i r_i u_i k_i) v;   then S <- diag(d) S + k v^T
    out = Wo concat_h (o_h / sqrt(mean(o_h^2) + eps) * n_h * silu(Wg mix_g)_h)      n: heads x dim values

The layer keeps nothing per position; per request it keeps one flat float32 state: the last input (hidden values), then S
(heads, dim, dim).  A state slot is zeroed when a request takes it, which is both "zeros before the first token" and "the
state starts at zero".

A step: one kernel makes the five mixes and replaces the kept input; the four wide products (one launch for decode steps);
the narrow product of the decay; one kernel that leaves r, k, v, the decays and the current token's shares in float32 -- in
small steps it applies W2 itself, larger ones hand that to a product --; the recurrence (a sequence's tokens in order,
whatever their number); the gated norm of its output; the output product.  Mixes, tanh, decays, the state, the recurrence
and the norm are float32 arithmetic.
"""
from ..cache.manager import StateNeed
from ..errors import ConfigError
from ..weights.loader import Want
from .base import register
from .conv import plan_sequences, step_sequences

STREAMS = ("r", "k", "v", "g", "w")
SMALL_STEP = 32         # steps of at most so many tokens apply W2 in the kernel that makes the decays (bfloat16)


class WkvMixing:
    graph_safe = True       # forward() depends on the batch only through the lengths of the step's arrays

    def __init__(self, hidden, heads, dim, eps, decay_rank=None, prefix="", names=None):
        self.D, self.H, self.dim, self.eps = int(hidden), int(heads), int(dim), float(eps)
        self.C = self.H * self.dim
        self.decay_rank = int(decay_rank) if decay_rank else -1        # None: whatever the stored tensors have
        n = dict(r="r", k="k", v="v", g="g", o="o", norm="norm", w1="w1", w2="w2", w0="w0", u="u")
        n.update({"mu_" + s: "mu." + s for s in STREAMS})
        n.update(names or {})
        self.n = {k: prefix + v for k, v in n.items()}
        self.state_offset = 0
        self.mu = self.w_in = self.w1 = self.w2 = self.w0 = self.u = self.norm_w = self.wo = None

    def wants(self):
        D, C = self.D, self.C
        return ([Want(self.n["mu_" + s], (D,), "vector") for s in STREAMS]
                + [Want(self.n[s], (C, D), "matrix") for s in "rkvg"]
                + [Want(self.n["w1"], (self.decay_rank, D), "matrix"), Want(self.n["w2"], (C, self.decay_rank), "matrix"),
                   Want(self.n["w0"], (C,), "vector"), Want(self.n["u"], (self.H, self.dim), "vector"),
                   Want(self.n["norm"], (C,), "vector"), Want(self.n["o"], (D, C), "matrix")])

    def bind(self, tensors, env):
        import torch
        t = lambda k: tensors[self.n[k]]
        if t("w1").shape[0] != t("w2").shape[1]:
            raise ConfigError("the two matrices of the decay's low-rank product do not fit each other")
        self.mu = torch.stack([t("mu_" + s) for s in STREAMS], 0).contiguous()
        self.w_in = torch.cat([t(s) for s in "rkvg"], 0).contiguous()      # the four groups of one launch, or four products
        self.w1, self.w2, self.w0, self.wo = t("w1"), t("w2"), t("w0"), t("o")
        self.u = t("u").reshape(-1).contiguous()
        self.norm_w = t("norm").view(self.H, self.dim)

    def cache_need(self):
        return None

    def state_floats(self):
        return self.D + self.C * self.dim

    def state_need(self):
        return StateNeed((self.state_floats(),), "float32")

    def prepare(self, ctx):
        plan_sequences(ctx)

    def forward(self, ctx, h, run, out="delta"):
        import torch
        ops, N = ctx.ops, ctx.N
        H, dim, C, D = self.H, self.dim, self.C, self.D
        f32 = torch.float32
        state = ctx.cache.state[run.state_id]
        off = self.state_offset
        mixes = ctx.ws.get("wkv_mixes", N * len(STREAMS), (D,), ctx.dtype,
                           reserve=ctx.ws.max_rows * len(STREAMS)).view(len(STREAMS), N, D)
        ops.token_mix(h, self.mu, state[:, off:off + D], step_sequences(ctx), mixes)
        rows = ctx.ws.get("wkv_in", N, (4 * C,), ctx.dtype)
        ops.linear_groups(mixes[:4], self.w_in, rows)
        R = self.w1.shape[0]
        low = ctx.ws.get("wkv_low", N, (R,), f32)
        ops.linear(mixes[4], self.w1, out=low, out_dtype=f32)
        r, k, v, g, o = (ctx.ws.get("wkv_" + x, N, (C,), f32) for x in ("r", "k", "v", "decay", "o"))
        share = ctx.ws.get("wkv_share", N, (H,), f32)
        if N <= SMALL_STEP and ctx.dtype == torch.bfloat16:
            ops.wkv_gates(rows, self.w0, self.u, r, k, v, g, share, H, dim, low=low, w2=self.w2)
        else:
            bent = ctx.ws.get("wkv_tanh", N, (R,), ctx.dtype)
            ops.tanh_rows(low, bent)
            z = ctx.ws.get("wkv_z", N, (C,), f32)
            ops.linear(bent, self.w2, out=z, out_dtype=f32)
            ops.wkv_gates(rows, self.w0, self.u, r, k, v, g, share, H, dim, z=z)
        ops.gated_scan(r, k, v, g, o, state[:, off + D:off + self.state_floats()],
                       (ctx.dev("q_start"), ctx.dev("q_len"), ctx.dev("state_slot")), H, H, dim, dim, per_head=False,
                       bonus=share)
        a = ctx.ws.get("wkv_gated", N, (C,), ctx.dtype)
        ops.gated_rms(o, rows[:, 3 * C:], self.norm_w, a, H, dim, self.eps, silu=True)
        y = ctx.ws.get(out, N, (D,), ctx.dtype)
        ops.linear(a, self.wo, out=y)
        return y, None


register("mixer", "wkv", WkvMixing)
