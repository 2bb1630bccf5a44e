"""Plain, slow implementation of the Lorozen decoder: whole sequences, no cache, no state carried between calls, one
function per mechanism.

It is the oracle the engine is compared with and shares no code with ``mashbox_b200``: it reads config.json's keys
itself (a dict) and works on CPU tensors in float64.

The design, in this file's notation.  T tokens at positions 0 .. T-1, width D, rms(x; w) = x / sqrt(mean(x^2) + eps) w.

  stream   : x = e = E[token];  per layer  x <- x + rms(mixer(rms(x; n1)); n1b);  x <- x + rms(ff(rms(x; n2)); n2b) when
             the layer has a feed-forward;  a run of neighbouring layers is passed through several times with the same
             weights, and before every pass but the first x <- x + e;  logits = cap tanh(W_head rms(x; nf) / cap)
  windowed : q, k, v = W h + b (kv heads shared by runs of query heads);  the first R dims of every q and k head rotated
             (dim i with dim i + R/2, long wavelengths slowed);  s_ij = scale q_i.k_j for 0 <= i - j < window;
             p_ij = e^s_ij / (e^sink_h + sum_j e^s_ij);  out = Wo concat_h sum_j p_ij v_j
  latent   : q_h = Wq h = [u_h (dim) | r_h (rot_dim)];  Wdkv h = [c' (kv_rank) | kr (rot_dim)], c = rms(c'; nkv);
             r_h and kr rotated (adjacent pairs);  s_ij = scale (u_i . Wuk_h c_j + r_i . kr_j), 0 <= i - j < window;
             out = Wo concat_h(sigmoid(Wg h)_h sum_j softmax(s)_ij Wuv_h c_j)
  wkv      : h' the input of the token before (zeros before the first), mix_s = h + (h' - h) mu_s for s in r, k, v, g, w;
             r, k, v = W_s mix_s (heads x dim);  d = exp(-exp(W2 tanh(W1 mix_w) + w0));
             per head  o = S^T r + (sum_i r_i u_i k_i) v;  S <- diag(d) S + k v^T;
             out = Wo (concat_h rms(o_h) n silu(W_g mix_g))
  dense    : Wd (gelu_tanh(Wg h) (Wu h))
  experts  : s = sigmoid(Wr h); the `top` largest; out = sum_e expert_e(s_e h) + shared(h), expert(z) = Wd (silu(Wg z) (Wu z))
"""
import math

import torch

F64 = torch.float64


def rms(x, eps, w=None):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def frequencies(rot):
    """one angle per position step for every rotated pair"""
    R, base = int(rot["dims"]), float(rot["base"])
    f = [base ** (-2.0 * i / R) for i in range(R // 2)]
    sc = rot.get("scaling")
    if not sc:
        return torch.tensor(f, dtype=F64)
    factor, low, high, original = (float(sc[k]) for k in ("factor", "low", "high", "original"))
    out = []
    for x in f:
        wave = 2 * math.pi / x
        if wave < original / high:
            out.append(x)
        elif wave > original / low:
            out.append(x / factor)
        else:
            s = (original / wave - low) / (high - low)
            out.append((1 - s) * x / factor + s * x)
    return torch.tensor(out, dtype=F64)


def rotate(x, positions, rot, layout):
    """x (T, heads, dim): the first rot["dims"] values of every head turn by position * frequency; layout "halves"
    pairs value i with value i + dims/2, "adjacent" pairs value 2i with value 2i + 1"""
    if not rot or not rot.get("dims"):
        return x
    R = int(rot["dims"])
    a = positions.to(F64)[:, None] * frequencies(rot)[None, :]
    c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    if layout == "halves":
        u, v = x[..., :R // 2], x[..., R // 2:R]
        return torch.cat([u * c - v * s, v * c + u * s, x[..., R:]], -1)
    u, v = x[..., 0:R:2], x[..., 1:R:2]
    turned = torch.stack([u * c - v * s, v * c + u * s], -1).reshape(*x.shape[:-1], R)
    return torch.cat([turned, x[..., R:]], -1)


def visible(T, mask):
    """(T, T): query i (row) sees key j; mask None: every earlier key and itself"""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    return seen & (i - j < int(mask["size"])) if mask else seen


def softmax_with_sink(s, sink):
    """s (H, T, T) with -inf where a key is not seen; sink (H,): one more term in the denominator that has no value"""
    b = sink[:, None, None].expand(s.shape[0], s.shape[1], 1)
    return torch.softmax(torch.cat([s, b], -1), -1)[..., :-1]


def windowed_attention(W, p, m, h, eps):
    T = h.shape[0]
    H, dim, vdim = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    G = int(m.get("kv_heads") or H)
    pos = torch.arange(T)
    q = rotate((h @ W[p + "q"].T + W[p + "q.b"]).view(T, H, dim), pos, m.get("rot"), "halves")
    k = rotate((h @ W[p + "k"].T + W[p + "k.b"]).view(T, G, dim), pos, m.get("rot"), "halves")
    v = (h @ W[p + "v"].T + W[p + "v.b"]).view(T, G, vdim)
    k, v = k.repeat_interleave(H // G, 1), v.repeat_interleave(H // G, 1)
    s = torch.einsum("ihd,jhd->hij", q, k) * float(m["scale"])
    w = softmax_with_sink(s.masked_fill(~visible(T, m.get("mask")), -math.inf), W[p + "sink"])
    return torch.einsum("hij,jhd->ihd", w, v).reshape(T, H * vdim) @ W[p + "o"].T


def latent_attention(W, p, m, h, eps):
    T = h.shape[0]
    H, dim, vdim = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    rd, rank = int(m.get("rot_dim") or 0), int(m["kv_rank"])
    pos = torch.arange(T)
    q = (h @ W[p + "q"].T).view(T, H, dim + rd)
    low = h @ W[p + "dkv"].T
    c = rms(low[:, :rank], eps, W[p + "dkv.norm"])
    k = (c @ W[p + "uk"].T).view(T, H, dim)
    v = (c @ W[p + "uv"].T).view(T, H, vdim)
    s = torch.einsum("ihd,jhd->hij", q[..., :dim], k)
    if rd:
        qr = rotate(q[..., dim:], pos, m.get("rot"), "adjacent")
        kr = rotate(low[:, None, rank:], pos, m.get("rot"), "adjacent")[:, 0]
        s = s + torch.einsum("ihd,jd->hij", qr, kr)
    w = torch.softmax((s * float(m["scale"])).masked_fill(~visible(T, m.get("mask")), -math.inf), -1)
    o = torch.einsum("hij,jhd->ihd", w, v) * torch.sigmoid(h @ W[p + "g"].T)[:, :, None]
    return o.reshape(T, H * vdim) @ W[p + "o"].T


def wkv(W, p, m, h, eps):
    T = h.shape[0]
    H, dim = int(m["heads"]), int(m["dim"])
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]], 0)

    def mixed(s):
        return h + (before - h) * W[p + "mu." + s]
    r, k, v = ((mixed(s) @ W[p + s].T).view(T, H, dim) for s in "rkv")
    d = torch.exp(-torch.exp(torch.tanh(mixed("w") @ W[p + "w1"].T) @ W[p + "w2"].T + W[p + "w0"])).view(T, H, dim)
    u = W[p + "u"].reshape(H, dim)
    S = torch.zeros(H, dim, dim, dtype=F64)
    o = torch.zeros(T, H, dim, dtype=F64)
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S + u[:, :, None] * kv, r[t])
        S = d[t][:, :, None] * S + kv
    o = rms(o, eps).reshape(T, H * dim) * W[p + "norm"] * silu(mixed("g") @ W[p + "g"].T)
    return o @ W[p + "o"].T


def gated_unit(W, p, h, act):
    return (act(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def experts(W, p, f, h):
    top = int(f["router"]["top"])
    s = torch.sigmoid(h @ W[p + "router"].T)
    best = torch.topk(s, top, -1)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for w, e in zip(best.values[t], best.indices[t]):
            out[t] += gated_unit(W, f"{p}e{int(e)}.", (w * h[t])[None], silu)[0]
    if f.get("shared"):
        out = out + gated_unit(W, p + "shared.", h, silu)
    return out


def feed_forward(W, p, f, h):
    if f.get("kind", "dense") == "dense":
        return gated_unit(W, p, h, gelu_tanh)
    return experts(W, p, f, h)


MIXERS = {"attention": windowed_attention, "latent_attention": latent_attention, "wkv": wkv}


def order_of_layers(cfg):
    """-> [(layer, whether the embedding is added to the stream right before it)]"""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    return ([(i, False) for i in range(a)] + [(i, t > 0 and i == a) for t in range(times) for i in range(a, b)]
            + [(i, False) for i in range(b, n)])


def forward(cfg, W, tokens, after_layers=None):
    """config.json as a dict, tensors by stored name (any float dtype), token ids -> float64 logits (T, vocab);
    after_layers: a list that receives the stream after every layer run"""
    W = {k: (v.to(F64) if v.is_floating_point() else v) for k, v in W.items()}
    eps = float(cfg["norm"]["eps"])
    x = start = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, again in order_of_layers(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if again:
            x = x + start
        y = MIXERS[layer["type"]](W, p + "mix.", layer["mixer"], rms(x, eps, W[p + "norm1"]), eps)
        x = x + rms(y, eps, W[p + "norm1b"])
        if layer.get("mlp") is not None:
            y = feed_forward(W, p + "mlp.", layer["mlp"], rms(x, eps, W[p + "norm2"]))
            x = x + rms(y, eps, W[p + "norm2b"])
        if after_layers is not None:
            after_layers.append(x.clone())
    logits = rms(x, eps, W["final.norm"]) @ W["head"].T
    cap = cfg.get("logit_softcap")
    return float(cap) * torch.tanh(logits / float(cap)) if cap else logits
