"""Plain, slow implementation of the Pobelorn decoder: whole sequences, no cache, no state carried between calls, one
function per mechanism.

It is the oracle the engine is compared with and shares no code with ``mashbox_b200``: it reads config.json's keys
itself (a dict) and works on CPU tensors in float64.

The design, in this file's notation.  T tokens at positions 0 .. T-1, width D, rms(x) = x / sqrt(mean(x^2) + eps).

  x        = c E[token]
  layer    : h = rms(x) w;  x <- x + mixer(h) + ff(h)      one norm, read by both; the layer may lack a feed-forward
  lightning: q = silu(Wq h), k = silu(Wk h) (heads x dim), v = silu(Wv h) (heads x vdim);
             per head  S <- decay_h S + k v^T;  o = S^T q;
             out = Wo (rms(concat_h o_h) n * sigmoid(Wg h)), the mean taken over all heads at once
  attention: q = Wq h (heads x dim), k = Wk h (kv_heads x dim), v = Wv h (kv_heads x vdim);
             the first R dims of every q and k head turn, dim 2i with dim 2i + 1, by p f_i, cos and sin times a gain;
             then q <- rms(q), k <- rms(k) per head, without weights;
             v <- (1 - lam) v + lam v0 where v0 are the values of the first layer that mixes (that layer keeps its own);
             weights: softmax over the seen keys of scale q_i . k_j;  i sees j <= i with i - j < size or j < keep_first
             out = Wo concat_h sum_j weight_j v_j
  frequencies: f_i = base^(-2i/R); bent when there is a scaling: index(t) = R ln(original / (2 pi t)) / (2 ln base),
             lo = max(floor(index(fast)), 0), hi = min(ceil(index(slow)), R - 1), r_i = clamp((i - lo) / max(hi - lo, 1e-3)),
             f_i <- r_i f_i / factor + (1 - r_i) f_i, gain = 0.1 ln(factor) + 1
  dense    : Wdown relu(Wup h)^2
  routed   : z = Wr h + b; the `top` largest z are chosen, weights softmax over the chosen z alone;
             out = sum weight_e expert_e(h) + shared(h);  expert(h) = Wdown (silu(Wgate h) * (Wup h))
  logits   = E rms(x) w_final                               the embedding table, without c
"""
import math

import torch

F64 = torch.float64


def rms(x, eps, w=None):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def silu(z):
    return z * torch.sigmoid(z)


def frequencies(rot):
    """-> (frequency per pair, gain of cos and sin)"""
    R, base = int(rot["dims"]), float(rot["base"])
    f = [base ** (-2.0 * i / R) for i in range(R // 2)]
    sc = rot.get("scaling")
    if not sc:
        return torch.tensor(f, dtype=F64), 1.0
    factor, original = float(sc["factor"]), float(sc["original"])

    def index(turns):
        return R * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(index(float(sc["fast"]))), 0), min(math.ceil(index(float(sc["slow"]))), R - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * ramp + fi * (1.0 - ramp))
    return torch.tensor(out, dtype=F64), 0.1 * math.log(factor) + 1.0


def rotate(x, positions, rot):
    """x (T, heads, dim): neighbours of the first rot["dims"] values of every head turn together"""
    if not rot or not rot.get("dims"):
        return x
    R = int(rot["dims"])
    f, gain = frequencies(rot)
    a = positions.to(F64)[:, None] * f[None, :]
    c, s = (gain * torch.cos(a))[:, None, :], (gain * torch.sin(a))[:, None, :]
    u, v = x[..., 0:R:2], x[..., 1:R:2]
    turned = torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2)
    return torch.cat([turned, x[..., R:]], -1)


def seen(T, mask):
    """-> (T, T) bool: whether the query of a row sees the key of a column"""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    ok = j <= i
    if mask and mask.get("size"):
        ok = ok & ((i - j < int(mask["size"])) | (j < int(mask.get("keep_first") or 0)))
    return ok


def mixed_values(v, first, lam):
    """v of this layer, v of the first layer that mixes (None: this is that layer)"""
    return v if first is None else (1.0 - lam) * v + lam * first


def attention(W, p, m, h, eps, first=None):
    """-> (output (T, D), this layer's own values (T, kv_heads vdim) before any mixing)"""
    T = h.shape[0]
    H, G = int(m["heads"]), int(m.get("kv_heads") or m["heads"])
    dim, vdim = int(m["dim"]), int(m["vdim"])
    pos = torch.arange(T)
    q = rms(rotate((h @ W[p + "q"].T).view(T, H, dim), pos, m.get("rot")), eps)
    k = rms(rotate((h @ W[p + "k"].T).view(T, G, dim), pos, m.get("rot")), eps)
    own = h @ W[p + "v"].T
    v = (mixed_values(own, first, W[p + "vmix"]) if m.get("v_mix") else own).view(T, G, vdim)
    ok = seen(T, m.get("mask"))
    out = torch.zeros(T, H, vdim, dtype=F64)
    for a in range(H):
        g = a // (H // G)
        s = (q[:, a] @ k[:, g].T) * float(m["scale"])
        out[:, a] = torch.softmax(torch.where(ok, s, torch.full_like(s, -math.inf)), -1) @ v[:, g]
    return out.reshape(T, H * vdim) @ W[p + "o"].T, own


def lightning(W, p, m, h, eps, state=None):
    """h (T, D) -> (T, D); state: None (zeros) or a (heads, dim, vdim) tensor that is updated in place"""
    T = h.shape[0]
    H, dim, vdim = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = silu(h @ W[p + "q"].T).view(T, H, dim)
    k = silu(h @ W[p + "k"].T).view(T, H, dim)
    v = silu(h @ W[p + "v"].T).view(T, H, vdim)
    decay = torch.tensor([float(d) for d in m["decay"]], dtype=F64)[:, None, None]
    S = state if state is not None else torch.zeros(H, dim, vdim, dtype=F64)
    o = torch.zeros(T, H, vdim, dtype=F64)
    for t in range(T):
        S.copy_(decay * S + k[t][:, :, None] * v[t][:, None, :])
        o[t] = (S * q[t][:, :, None]).sum(1)
    return (rms(o.reshape(T, H * vdim), eps, W[p + "norm"]) * torch.sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def dense(W, p, h):
    return torch.clamp(h @ W[p + "up"].T, min=0.0) ** 2 @ W[p + "down"].T


def expert(W, p, h):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def choose(z, top):
    """z (T, E) logits -> (T, top) indexes of the chosen experts, largest first, lower index on ties"""
    c, ids = z.clone(), []
    for _ in range(top):
        at = c.argmax(-1)          # torch returns the first of equal values
        ids.append(at)
        c[torch.arange(z.shape[0]), at] = -math.inf
    return torch.stack(ids, 1)


def routed(W, p, f, h):
    z = h @ W[p + "router"].T + W[p + "router.b"]
    ids = choose(z, int(f["router"]["top"]))
    wts = torch.softmax(torch.gather(z, 1, ids), -1)
    out = torch.zeros_like(h)
    for e in range(int(f["router"]["experts"])):
        t, place = torch.nonzero(ids == e, as_tuple=True)
        if len(t):
            out[t] += wts[t, place][:, None] * expert(W, f"{p}e{e}.", h[t])
    if f.get("shared"):
        out = out + expert(W, p + "shared.", h)
    return out


def forward(cfg, W, tokens, keep_layers=False):
    """-> logits (T, vocab) float64 (and the stream after every layer, when asked)"""
    W = {k: v.to(F64) if v.is_floating_point() else v for k, v in W.items()}
    eps = float(cfg["norm"]["eps"])
    t = torch.as_tensor(tokens, dtype=torch.long)
    x = W["embed"][t] * float(cfg["embedding"]["scale"])
    first, handed = None, []
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer.get("mlp")
        h = rms(x, eps, W[p + "norm1"])
        if layer["type"] == "lightning":
            y = lightning(W, p + "mix.", m, h, eps)
        elif layer["type"] == "attention":
            y, own = attention(W, p + "mix.", m, h, eps, first)
            if m.get("v_mix") and first is None:
                first = own
        else:
            raise ValueError(layer["type"])
        if f:
            y = y + (dense(W, p + "mlp.", h) if f["kind"] == "dense" else routed(W, p + "mlp.", f, h))
        x = x + y
        handed.append(x)
    logits = rms(x, eps, W["final.norm"]) @ W["embed"].T
    return (logits, torch.stack(handed)) if keep_layers else logits
