"""The Pobelorn decoder as data: which parts each layer has, in which order layers run and which tensors exist under which
names.

Token rows enter the stream times a constant.  Every layer is a parallel block with ONE RMS norm that both sublayers read.
A layer's mixer is attention -- heads rotated in part, neighbours together, and normed after the rotation; a sliding
window behind which the first positions stay visible; values mixed with those of the first layer that does so -- or
lightning attention (a matrix state per head with a fixed decay, nothing kept per position).  Its feed-forward is a dense
unit with a squared ReLU, routed experts whose weights are the softmax over the chosen logits beside an expert every token
uses, or absent.  The output head is the embedding table.  An attention layer names cache i, a lightning layer state i.
Stored names: `embed`, `l<i>.norm1`, `l<i>.mix.*`, `l<i>.mlp.up|down|router[.b]|e<j>.gate|up|down|shared.gate|up|down`,
`final.norm`.
"""
from ..config.pobelorn import DenseFF, PobelornConfig
from ..parts.base import LayerRun, LayerSpec, ModelSpec, PartSpec

YARN_GAIN = 0.1         # cos and sin of a scaled rotation are multiplied by YARN_GAIN ln(factor) + 1


def _rope(rot, head_dim):
    if rot is None:
        return None
    scaling = ("yarn",) + tuple(rot.scaling) + (YARN_GAIN,) if rot.scaling else None
    return PartSpec("rope", head_dim=head_dim, rotary_dim=rot.dims, theta=rot.base, pairing="adjacent", scaling=scaling)


def _first_mixing(c):
    """the first layer whose values are kept for the layers that mix theirs with them (None: no layer mixes)"""
    return next((i for i, layer in enumerate(c.layers) if layer.type == "attention" and layer.mixer.v_mix), None)


def model_spec(c: PobelornConfig) -> ModelSpec:
    D, eps, first = c.width, c.norm_eps, _first_mixing(c)
    norm = PartSpec("rms", width=D, eps=eps)
    layers, schedule = [], []
    for i, layer in enumerate(c.layers):
        m, f = layer.mixer, layer.mlp
        if layer.type == "lightning":
            mixer = PartSpec("lightning", hidden=D, heads=m.heads, dim=m.dim, vdim=m.vdim, decay=list(m.decay), eps=eps,
                             names={k: "mix." + k for k in ("q", "k", "v", "g", "o", "norm")})
            run = LayerRun(layer=i, cache=None, write=False, state=i)
        else:
            mix = None if not m.v_mix else ("keep" if i == first else "mix")
            mixer = PartSpec("gated_attention", hidden=D, heads=m.heads, kv_heads=m.kv_heads, head_dim=m.dim, vdim=m.vdim,
                             scale=m.scale, qk_norm="after", eps=eps, position=_rope(m.rot, m.dim), window=m.window,
                             keep_first=m.keep_first, value_mix=mix,
                             names={k: "mix." + k for k in ("q", "k", "v", "o", "vmix")})
            run = LayerRun(layer=i, cache=i, write=True)
        if f is None:
            ffn = None
        elif isinstance(f, DenseFF):
            ffn = PartSpec("dense_relu2", hidden=D, intermediate=f.ff, names=dict(up="mlp.up", down="mlp.down"))
        else:
            shared = None
            if f.shared_ff:
                shared = PartSpec("swiglu", hidden=D, intermediate=f.shared_ff, names=dict(gate="gate", up="up", down="down"))
            ffn = PartSpec("routed_experts", hidden=D, intermediate=f.ff, experts=f.experts, top=f.top, limit=None, alpha=1.0,
                           shift=0.0, correction=False, score="softmax_chosen", router_bias="mlp.router.b", shared=shared,
                           shared_prefix="mlp.shared.")
        layers.append(LayerSpec(prefix=f"l{i}.", block=PartSpec("parallel", mixer=mixer, ffn=ffn, norm1=norm,
                                                                one_norm=True)))
        schedule.append(run)
    return ModelSpec(hidden=D, vocab=c.vocab,
                     embedding=PartSpec("table", vocab=c.vocab, hidden=D, name="embed", scale=c.embedding_scale),
                     layers=layers, schedule=schedule,
                     final_norm=PartSpec("rms", width=D, eps=eps, name="final.norm"),
                     head=PartSpec("linear", vocab=c.vocab, hidden=D, tied=True, tied_to="embed"))


def canonical_names(c: PobelornConfig):
    """stored names are the canonical ones, except that the shared expert's matrices get the `.weight` its part appends;
    the mixing weight of the first layer that mixes is stored and not read; a name outside the configuration's table is
    unexpected"""
    known, first = set(stored_tensors(c)), _first_mixing(c)

    def canonical(name):
        if name not in known:
            raise KeyError(name)
        if first is not None and name == f"l{first}.mix.vmix":
            return None
        return (name + ".weight" if ".mlp.shared." in name else name), None
    return canonical


def stored_tensors(c: PobelornConfig):
    """names, shapes and kinds of the tensors a checkpoint of this configuration holds"""
    D = c.width
    out = {"embed": ((c.vocab, D), "matrix")}
    for i, layer in enumerate(c.layers):
        p, m, f = f"l{i}.", layer.mixer, layer.mlp
        x = p + "mix."
        out[p + "norm1"] = ((D,), "norm")
        if layer.type == "lightning":
            for r, w in (("q", m.dim), ("k", m.dim), ("v", m.vdim), ("g", m.vdim)):
                out[x + r] = ((m.heads * w, D), "matrix")
            out[x + "norm"] = ((m.heads * m.vdim,), "norm")
        else:
            out[x + "q"] = ((m.heads * m.dim, D), "matrix")
            out[x + "k"] = ((m.kv_heads * m.dim, D), "matrix")
            out[x + "v"] = ((m.kv_heads * m.vdim, D), "matrix")
            if m.v_mix:
                out[x + "vmix"] = ((), "fraction")
        out[x + "o"] = ((D, m.heads * m.vdim), "matrix")
        if isinstance(f, DenseFF):
            out[p + "mlp.up"] = ((f.ff, D), "matrix")
            out[p + "mlp.down"] = ((D, f.ff), "matrix")
        elif f is not None:
            for y, ff in [(f"{p}mlp.e{e}.", f.ff) for e in range(f.experts)] + \
                    ([(p + "mlp.shared.", f.shared_ff)] if f.shared_ff else []):
                out[y + "gate"] = ((ff, D), "matrix")
                out[y + "up"] = ((ff, D), "matrix")
                out[y + "down"] = ((D, ff), "matrix")
            out[p + "mlp.router"] = ((f.experts, D), "matrix")
            out[p + "mlp.router.b"] = ((f.experts,), "bias")
    out["final.norm"] = ((D,), "norm")
    return out
