"""The Lorozen decoder as data: which parts each layer has, in which order layers run and which tensors exist under which
names.

Token rows enter the stream as they are.  Every layer is a sandwich block -- a norm before and after each sublayer.  A
layer's mixer is attention (biases on q, k and v; heads rotated in part, halves paired, long wavelengths slowed; a sliding
window; a sink per head), latent attention (queries straight from the input, one latent vector and one rotated key strip
kept per position, a sliding window, a gate per head) or wkv (inputs mixed with the token before, a matrix state per head
with a decay per key channel, nothing kept per position).  Its feed-forward is a dense unit gated by the tanh form of gelu,
routed experts whose weights are sigmoid scores that meet the experts' inputs, beside an expert every token uses, or absent.
A run of neighbouring layers may be passed through several times with the same weights: the schedule names those layers
again, every run with a cache or state of its own (numbered by the run), and the embedding's output joins the stream before
every pass but the first.  Stored names: `embed`, `l<i>.norm1|norm1b|norm2|norm2b`, `l<i>.mix.*`,
`l<i>.mlp.gate|up|down|router|e<j>.gate|up|down|shared.gate|up|down`, `final.norm`, `head`.
"""
from ..config.lorozen import DenseFF, LorozenConfig
from ..parts.base import LayerRun, LayerSpec, ModelSpec, PartSpec

DEFAULT_RANK = 16       # inner width of a wkv layer's decay product when random weights are made and none is given


def _rope(rot, head_dim, pairing):
    if rot is None:
        return None
    scaling = ("llama3",) + tuple(rot.scaling) if rot.scaling else None
    return PartSpec("rope", head_dim=head_dim, rotary_dim=rot.dims, theta=rot.base, pairing=pairing, scaling=scaling)


def _mixer(layer, D, eps):
    m = layer.mixer
    if layer.type == "attention":
        return PartSpec("gated_attention", hidden=D, heads=m.heads, kv_heads=m.kv_heads, head_dim=m.dim, vdim=m.vdim,
                        scale=m.scale, eps=eps, bias=True, sink="mix.sink", window=m.window,
                        position=_rope(m.rot, m.dim, "halves"), names={k: "mix." + k for k in "qkvo"})
    if layer.type == "latent_attention":
        return PartSpec("latent_attention", hidden=D, heads=m.heads, dim=m.dim, vdim=m.vdim, q_rank=None, kv_rank=m.kv_rank,
                        eps=eps, scale=m.scale, gate="head", rot_dim=m.rot_dim, window=m.window,
                        position=_rope(m.rot, m.rot_dim, "adjacent"),
                        names={k: "mix." + v for k, v in dict(q="q", dkv="dkv", dkv_norm="dkv.norm", uk="uk", uv="uv", g="g",
                                                              o="o").items()})
    names = {k: "mix." + k for k in ("r", "k", "v", "g", "o", "norm", "w1", "w2", "w0", "u")}
    names.update({"mu_" + s: "mix.mu." + s for s in "rkvgw"})
    return PartSpec("wkv", hidden=D, heads=m.heads, dim=m.dim, eps=eps, decay_rank=m.decay_rank, names=names)


def _feed_forward(f, D):
    if f is None:
        return None
    if isinstance(f, DenseFF):
        return PartSpec("geglu", hidden=D, intermediate=f.ff, names=dict(gate="mlp.gate", up="mlp.up", down="mlp.down"))
    shared = None
    if f.shared_ff:
        shared = PartSpec("swiglu", hidden=D, intermediate=f.shared_ff, names=dict(gate="gate", up="up", down="down"))
    return PartSpec("routed_experts", hidden=D, intermediate=f.ff, experts=f.experts, top=f.top, limit=None, alpha=1.0,
                    shift=0.0, correction=False, weigh="input", shared=shared, shared_prefix="mlp.shared.")


def model_spec(c: LorozenConfig) -> ModelSpec:
    D, eps = c.width, c.norm_eps
    norm = PartSpec("rms", width=D, eps=eps)
    layers = [LayerSpec(prefix=f"l{i}.", block=PartSpec("sandwich", mixer=_mixer(layer, D, eps),
                                                        ffn=_feed_forward(layer.mlp, D), norm=norm))
              for i, layer in enumerate(c.layers)]
    schedule = []
    for run, (i, again) in enumerate(c.order()):
        keeps = c.layers[i].type != "wkv"
        schedule.append(LayerRun(layer=i, cache=run if keeps else None, write=keeps, state=None if keeps else run,
                                 rejoin=again))
    return ModelSpec(hidden=D, vocab=c.vocab,
                     embedding=PartSpec("table", vocab=c.vocab, hidden=D, name="embed"),
                     layers=layers, schedule=schedule,
                     final_norm=PartSpec("rms", width=D, eps=eps, name="final.norm"),
                     head=PartSpec("linear", vocab=c.vocab, hidden=D, tied=False, name="head", softcap=c.logit_softcap))


def canonical_names(c: LorozenConfig):
    """stored names are the canonical ones, except that the dense units' matrices get the `.weight` their part appends; a
    name outside the configuration's table is unexpected"""
    known = set(stored_tensors(c))
    dense = {f"l{i}.mlp.{r}" for i, layer in enumerate(c.layers) if isinstance(layer.mlp, DenseFF) for r in ("gate", "up", "down")}

    def canonical(name):
        if name not in known:
            raise KeyError(name)
        return (name + ".weight" if name in dense or ".mlp.shared." in name else name), None
    return canonical


def stored_tensors(c: LorozenConfig):
    """names, shapes and kinds of the tensors a checkpoint of this configuration holds"""
    D = c.width
    out = {"embed": ((c.vocab, D), "matrix")}
    for i, layer in enumerate(c.layers):
        p, m, f = f"l{i}.", layer.mixer, layer.mlp
        for n in ("norm1", "norm1b"):
            out[p + n] = ((D,), "norm")
        x = p + "mix."
        if layer.type == "attention":
            for r, rows in (("q", m.heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.kv_heads * m.vdim)):
                out[x + r] = ((rows, D), "matrix")
                out[x + r + ".b"] = ((rows,), "bias")
            out[x + "sink"] = ((m.heads,), "bias")
            out[x + "o"] = ((D, m.heads * m.vdim), "matrix")
        elif layer.type == "latent_attention":
            out[x + "q"] = ((m.heads * (m.dim + m.rot_dim), D), "matrix")
            out[x + "dkv"] = ((m.kv_rank + m.rot_dim, D), "matrix")
            out[x + "dkv.norm"] = ((m.kv_rank,), "norm")
            out[x + "uk"] = ((m.heads * m.dim, m.kv_rank), "matrix")
            out[x + "uv"] = ((m.heads * m.vdim, m.kv_rank), "matrix")
            out[x + "g"] = ((m.heads, D), "matrix")
            out[x + "o"] = ((D, m.heads * m.vdim), "matrix")
        else:
            C, rank = m.heads * m.dim, m.decay_rank or DEFAULT_RANK
            for s in "rkvgw":
                out[x + "mu." + s] = ((D,), "fraction")
            for r in "rkvg":
                out[x + r] = ((C, D), "matrix")
            out[x + "w1"] = ((rank, D), "matrix")
            out[x + "w2"] = ((C, rank), "matrix")
            out[x + "w0"] = ((C,), "bias")
            out[x + "u"] = ((m.heads, m.dim), "bias")
            out[x + "norm"] = ((C,), "norm")
            out[x + "o"] = ((D, C), "matrix")
        if f is not None:
            for n in ("norm2", "norm2b"):
                out[p + n] = ((D,), "norm")
        if isinstance(f, DenseFF):
            out[p + "mlp.gate"] = ((f.ff, D), "matrix")
            out[p + "mlp.up"] = ((f.ff, D), "matrix")
            out[p + "mlp.down"] = ((D, f.ff), "matrix")
        elif f is not None:
            for y, ff in [(f"{p}mlp.e{e}.", f.ff) for e in range(f.experts)] + \
                    ([(p + "mlp.shared.", f.shared_ff)] if f.shared_ff else []):
                out[y + "gate"] = ((ff, D), "matrix")
                out[y + "up"] = ((ff, D), "matrix")
                out[y + "down"] = ((D, ff), "matrix")
            out[p + "mlp.router"] = ((f.experts, D), "matrix")
    out["final.norm"] = ((D,), "norm")
    out["head"] = ((c.vocab, D), "matrix")
    return out
