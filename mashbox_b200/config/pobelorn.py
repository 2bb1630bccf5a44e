"""Typed configuration of the Pobelorn decoder, read from config.json's own keys.

config.json: `architecture` (a string), `width`, `vocab`, `norm.eps`, `embedding.scale` (absent: 1) and `layers`, a list
with one entry per layer: `type` ("attention" or "lightning"), `mixer` (its sizes and constants) and `mlp`, which is
{"kind": "dense", "ff"}, {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top"}, "shared": {"ff"} or absent} or
null.  Every layer has its own sizes; nothing is assumed equal between layers, except that the layers which mix their
values with those of the first such layer have as many values per token.

An attention mixer: heads, kv_heads (absent: heads), dim, vdim, scale, rot {base, dims, scaling {factor, original, fast,
slow} or absent} or absent, mask {size, keep_first (absent: 0)} or absent (every earlier key is seen), v_mix (absent:
false).  A lightning mixer: heads, dim, vdim, decay (a number per head).
"""
from dataclasses import dataclass, field
from typing import Optional

from ..errors import ConfigError


@dataclass(frozen=True)
class Rotation:
    dims: int
    base: float
    scaling: Optional[tuple] = None     # (factor, original, fast, slow) or None


@dataclass(frozen=True)
class AttentionMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Optional[Rotation] = None
    window: Optional[int] = None        # None: every earlier key
    keep_first: int = 0                 # so many first positions stay visible behind the window
    v_mix: bool = False


@dataclass(frozen=True)
class LightningMixer:
    heads: int
    dim: int
    vdim: int
    decay: tuple


@dataclass(frozen=True)
class DenseFF:
    ff: int


@dataclass(frozen=True)
class ExpertsFF:
    ff: int
    experts: int
    top: int
    shared_ff: Optional[int] = None     # None: no shared expert


@dataclass(frozen=True)
class PobelornLayer:
    type: str
    mixer: object
    mlp: object                         # DenseFF, ExpertsFF or None


@dataclass(frozen=True)
class PobelornConfig:
    architecture: str
    width: int
    vocab: int
    norm_eps: float
    layers: tuple
    embedding_scale: float = 1.0
    extra: dict = field(default_factory=dict, compare=False, hash=False)

    @property
    def num_layers(self):
        return len(self.layers)

    @classmethod
    def from_hf(cls, cfg: dict) -> "PobelornConfig":
        arch = cfg.get("architecture") or (cfg.get("architectures") or [None])[0]

        def need(d, key, where):
            if not isinstance(d, dict) or d.get(key) is None:
                raise ConfigError(f"config.json has no `{where}{key}`")
            return d[key]

        def rotation(m, w, most):
            rot = m.get("rot") or None
            if not rot or not rot.get("dims"):
                return None
            dims = int(rot["dims"])
            if dims % 2 or dims > most:
                raise ConfigError(f"config.json {w}rot.dims = {dims} must be even and at most dim = {most}")
            sc = rot.get("scaling") or None
            scaling = None
            if sc:
                scaling = tuple(float(need(sc, k, w + "rot.scaling.")) for k in ("factor", "original", "fast", "slow"))
            return Rotation(dims=dims, base=float(need(rot, "base", w + "rot.")), scaling=scaling)

        def attention(m, w):
            heads = int(need(m, "heads", w))
            kv = int(m.get("kv_heads") or heads)
            if kv < 1 or heads % kv:
                raise ConfigError(f"config.json {w}kv_heads = {kv} does not divide heads = {heads}")
            dim, mask = int(need(m, "dim", w)), m.get("mask") or None
            window, keep = None, 0
            if mask:
                window, keep = int(need(mask, "size", w + "mask.")), int(mask.get("keep_first") or 0)
                if window < 1 or keep < 0:
                    raise ConfigError(f"config.json {w}mask: a window of {window} with {keep} kept tokens")
            return AttentionMixer(heads=heads, kv_heads=kv, dim=dim, vdim=int(need(m, "vdim", w)),
                                  scale=float(need(m, "scale", w)), rot=rotation(m, w, dim), window=window,
                                  keep_first=keep, v_mix=bool(m.get("v_mix")))

        def lightning(m, w):
            heads, decay = int(need(m, "heads", w)), tuple(float(d) for d in need(m, "decay", w))
            if len(decay) != heads:
                raise ConfigError(f"config.json {w}decay has {len(decay)} values for {heads} heads")
            return LightningMixer(heads=heads, dim=int(need(m, "dim", w)), vdim=int(need(m, "vdim", w)), decay=decay)

        layers, mixing = [], None
        for i, e in enumerate(need(cfg, "layers", "")):
            w = f"layers[{i}]."
            kind, m = need(e, "type", w), need(e, "mixer", w)
            if kind == "attention":
                mixer = attention(m, w + "mixer.")
                if mixer.v_mix:
                    per_token = mixer.kv_heads * mixer.vdim
                    if mixing is not None and mixing != per_token:
                        raise ConfigError(f"config.json {w}mixer mixes {per_token} values a token with the {mixing} of the "
                                          f"first layer that does (kv_heads * vdim must agree)")
                    mixing = per_token
            elif kind == "lightning":
                mixer = lightning(m, w + "mixer.")
            else:
                raise ConfigError(f"config.json layers[{i}].type = {kind!r} is not supported for {arch}")
            mlp, w = e.get("mlp"), f"layers[{i}].mlp."
            if mlp is None:
                ff = None
            elif mlp.get("kind", "dense") == "dense":
                ff = DenseFF(ff=int(need(mlp, "ff", w)))
            elif mlp["kind"] == "moe":
                ex, r, shared = need(mlp, "expert", w), need(mlp, "router", w), mlp.get("shared") or {}
                ff = ExpertsFF(ff=int(need(ex, "ff", w + "expert.")), experts=int(need(r, "experts", w + "router.")),
                               top=int(need(r, "top", w + "router.")),
                               shared_ff=int(shared["ff"]) if shared.get("ff") else None)
                if not 1 <= ff.top <= ff.experts:
                    raise ConfigError(f"config.json {w}router: {ff.top} of {ff.experts} experts cannot be chosen")
            else:
                raise ConfigError(f"config.json {w}kind = {mlp.get('kind')!r} is not supported for {arch}")
            layers.append(PobelornLayer(kind, mixer, ff))
        scale = (cfg.get("embedding") or {}).get("scale")
        return cls(architecture=arch, width=int(need(cfg, "width", "")), vocab=int(need(cfg, "vocab", "")),
                   norm_eps=float(need(cfg.get("norm"), "eps", "norm.")), layers=tuple(layers),
                   embedding_scale=1.0 if scale is None else float(scale),
                   extra={k: cfg[k] for k in ("bos_token_id", "eos_token_id") if k in cfg})

    def to_hf(self) -> dict:
        """The config.json that `from_hf` reads back to this configuration (random-weights mode writes it)."""
        def attention(m):
            e = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale, "v_mix": m.v_mix}
            if m.rot:
                e["rot"] = {"base": m.rot.base, "dims": m.rot.dims}
                if m.rot.scaling:
                    e["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), m.rot.scaling))
            if m.window:
                e["mask"] = {"size": m.window, "keep_first": m.keep_first}
            return e

        layers = []
        for layer in self.layers:
            m, f = layer.mixer, layer.mlp
            if layer.type == "attention":
                e = attention(m)
            else:
                e = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "decay": list(m.decay)}
            mlp = None
            if isinstance(f, DenseFF):
                mlp = {"kind": "dense", "ff": f.ff}
            elif f is not None:
                mlp = {"kind": "moe", "expert": {"ff": f.ff}, "router": {"experts": f.experts, "top": f.top}}
                if f.shared_ff:
                    mlp["shared"] = {"ff": f.shared_ff}
            layers.append({"type": layer.type, "mixer": e, "mlp": mlp})
        return {"architecture": self.architecture, "width": self.width, "vocab": self.vocab, "norm": {"eps": self.norm_eps},
                "embedding": {"scale": self.embedding_scale}, "layers": layers, **self.extra}
