"""Typed configuration of the Lorozen decoder, read from config.json's own keys.

config.json: `architecture` (a string), `width`, `vocab`, `norm.eps`, `logit_softcap` (absent: none), `loop` {start, stop,
times} (absent: every layer runs once) and `layers`, a list with one entry per layer: `type` ("attention",
"latent_attention" or "wkv"), `mixer` (its sizes and constants) and `mlp`, which is {"kind": "dense", "ff"}, {"kind": "moe",
"expert": {"ff"}, "router": {"experts", "top"}, "shared": {"ff"} or absent} or null.  Every layer has its own sizes;
nothing is assumed equal between layers.

An attention mixer: heads, kv_heads (absent: heads), dim, vdim, scale, rot {base, dims, scaling {factor, low, high,
original} or absent} or absent, mask {size} or absent (every earlier key is seen).  A latent_attention mixer: heads, dim
(unrotated), rot_dim (rotated; absent: none), vdim, kv_rank, scale, rot {base, dims} or absent, mask as above.  A wkv mixer:
heads, dim; the inner width of its decay's low-rank product is not in config.json: the stored tensors have it
(`decay_rank` here is None then; random-weights mode sets it and writes it as a key of its own).
"""
from dataclasses import dataclass, field
from typing import Optional

from ..errors import ConfigError


@dataclass(frozen=True)
class Rotation:
    dims: int
    base: float
    scaling: Optional[tuple] = None     # (factor, low, high, original) or None


@dataclass(frozen=True)
class AttentionMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Optional[Rotation] = None
    window: Optional[int] = None        # None: every earlier key


@dataclass(frozen=True)
class LatentMixer:
    heads: int
    dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot_dim: int = 0
    rot: Optional[Rotation] = None
    window: Optional[int] = None


@dataclass(frozen=True)
class WkvMixer:
    heads: int
    dim: int
    decay_rank: Optional[int] = None    # inner width of the decay's low-rank product; None: as stored


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
class Loop:
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class LorozenLayer:
    type: str
    mixer: object
    mlp: object                         # DenseFF, ExpertsFF or None


SCALING = ("factor", "low", "high", "original")


@dataclass(frozen=True)
class LorozenConfig:
    architecture: str
    width: int
    vocab: int
    norm_eps: float
    layers: tuple
    loop: Optional[Loop] = None
    logit_softcap: Optional[float] = None
    extra: dict = field(default_factory=dict, compare=False, hash=False)

    @property
    def num_layers(self):
        return len(self.layers)

    def order(self):
        """-> [(layer, whether a pass of the loop but the first starts with it)] in the order layers run"""
        n, lp = len(self.layers), self.loop
        if lp is None:
            return [(i, False) for i in range(n)]
        passes = [(i, t > 0 and i == lp.start) for t in range(lp.times) for i in range(lp.start, lp.stop)]
        return [(i, False) for i in range(lp.start)] + passes + [(i, False) for i in range(lp.stop, n)]

    @classmethod
    def from_hf(cls, cfg: dict) -> "LorozenConfig":
        arch = cfg.get("architecture") or (cfg.get("architectures") or [None])[0]

        def need(d, key, where):
            if not isinstance(d, dict) or d.get(key) is None:
                raise ConfigError(f"config.json has no `{where}{key}`")
            return d[key]

        def rotation(m, w, most, scaled):
            rot = m.get("rot") or None
            if not rot or not rot.get("dims"):
                return None
            dims = int(rot["dims"])
            if dims % 2 or dims > most:
                raise ConfigError(f"config.json {w}rot.dims = {dims} must be even and at most {most}")
            sc = rot.get("scaling") or None
            if sc and not scaled:
                raise ConfigError(f"config.json {w}rot.scaling is not supported here")
            scaling = tuple(float(need(sc, k, w + "rot.scaling.")) for k in SCALING) if sc else None
            return Rotation(dims=dims, base=float(need(rot, "base", w + "rot.")), scaling=scaling)

        def window(m, w):
            mask = m.get("mask")
            if mask is None:
                return None
            size = int(need(mask, "size", w + "mask."))
            if size < 1:
                raise ConfigError(f"config.json {w}mask.size = {size} must be 1 or more")
            return size

        def attention(m, w):
            heads = int(need(m, "heads", w))
            kv = int(m.get("kv_heads") or heads)
            if kv < 1 or heads % kv:
                raise ConfigError(f"config.json {w}kv_heads = {kv} does not divide heads = {heads}")
            dim = int(need(m, "dim", w))
            return AttentionMixer(heads=heads, kv_heads=kv, dim=dim, vdim=int(need(m, "vdim", w)),
                                  scale=float(need(m, "scale", w)), rot=rotation(m, w, dim, True), window=window(m, w))

        def latent(m, w):
            rd = int(m.get("rot_dim") or 0)
            return LatentMixer(heads=int(need(m, "heads", w)), dim=int(need(m, "dim", w)), vdim=int(need(m, "vdim", w)),
                               kv_rank=int(need(m, "kv_rank", w)), scale=float(need(m, "scale", w)), rot_dim=rd,
                               rot=rotation(m, w, rd, False) if rd else None, window=window(m, w))

        def wkv(m, w):
            return WkvMixer(heads=int(need(m, "heads", w)), dim=int(need(m, "dim", w)),
                            decay_rank=int(m["decay_rank"]) if m.get("decay_rank") else None)

        kinds = {"attention": attention, "latent_attention": latent, "wkv": wkv}
        layers = []
        for i, e in enumerate(need(cfg, "layers", "")):
            w = f"layers[{i}]."
            kind, m = need(e, "type", w), need(e, "mixer", w)
            if kind not in kinds:
                raise ConfigError(f"config.json layers[{i}].type = {kind!r} is not supported for {arch}")
            mixer = kinds[kind](m, w + "mixer.")
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
            layers.append(LorozenLayer(kind, mixer, ff))
        loop = cfg.get("loop") or None
        if loop:
            loop = Loop(*(int(need(loop, k, "loop.")) for k in ("start", "stop", "times")))
            if not 0 <= loop.start < loop.stop <= len(layers) or loop.times < 1:
                raise ConfigError(f"config.json loop: layers {loop.start} .. {loop.stop - 1} of {len(layers)}, "
                                  f"{loop.times} times, is not a run of layers")
        cap = cfg.get("logit_softcap")
        return cls(architecture=arch, width=int(need(cfg, "width", "")), vocab=int(need(cfg, "vocab", "")),
                   norm_eps=float(need(cfg.get("norm"), "eps", "norm.")), layers=tuple(layers), loop=loop,
                   logit_softcap=float(cap) if cap else None,
                   extra={k: cfg[k] for k in ("bos_token_id", "eos_token_id") if k in cfg})

    def to_hf(self) -> dict:
        """The config.json that `from_hf` reads back to this configuration (random-weights mode writes it)."""
        def positions(m, e):
            if m.rot:
                e["rot"] = {"base": m.rot.base, "dims": m.rot.dims}
                if m.rot.scaling:
                    e["rot"]["scaling"] = dict(zip(SCALING, m.rot.scaling))
            if m.window:
                e["mask"] = {"size": m.window}
            return e

        layers = []
        for layer in self.layers:
            m, f = layer.mixer, layer.mlp
            if layer.type == "attention":
                e = positions(m, {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale})
            elif layer.type == "latent_attention":
                e = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "kv_rank": m.kv_rank, "scale": m.scale}
                if m.rot_dim:
                    e["rot_dim"] = m.rot_dim
                e = positions(m, e)
            else:
                e = {"heads": m.heads, "dim": m.dim}
                if m.decay_rank:
                    e["decay_rank"] = m.decay_rank
            mlp = None
            if isinstance(f, DenseFF):
                mlp = {"kind": "dense", "ff": f.ff}
            elif f is not None:
                mlp = {"kind": "moe", "expert": {"ff": f.ff}, "router": {"experts": f.experts, "top": f.top}}
                if f.shared_ff:
                    mlp["shared"] = {"ff": f.shared_ff}
            layers.append({"type": layer.type, "mixer": e, "mlp": mlp})
        out = {"architecture": self.architecture, "width": self.width, "vocab": self.vocab, "norm": {"eps": self.norm_eps},
               "layers": layers}
        if self.loop:
            out["loop"] = {"start": self.loop.start, "stop": self.loop.stop, "times": self.loop.times}
        if self.logit_softcap:
            out["logit_softcap"] = self.logit_softcap
        out.update(self.extra)
        return out
