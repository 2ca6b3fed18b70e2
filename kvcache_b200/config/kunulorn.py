"""Configuration of the Kunulorn decoder, read from its own config.json keys.

config.json of this design is nested: `layers` is a list with one object per layer (`type` names the mixer, its sizes lie
under `mixer`, the feed-forward under `mlp` or null), `embedding.scale`, `norm.eps`, `vocab`, `width`.  The mixer is
`attention`: grouped keys, a norm over the whole query and key projections, neighbouring numbers rotated as pairs, a mask
of chunks (`mask.size`), optionally the keys and values of an earlier layer (`kv_from`).  Feed-forwards: `dense` (a clamped
gated activation with `limit`) or `moe` (sigmoid scores, a correction of the choice, groups of experts, a shared expert
with a gate).  Every size and every constant that can differ between models is read here.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple, Union

from .base import KeyReader, ModelConfig

KUNULORN_ARCHITECTURE = "Kunulorn"


@dataclass(frozen=True)
class RotarySpec:
    base: float
    dims: int


@dataclass(frozen=True)
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: Optional[int]             # a query sees the keys of its own chunk of this many tokens, up to itself; None: all
    rot: Optional[RotarySpec]
    kv_from: Optional[int] = None    # the layer whose cached keys and values this layer reads instead of its own


@dataclass(frozen=True)
class DenseSpec:
    ff: int
    limit: float


@dataclass(frozen=True)
class GroupSpec:
    count: int
    keep: int


@dataclass(frozen=True)
class RoutedSpec:
    expert_ff: int
    experts: int
    top: int
    weight_scale: float
    groups: Optional[GroupSpec]
    shared_ff: Optional[int]


@dataclass(frozen=True)
class LayerSpec:
    type: str
    mixer: Optional[AttentionSpec]
    mlp: Union[DenseSpec, RoutedSpec, None]


def _read_attention(lr: KeyReader) -> Optional[AttentionSpec]:
    m = lr.sub("mixer")
    if m is None:
        return None
    mask = m.sub("mask", required=False)
    chunk = mask.integer("size", minimum=1) if mask is not None else None
    m.absorb(mask)
    rot = m.sub("rot", required=False)
    rotary = None
    if rot is not None:
        rotary = RotarySpec(rot.number("base", positive=True), rot.integer("dims", minimum=2))
        if rotary.dims is not None and rotary.dims % 2:
            rot.fail(f"'dims' must be even, got {rotary.dims}")
        m.absorb(rot)
    spec = AttentionSpec(heads=m.integer("heads", minimum=1), kv_heads=m.integer("kv_heads", minimum=1), dim=m.integer("dim", minimum=1),
                         vdim=m.integer("vdim", minimum=1), scale=m.number("scale", positive=True), chunk=chunk, rot=rotary,
                         kv_from=m.integer("kv_from", default=None, minimum=0))
    if None not in (spec.heads, spec.kv_heads) and spec.kv_heads >= 1 and spec.heads % spec.kv_heads:
        m.fail(f"heads {spec.heads} is not a multiple of kv_heads {spec.kv_heads}")
    if rotary is not None and None not in (rotary.dims, spec.dim) and rotary.dims > spec.dim:
        m.fail(f"rot.dims {rotary.dims} exceeds dim {spec.dim}")
    lr.absorb(m)
    return spec


def _read_router(m: KeyReader):
    """(experts, top, weight scale, groups) of a routed feed-forward."""
    router = m.sub("router")
    if router is None:
        return 0, 0, 1.0, None
    experts, top = router.integer("experts", minimum=1), router.integer("top", minimum=1)
    scale = router.number("scale", default=1.0, positive=True)
    groups = None
    g = router.sub("groups", required=False)
    if g is not None:
        groups = GroupSpec(g.integer("count", minimum=1), g.integer("keep", minimum=1))
        router.absorb(g)
    if None not in (experts, top):
        usable = experts
        if groups is not None and None not in (groups.count, groups.keep) and groups.count >= 1:
            if experts % groups.count:
                router.fail(f"experts {experts} is not a multiple of groups.count {groups.count}")
            if groups.keep > groups.count:
                router.fail(f"groups.keep {groups.keep} exceeds groups.count {groups.count}")
            usable = experts // groups.count * min(groups.keep, groups.count)
        if top > usable:
            router.fail(f"top {top} exceeds the {usable} experts that can be chosen")
    m.absorb(router)
    return experts or 0, top or 0, scale, groups


def _read_mlp(lr: KeyReader):
    m = lr.sub("mlp", required=False)
    if m is None:
        return None
    kind = m.string("kind")
    spec = None
    if kind == "dense":
        spec = DenseSpec(m.integer("ff", minimum=1), m.number("limit", positive=True))
    elif kind == "moe":
        experts, top, scale, groups = _read_router(m)
        expert, shared = m.sub("expert"), m.sub("shared", required=False)
        spec = RoutedSpec(expert.integer("ff", minimum=1) if expert is not None else None, experts, top, scale, groups,
                          shared.integer("ff", minimum=1) if shared is not None else None)
        for child in (expert, shared):
            m.absorb(child)
    elif kind is not None:
        m.fail(f"unknown feed-forward kind '{kind}' (dense, moe)")
    lr.absorb(m)
    return spec


@dataclass(frozen=True)
class KunulornConfig(ModelConfig):
    vocab_size: int
    width: int
    norm_eps: float
    layers: Tuple[LayerSpec, ...]
    embed_scale: float = 1.0
    eos_token_ids: Tuple[int, ...] = ()
    initializer_range: float = 0.05

    @classmethod
    def from_dict(cls, data: Mapping[str, Any], where: str = "config.json") -> "KunulornConfig":
        r = KeyReader(data, where)
        vocab, width = r.integer("vocab", minimum=1), r.integer("width", minimum=1)
        norm = r.sub("norm")
        eps = norm.number("eps", positive=True) if norm is not None else None
        r.absorb(norm)
        emb = r.sub("embedding", required=False)
        scale = emb.number("scale", default=1.0) if emb is not None else 1.0
        r.absorb(emb)
        raw_layers = data.get("layers")
        layers = []
        if not isinstance(raw_layers, (list, tuple)) or not raw_layers:
            r.fail("'layers' must be a non-empty list")
        else:
            for i, item in enumerate(raw_layers):
                if not isinstance(item, Mapping):
                    r.fail(f"layers[{i}] must be an object")
                    layers.append(LayerSpec("", None, None))
                    continue
                lr = KeyReader(item, f"{where}: layers[{i}]")
                kind = lr.string("type")
                if kind is not None and kind != "attention":
                    lr.fail(f"unknown mixer type '{kind}' (attention)")
                    kind = None
                layers.append(LayerSpec(kind, _read_attention(lr) if kind is not None else None, _read_mlp(lr)))
                r.absorb(lr)
            # A layer that reads another's keys and values: the other lies before it, projects its own, and agrees in what
            # is cached.
            for i, layer in enumerate(layers):
                m = layer.mixer
                if m is None or m.kv_from is None:
                    continue
                j = m.kv_from
                src = layers[j].mixer if j < i else None
                if src is None or src.kv_from is not None:
                    r.fail(f"layers[{i}]: kv_from {j} must name an earlier attention layer that keeps its own keys and values")
                elif (src.kv_heads, src.dim, src.vdim, src.rot) != (m.kv_heads, m.dim, m.vdim, m.rot):
                    r.fail(f"layers[{i}]: kv_heads, dim, vdim and rot must equal those of layer {j}, whose keys and values it reads")
        eos = r.int_list("eos_token_id", default=())
        init_range = r.number("initializer_range", default=0.05, positive=True)
        r.finish()
        return cls(architecture=KUNULORN_ARCHITECTURE, vocab_size=vocab, width=width, norm_eps=eps, layers=tuple(layers),
                   embed_scale=scale, eos_token_ids=eos, initializer_range=init_range)

    def to_dict(self) -> Dict[str, Any]:
        def mixer(s: AttentionSpec):
            out: Dict[str, Any] = {"heads": s.heads, "kv_heads": s.kv_heads, "dim": s.dim, "vdim": s.vdim, "scale": s.scale}
            if s.chunk is not None:
                out["mask"] = {"size": s.chunk}
            if s.rot is not None:
                out["rot"] = {"base": s.rot.base, "dims": s.rot.dims}
            if s.kv_from is not None:
                out["kv_from"] = s.kv_from
            return out

        def mlp(s):
            if s is None:
                return None
            if isinstance(s, DenseSpec):
                return {"kind": "dense", "ff": s.ff, "limit": s.limit}
            router: Dict[str, Any] = {"experts": s.experts, "top": s.top, "scale": s.weight_scale}
            if s.groups is not None:
                router["groups"] = {"count": s.groups.count, "keep": s.groups.keep}
            out: Dict[str, Any] = {"kind": "moe", "expert": {"ff": s.expert_ff}, "router": router}
            if s.shared_ff is not None:
                out["shared"] = {"ff": s.shared_ff}
            return out

        out: Dict[str, Any] = {
            "architecture": self.architecture, "vocab": self.vocab_size, "width": self.width, "norm": {"eps": self.norm_eps},
            "embedding": {"scale": self.embed_scale},
            "layers": [{"type": l.type, "mixer": mixer(l.mixer), "mlp": mlp(l.mlp)} for l in self.layers],
            "initializer_range": self.initializer_range,
        }
        if len(self.eos_token_ids) == 1:
            out["eos_token_id"] = self.eos_token_ids[0]
        elif len(self.eos_token_ids) > 1:
            out["eos_token_id"] = list(self.eos_token_ids)
        return out
