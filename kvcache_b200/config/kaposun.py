"""Configuration of the Kaposun decoder, read from its own config.json keys.

config.json of this design is nested: `layers` is a list with one object per layer (`type` names the mixer, its sizes lie under
`mixer`, the feed-forward under `mlp` or null), `loop` (layers start .. stop - 1 run `times` times in a row), `norm.eps`,
`residual_mult`, `vocab`, `width`.  Mixers: `attention` (rotated, all keys), `parallel` (`left`: attention without rotation over
a window that keeps the first tokens; `right`: the gated delta rule; summed with `left_scale` and `right_scale`), `mamba2` (a
state space).  Every size and every constant that can differ between models is read here; the ranks of the delta rule's
low-rank maps are what the checkpoint's tensors have unless `decay_rank` and `gate_rank` state them (random weights need them).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple, Union

from .base import KeyReader, ModelConfig

KAPOSUN_ARCHITECTURE = "Kaposun"


@dataclass(frozen=True)
class RotarySpec:
    base: float
    dims: int
    factor: float = 1.0              # every frequency is divided by it


@dataclass(frozen=True)
class MaskSpec:
    size: int                        # a query sees the last `size` keys, its own included ...
    keep_first: int = 0              # ... and the first this many of the sequence


@dataclass(frozen=True)
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Optional[RotarySpec] = None
    mask: Optional[MaskSpec] = None


@dataclass(frozen=True)
class DeltaSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int
    decay_rank: Optional[int] = None
    gate_rank: Optional[int] = None


@dataclass(frozen=True)
class ParallelSpec:
    left: AttentionSpec
    right: DeltaSpec
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class StateSpaceSpec:
    heads: int
    vdim: int
    state: int
    groups: int
    norm_groups: int
    taps: int


@dataclass(frozen=True)
class LayerSpec:
    type: str
    mixer: Union[AttentionSpec, ParallelSpec, StateSpaceSpec, None]
    ff: Optional[int]                # the feed-forward's inner width; None: the layer has none


@dataclass(frozen=True)
class LoopSpec:
    start: int
    stop: int
    times: int


def _read_heads(m: KeyReader):
    heads, kv_heads = m.integer("heads", minimum=1), m.integer("kv_heads", minimum=1)
    if None not in (heads, kv_heads) and kv_heads >= 1 and heads % kv_heads:
        m.fail(f"heads {heads} is not a multiple of kv_heads {kv_heads}")
    return heads, kv_heads, m.integer("dim", minimum=1), m.integer("vdim", minimum=1)


def _read_attention(m: KeyReader) -> AttentionSpec:
    heads, kv_heads, dim, vdim = _read_heads(m)
    rotary = mask = None
    rot = m.sub("rot", required=False)
    if rot is not None:
        scaling = rot.sub("scaling", required=False)
        factor = scaling.number("factor", positive=True) if scaling is not None else 1.0
        rot.absorb(scaling)
        rotary = RotarySpec(rot.number("base", positive=True), rot.integer("dims", minimum=2), factor)
        if rotary.dims is not None and rotary.dims % 2:
            rot.fail(f"'dims' must be even, got {rotary.dims}")
        if None not in (rotary.dims, dim) and rotary.dims > dim:
            rot.fail(f"dims {rotary.dims} exceeds dim {dim}")
        m.absorb(rot)
    msk = m.sub("mask", required=False)
    if msk is not None:
        mask = MaskSpec(msk.integer("size", minimum=1), msk.integer("keep_first", default=0, minimum=0))
        m.absorb(msk)
    return AttentionSpec(heads, kv_heads, dim, vdim, m.number("scale", positive=True), rotary, mask)


def _read_delta(m: KeyReader) -> DeltaSpec:
    heads, kv_heads, dim, vdim = _read_heads(m)
    return DeltaSpec(heads, kv_heads, dim, vdim, m.integer("conv", minimum=1), m.integer("decay_rank", default=None, minimum=1),
                     m.integer("gate_rank", default=None, minimum=1))


def _read_parallel(m: KeyReader) -> ParallelSpec:
    left, right = m.sub("left"), m.sub("right")
    spec = ParallelSpec(_read_attention(left) if left is not None else None, _read_delta(right) if right is not None else None,
                        m.number("left_scale", default=1.0), m.number("right_scale", default=1.0))
    m.absorb(left)
    m.absorb(right)
    return spec


def _read_state_space(m: KeyReader) -> StateSpaceSpec:
    spec = StateSpaceSpec(m.integer("heads", minimum=1), m.integer("vdim", minimum=1), m.integer("state", minimum=1),
                          m.integer("groups", default=1, minimum=1), m.integer("norm_groups", default=1, minimum=1), m.integer("conv", minimum=1))
    if None not in (spec.heads, spec.groups) and spec.groups >= 1 and spec.heads % spec.groups:
        m.fail(f"heads {spec.heads} is not a multiple of groups {spec.groups}")
    if None not in (spec.heads, spec.vdim, spec.norm_groups) and spec.norm_groups >= 1 and spec.heads * spec.vdim % spec.norm_groups:
        m.fail(f"heads * vdim {spec.heads * spec.vdim} is not a multiple of norm_groups {spec.norm_groups}")
    return spec


_MIXERS = {"attention": _read_attention, "parallel": _read_parallel, "mamba2": _read_state_space}


def _read_layer(lr: KeyReader) -> LayerSpec:
    kind = lr.string("type")
    if kind is not None and kind not in _MIXERS:
        lr.fail(f"unknown mixer type '{kind}' ({', '.join(sorted(_MIXERS))})")
        kind = None
    mixer = None
    m = lr.sub("mixer")
    if m is not None and kind is not None:
        mixer = _MIXERS[kind](m)
        lr.absorb(m)
    ff = None
    mlp = lr.sub("mlp", required=False)
    if mlp is not None:
        what = mlp.string("kind")
        if what is not None and what != "dense":
            mlp.fail(f"unknown feed-forward kind '{what}' (dense)")
        ff = mlp.integer("ff", minimum=1)
        lr.absorb(mlp)
    return LayerSpec(kind, mixer, ff)


@dataclass(frozen=True)
class KaposunConfig(ModelConfig):
    vocab_size: int
    width: int
    norm_eps: float
    residual_mult: float
    layers: Tuple[LayerSpec, ...]
    loop: Optional[LoopSpec] = None
    eos_token_ids: Tuple[int, ...] = ()
    initializer_range: float = 0.05

    @classmethod
    def from_dict(cls, data: Mapping[str, Any], where: str = "config.json") -> "KaposunConfig":
        r = KeyReader(data, where)
        vocab, width = r.integer("vocab", minimum=1), r.integer("width", minimum=1)
        norm = r.sub("norm")
        eps = norm.number("eps", positive=True) if norm is not None else None
        r.absorb(norm)
        gain = r.number("residual_mult", default=1.0)
        raw_layers = data.get("layers")
        layers = []
        if not isinstance(raw_layers, (list, tuple)) or not raw_layers:
            r.fail("'layers' must be a non-empty list")
        else:
            for i, item in enumerate(raw_layers):
                if not isinstance(item, Mapping):
                    r.fail(f"layers[{i}] must be an object")
                    continue
                lr = KeyReader(item, f"{where}: layers[{i}]")
                layers.append(_read_layer(lr))
                r.absorb(lr)
        loop = None
        lp = r.sub("loop", required=False)
        if lp is not None:
            loop = LoopSpec(lp.integer("start", minimum=0), lp.integer("stop", minimum=0), lp.integer("times", minimum=1))
            if None not in (loop.start, loop.stop) and layers and not loop.start < loop.stop <= len(layers):
                lp.fail(f"start {loop.start} and stop {loop.stop} must enclose layers of the {len(layers)}")
            r.absorb(lp)
        eos = r.int_list("eos_token_id", default=())
        init_range = r.number("initializer_range", default=0.05, positive=True)
        r.finish()
        return cls(architecture=KAPOSUN_ARCHITECTURE, vocab_size=vocab, width=width, norm_eps=eps, residual_mult=gain,
                   layers=tuple(layers), loop=loop, eos_token_ids=eos, initializer_range=init_range)

    def layer_order(self) -> Tuple[int, ...]:
        """The layers in the order in which they run, those of the loop once per pass."""
        n = len(self.layers)
        if self.loop is None:
            return tuple(range(n))
        inner = tuple(range(self.loop.start, self.loop.stop))
        return tuple(range(self.loop.start)) + inner * self.loop.times + tuple(range(self.loop.stop, n))

    def to_dict(self) -> Dict[str, Any]:
        def attention(s: AttentionSpec) -> Dict[str, Any]:
            out: Dict[str, Any] = {"heads": s.heads, "kv_heads": s.kv_heads, "dim": s.dim, "vdim": s.vdim, "scale": s.scale}
            if s.rot is not None:
                out["rot"] = {"base": s.rot.base, "dims": s.rot.dims, "scaling": {"factor": s.rot.factor}}
            if s.mask is not None:
                out["mask"] = {"size": s.mask.size, "keep_first": s.mask.keep_first}
            return out

        def mixer(s) -> Dict[str, Any]:
            if isinstance(s, AttentionSpec):
                return attention(s)
            if isinstance(s, StateSpaceSpec):
                return {"heads": s.heads, "vdim": s.vdim, "state": s.state, "groups": s.groups, "norm_groups": s.norm_groups, "conv": s.taps}
            d = s.right
            right: Dict[str, Any] = {"heads": d.heads, "kv_heads": d.kv_heads, "dim": d.dim, "vdim": d.vdim, "conv": d.taps}
            right.update({name: rank for name, rank in (("decay_rank", d.decay_rank), ("gate_rank", d.gate_rank)) if rank is not None})
            return {"left": attention(s.left), "right": right, "left_scale": s.left_scale, "right_scale": s.right_scale}

        out: Dict[str, Any] = {
            "architecture": self.architecture, "vocab": self.vocab_size, "width": self.width, "norm": {"eps": self.norm_eps},
            "residual_mult": self.residual_mult,
            "layers": [{"type": l.type, "mixer": mixer(l.mixer), "mlp": None if l.ff is None else {"kind": "dense", "ff": l.ff}}
                       for l in self.layers],
            "initializer_range": self.initializer_range,
        }
        if self.loop is not None:
            out["loop"] = {"start": self.loop.start, "stop": self.loop.stop, "times": self.loop.times}
        if len(self.eos_token_ids) == 1:
            out["eos_token_id"] = self.eos_token_ids[0]
        elif len(self.eos_token_ids) > 1:
            out["eos_token_id"] = list(self.eos_token_ids)
        return out
