"""The Kaposun decoder put together from parts, layer by layer, from its configuration.

Tensor names: `embed` (also the output matrix), `final.norm`, and per layer i `l<i>.norm1`, `l<i>.mix.*` (the mixer; the two
sides of a parallel mixer under `left.` and `right.`), `l<i>.mlp.up` / `.down`.  A layer is one norm whose rows both sublayers
read, x += m (mixer(h) + ff(h)), with m the configuration's residual multiplier.  The layers of `loop` run `times` times in a
row with the same weights, each pass with a cache entry of its own per layer.  Mixers: `attention` - queries and keys normalised
over their whole projections, then rotated (frequencies divided by a factor); `parallel` - attention without rotation over a
window that keeps the first tokens, with a gate per channel, beside the gated delta rule; `mamba2` - a state space.
"""
from __future__ import annotations

from typing import Dict, Optional

from ..config.kaposun import KAPOSUN_ARCHITECTURE, AttentionSpec, KaposunConfig, RotarySpec, StateSpaceSpec
from ..config.registry import register_architecture
from ..parts.attention import GQAAttention
from ..parts.block import ParallelBlock
from ..parts.feedforward import PlainMLP
from ..parts.model import DecoderModel, LayerCall
from ..parts.norm import RMSNorm
from ..parts.position import LinearScaling, RotaryHalf
from ..parts.recurrent import GatedDeltaMixer, ParallelMixer, StateSpaceMixer

# Until the engine tells how long a request may get (it always does), rotation tables are made for this many positions.
DEFAULT_POSITIONS = 4096


def build_kaposun(config: KaposunConfig, dtype: str = "bfloat16", device: str = "cuda:0",
                  max_positions: Optional[int] = None) -> DecoderModel:
    c = config
    positions = max_positions or DEFAULT_POSITIONS
    rotations: Dict[RotarySpec, RotaryHalf] = {}     # layers with equal rotation constants share one table

    def rotation(spec: Optional[RotarySpec]) -> Optional[RotaryHalf]:
        if spec is None:
            return None
        if spec not in rotations:
            rotations[spec] = RotaryHalf(spec.dims, spec.base, positions, None if spec.factor == 1.0 else LinearScaling(spec.factor))
        return rotations[spec]

    def attention(a: AttentionSpec, p: str, gate: Optional[str]) -> GQAAttention:
        return GQAAttention(c.width, a.heads, a.kv_heads, a.dim, qkv_bias=False, out_bias=False, position=rotation(a.rot),
                            window=None if a.mask is None else a.mask.size, keep_first=0 if a.mask is None else a.mask.keep_first,
                            prefix=p, dtype=dtype, scale=a.scale, value_dim=a.vdim, names=("q", "k", "v", "o"), qk_norm_eps=c.norm_eps,
                            qk_norm_scope="all", head_gate=gate, head_gate_scope="channel", pad_values=True)

    def mixer(spec, p: str):
        if isinstance(spec, AttentionSpec):
            return attention(spec, p, None)
        if isinstance(spec, StateSpaceSpec):
            return StateSpaceMixer(c.width, spec.heads, spec.vdim, spec.state, spec.groups, spec.norm_groups, spec.taps, eps=c.norm_eps,
                                   prefix=p, dtype=dtype)
        d = spec.right
        right = GatedDeltaMixer(c.width, d.heads, d.kv_heads, d.dim, d.vdim, d.taps, eps=c.norm_eps, prefix=p + "right.", dtype=dtype,
                                decay_rank=d.decay_rank, gate_rank=d.gate_rank)
        return ParallelMixer(c.width, attention(spec.left, p + "left.", "g"), right, spec.left_scale, spec.right_scale, dtype)

    blocks = []
    for i, layer in enumerate(c.layers):
        p = f"l{i}."
        ffn = None if layer.ff is None else PlainMLP(c.width, layer.ff, activation="gelu", prefix=p + "mlp.", dtype=dtype)
        blocks.append(ParallelBlock(c.width, RMSNorm(c.width, c.norm_eps, p + "norm1"), mixer(layer.mixer, p + "mix."), ffn, dtype,
                                    gain=c.residual_mult))
    schedule = [LayerCall(i, run) for run, i in enumerate(c.layer_order())]
    return DecoderModel(config=c, dtype=dtype, vocab_size=c.vocab_size, width=c.width, embed_name="embed", head_name=None,
                        blocks=blocks, schedule=schedule, final_norm=RMSNorm(c.width, c.norm_eps, "final.norm"), position=None)


register_architecture(KAPOSUN_ARCHITECTURE, KaposunConfig, build_kaposun, replace=True)
