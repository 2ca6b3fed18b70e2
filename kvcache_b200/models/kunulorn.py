"""The Kunulorn decoder put together from parts, layer by layer, from its configuration.

Tensor names: `embed` (also the output matrix), `final.norm`, and per layer i `l<i>.norm1`, `l<i>.norm2`, `l<i>.mix.*` (`q`,
`k`, `v`, `o`, their biases `<name>.b`, the norms `q.norm` and `k.norm`), `l<i>.mlp.*` (dense: `gate`, `up`, `down`; routed:
`router`, `correction`, experts `e<j>.`, `shared.` with its gate `shared.sg`).  A layer is x += mixer(norm1(x)); x +=
ff(norm2(x)), the norms taking the mean off before they divide.  The mixer is grouped-key attention over the query's own
chunk of the sequence; with `kv_from` a layer reads the cache entry of an earlier layer instead of projecting keys and
values.
"""
from __future__ import annotations

from typing import Dict, Optional

from ..config.kunulorn import KUNULORN_ARCHITECTURE, DenseSpec, KunulornConfig, RotarySpec
from ..config.registry import register_architecture
from ..parts.attention import GQAAttention
from ..parts.block import PreNormBlock
from ..parts.feedforward import GatedMLP, RoutedMLP
from ..parts.model import DecoderModel, LayerCall
from ..parts.norm import LayerNorm
from ..parts.position import RotaryHalf

# Until the engine tells how long a request may get (it always does), rotation tables are made for this many positions.
DEFAULT_POSITIONS = 4096


def build_kunulorn(config: KunulornConfig, dtype: str = "bfloat16", device: str = "cuda:0",
                   max_positions: Optional[int] = None) -> DecoderModel:
    c = config
    positions = max_positions or DEFAULT_POSITIONS
    rotations: Dict[tuple, RotaryHalf] = {}          # layers with equal rotation constants share one table

    def rotation(spec: Optional[RotarySpec]) -> Optional[RotaryHalf]:
        if spec is None:
            return None
        key = (spec.dims, spec.base)
        if key not in rotations:
            rotations[key] = RotaryHalf(spec.dims, spec.base, positions)
        return rotations[key]

    def feed_forward(m, p: str):
        names = ("gate", "up", "down")
        if isinstance(m, DenseSpec):
            return GatedMLP(c.width, m.ff, activation="clamped_swiglu", limit=m.limit, prefix=p, dtype=dtype, names=names)
        shared = None
        if m.shared_ff is not None:
            shared = GatedMLP(c.width, m.shared_ff, activation="silu", prefix=p + "shared.", dtype=dtype, names=names)
        return RoutedMLP(c.width, m.expert_ff, m.experts, m.top, activation="swiglu", scores="sigmoid", prefix=p, dtype=dtype,
                         shared=shared, shared_gate="shared.sg" if shared is not None else None, correction="correction",
                         groups=None if m.groups is None else (m.groups.count, m.groups.keep), weight_scale=m.weight_scale)

    blocks, schedule, cache_of = [], [], {}
    for i, layer in enumerate(c.layers):
        p, a = f"l{i}.", layer.mixer
        mixer = GQAAttention(c.width, a.heads, a.kv_heads, a.dim, qkv_bias=True, out_bias=True, position=rotation(a.rot), window=None,
                             chunk=a.chunk, prefix=p + "mix.", dtype=dtype, scale=a.scale, value_dim=a.vdim, names=("q", "k", "v", "o"),
                             qk_norm_eps=c.norm_eps, qk_norm_scope="all", rotary_layout="interleaved", pad_values=True,
                             own_kv=a.kv_from is None)
        ffn = norm2 = None
        if layer.mlp is not None:
            ffn, norm2 = feed_forward(layer.mlp, p + "mlp."), LayerNorm(c.width, c.norm_eps, p + "norm2")
        blocks.append(PreNormBlock(c.width, LayerNorm(c.width, c.norm_eps, p + "norm1"), mixer, norm2, ffn, dtype))
        # A layer that reads another's keys and values has no cache entry of its own: its call reads the other's, which then
        # keeps what any of its readers sees.
        if a.kv_from is None:
            cache_of[i] = len(cache_of)
            schedule.append(LayerCall(i, cache_of[i]))
        else:
            blocks[a.kv_from].mixer.keep_for(mixer)
            schedule.append(LayerCall(i, cache_of[a.kv_from], writes_cache=False))
    # A checkpoint may carry the second norm of a layer that has no feed-forward: it is left alone.
    unused = [f"l{i}.norm2" for i, layer in enumerate(c.layers) if layer.mlp is None]
    return DecoderModel(config=c, dtype=dtype, vocab_size=c.vocab_size, width=c.width, embed_name="embed", head_name=None,
                        blocks=blocks, schedule=schedule, final_norm=LayerNorm(c.width, c.norm_eps, "final.norm"), position=None,
                        ignorable_tensors=unused, embed_scale=c.embed_scale)


register_architecture(KUNULORN_ARCHITECTURE, KunulornConfig, build_kunulorn, replace=True)
