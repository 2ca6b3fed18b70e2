"""The Kaposun model in the engine (step function, cache manager, scheduler) on the CPU stand-in kernels against the plain
implementation; its parts alone against the plain functions; its configuration."""
import copy

import pytest
import torch

import plain_kaposun as plain
import replay_modes
from helpers import assert_close, make_runner, paged_scenario, random_tokens
from kaposun_configs import CONFIGS, PAGE_SIZE, config_dict, enliven, make_kaposun_folder
from torch_kernels import TorchKernels

REL = 1e-4


def _runner(tmp_path, name, num_pages=64, sharpen=1.0, **kw):
    folder = make_kaposun_folder(tmp_path, name, sharpen=sharpen)
    runner = make_runner(folder, TorchKernels(), dtype="float32", device="cpu", page_size=PAGE_SIZE[name], num_pages=num_pages, **kw)
    config, weights = plain.read_folder(folder)
    return runner, config, weights


# ---- configuration --------------------------------------------------------------------------------------------------
def test_config_round_trip():
    from kvcache_b200.config import config_from_dict
    for name in CONFIGS:
        c = config_from_dict(config_dict(name))
        assert config_from_dict(c.to_dict()) == c
    a = config_from_dict(config_dict("A"))
    left, right = a.layers[0].mixer.left, a.layers[0].mixer.right
    assert (left.heads, left.kv_heads, left.dim, left.vdim, left.scale, left.rot, left.mask.size, left.mask.keep_first) == (4, 2, 12, 20, 0.3, None, 11, 3)
    assert (right.heads, right.kv_heads, right.dim, right.vdim, right.taps, right.decay_rank, right.gate_rank) == (4, 2, 10, 14, 4, 6, 9)
    assert (a.layers[0].mixer.left_scale, a.layers[0].mixer.right_scale, a.layers[0].ff) == (0.7, 1.4, 56)
    rot, space = a.layers[1].mixer.rot, a.layers[2].mixer
    assert (rot.base, rot.dims, rot.factor) == (5000.0, 6, 3.0)
    assert (space.heads, space.vdim, space.state, space.groups, space.norm_groups, space.taps) == (6, 8, 10, 3, 2, 3)
    assert a.residual_mult == 0.6 and a.layer_order() == (0, 1, 0, 1, 2)
    b = config_from_dict(config_dict("B"))
    assert b.loop is None and b.layer_order() == (0, 1, 2) and b.layers[2].mixer.rot.factor == 1.0 and b.layers[1].ff is None
    assert config_from_dict(config_dict("C")).layer_order() == (0, 1, 2, 1, 2, 1, 2)
    assert config_from_dict(config_dict("D")).layers[0].mixer.left.mask is None
    bare = config_dict("B")
    for key in ("decay_rank", "gate_rank"):
        del bare["layers"][1]["mixer"]["right"][key]
    assert config_from_dict(bare).layers[1].mixer.right.decay_rank is None


def test_config_faults_are_all_reported():
    from kvcache_b200.config import ConfigError, config_from_dict
    bad = config_dict("A")
    bad["layers"][0]["mixer"]["left"].pop("vdim")
    bad["layers"][0]["mixer"]["left"]["mask"]["size"] = 0
    bad["layers"][0]["mixer"]["right"]["kv_heads"] = 3
    bad["layers"][1]["mixer"]["rot"]["dims"] = 12
    bad["layers"][1]["mlp"]["kind"] = "sparse"
    bad["layers"][2]["mixer"]["groups"] = 4
    bad["layers"][2]["mixer"]["norm_groups"] = 5
    bad["loop"]["stop"] = 4
    bad["layers"].append({"type": "convolution", "mixer": {}, "mlp": None})
    bad["layers"].append({"type": "mamba2", "mlp": None})
    bad["loop"]["stop"] = 9
    del bad["norm"]
    with pytest.raises(ConfigError) as info:
        config_from_dict(bad)
    text = str(info.value)
    for piece in ("vdim", "'size' must be >= 1", "heads 4 is not a multiple of kv_heads 3", "dims 12 exceeds dim 10", "sparse",
                  "heads 6 is not a multiple of groups 4", "not a multiple of norm_groups 5", "stop 9", "convolution", "missing key 'mixer'", "norm"):
        assert piece in text, piece


def test_model_as_data(tmp_path):
    """Every pass of a loop has an entry of its own; an entry holds pages, states or both; the last products are one matrix."""
    from kvcache_b200.engine.loading import load_model
    model = load_model(make_kaposun_folder(tmp_path, "A"), "float32", "cpu", max_positions=64)
    assert [(c.layer, c.cache, c.writes_cache) for c in model.schedule] == [(0, 0, True), (1, 1, True), (0, 2, True), (1, 3, True), (2, 4, True)]
    entries = model.cache_entries()
    kv = entries[2].kv
    assert (kv.num_kv_heads, kv.head_dim, kv.v_head_dim, kv.window, kv.keep_first) == (2, 12, 20, 11, 3)
    assert {k: s.shape for k, s in entries[0].state.items()} == {"right.memory": (4, 10, 14), "right.conv": (3, 2 * 2 * 10 + 4 * 14)}
    assert entries[1].state is None and entries[1].kv.window is None
    assert entries[4].kv is None and {k: s.shape for k, s in entries[4].state.items()} == {"memory": (6, 10, 8), "conv": (2, 48 + 60)}
    assert all(s.dtype == "float32" for e in entries if e.state for s in e.state.values())
    assert model.tied and model.blocks[0].w_out.shape == (72, 4 * 20 + 4 * 14 + 56)
    assert model.blocks[0].mixer.w_o is None and model.blocks[0].ffn.w_down is None, "the matrices are not kept twice"
    b = load_model(make_kaposun_folder(tmp_path, "B"), "float32", "cpu", max_positions=64)
    assert b.blocks[0].gain is None and b.blocks[1].ffn is None and b.cache_entries()[0].state["conv"].shape == (0, 3 * 20 + 14)
    e = load_model(make_kaposun_folder(tmp_path, "E"), "bfloat16", "cpu", max_positions=64)
    assert [(x.kv.head_dim, x.kv.v_head_dim) for x in e.cache_entries() if x.kv] == [(64, 64)] * 4


def test_low_rank_sizes_come_from_the_checkpoint(tmp_path):
    from kvcache_b200.engine.loading import load_model
    import json, os
    folder = make_kaposun_folder(tmp_path, "B")
    data = config_dict("B")
    for key in ("decay_rank", "gate_rank"):
        del data["layers"][1]["mixer"]["right"][key]
    with open(os.path.join(folder, "config.json"), "w") as fh:
        json.dump(data, fh)
    right = load_model(folder, "float32", "cpu", max_positions=64).blocks[1].mixer.right
    assert right.decay_rank is None and right.w_low.shape == (32, 96) and right.w_high.shape == (3 * 12 + 3 * 12, 32)


# ---- mechanisms alone ---------------------------------------------------------------------------------------------------
def _context(batch=None, kv=None, state=None):
    from kvcache_b200.engine.workspace import Workspace
    from kvcache_b200.parts.base import LayerContext
    return LayerContext(batch=batch, kernels=TorchKernels(wide=True), workspace=Workspace("cpu"), kv=kv, state=state)


def _weights(specs, seed, std=0.3):
    g = torch.Generator().manual_seed(seed)
    w = {name: (torch.randn(spec.shape, generator=g) * std + (1.0 if name.endswith("norm") else 0.0)).to(torch.bfloat16)
         for name, spec in specs.items()}
    return enliven(w, seed)


def _scenario(segments, spec=None, page_size=4, slots=None):
    from kvcache_b200.parts.base import PagedKVView
    heads, dim = (1, 4) if spec is None else (spec.num_kv_heads, spec.head_dim)
    batch, kv = paged_scenario(segments, num_kv_heads=heads, head_dim=dim, page_size=page_size, dtype=torch.float32, device="cpu", fill_history=False)
    if slots is not None:
        batch.seg_slot.copy_(torch.tensor(slots, dtype=torch.int32))
    if spec is None:
        return batch, None
    return batch, PagedKVView(spec=spec, k_pages=kv.k_pages, v_pages=torch.zeros(*kv.k_pages.shape[:-1], spec.v_head_dim),
                              block_table=kv.block_table, page_size=page_size, writes=True)


def _states(part, slots=3, fill=0.0):
    spec = part.state_spec()
    return {name: torch.full((slots, *s.shape), fill) for name, s in spec.items()} if isinstance(spec, dict) else spec


def _attention_part(W, m, gate=None, prefix="m.", eps=1e-5, positions=512):
    from kvcache_b200.parts.attention import GQAAttention
    from kvcache_b200.parts.position import LinearScaling, RotaryHalf
    rot, mask = m.get("rot"), m.get("mask") or {}
    position = None
    if rot is not None:
        position = RotaryHalf(rot["dims"], rot["base"], positions, LinearScaling(rot["scaling"]["factor"]) if rot.get("scaling") else None)
    return GQAAttention(W, m["heads"], m["kv_heads"], m["dim"], qkv_bias=False, out_bias=False, position=position, window=mask.get("size"),
                        keep_first=mask.get("keep_first", 0), prefix=prefix, dtype="float32", scale=m["scale"], value_dim=m["vdim"],
                        names=("q", "k", "v", "o"), qk_norm_eps=eps, qk_norm_scope="all", head_gate=gate, head_gate_scope="channel", pad_values=True)


def test_linear_scaling_divides_every_frequency():
    from kvcache_b200.parts.position import LinearScaling, RotaryHalf
    import numpy as np
    plain_rope, slow = RotaryHalf(10, 700.0, 64), RotaryHalf(10, 700.0, 64, LinearScaling(5.0))
    assert np.allclose(slow.frequencies() * 5.0, plain_rope.frequencies()) and LinearScaling(5.0).gain() == 1.0
    slow.bind({}, torch.device("cpu"))
    x = torch.randn(64, 1, 12, dtype=torch.float64, generator=torch.Generator().manual_seed(1))
    want = plain.rotate_halves(x, torch.arange(64), {"dims": 10, "base": 700.0, "scaling": {"factor": 5.0}})
    c, s = slow.rotation().cos.double()[:, None], slow.rotation().sin.double()[:, None]
    u, v = x[..., :5], x[..., 5:10]
    assert_close(torch.cat([u * c - v * s, v * c + u * s, x[..., 10:]], dim=-1), want, 1e-6)


SIZES = [dict(heads=4, kv_heads=2, dim=12, vdim=20, scale=1.0, rot={"base": 777.0, "dims": 8, "scaling": {"factor": 2.5}}),
         dict(heads=3, kv_heads=1, dim=8, vdim=4, scale=2.0, mask={"size": 6, "keep_first": 2}),
         dict(heads=2, kv_heads=2, dim=6, vdim=6, scale=2.0, mask={"size": 1, "keep_first": 1}),
         dict(heads=6, kv_heads=3, dim=10, vdim=3, scale=1.5, mask={"size": 4, "keep_first": 9}),
         dict(heads=5, kv_heads=5, dim=10, vdim=3, scale=1.5, rot={"base": 1000.0, "dims": 10})]


@pytest.mark.parametrize("m", SIZES)
@pytest.mark.parametrize("gated", [False, True])
def test_attention_part_alone(m, gated):
    """Sharp scores, whole and cut in three: norms over whole projections, the window's edge and the kept tokens' edge, a gate for
    every number of the heads' results."""
    T, W, eps = 29, 40, 1e-5
    part = _attention_part(W, m, "g" if gated else None)
    w = _weights(part.tensor_specs(), 3)
    part.bind(w, torch.device("cpu"))
    x = torch.randn(T, W, generator=torch.Generator().manual_seed(4))
    wd = {k: v.double() for k, v in w.items()}
    forward = plain.gated_attention if gated else plain.attention
    run = lambda mm, ww: forward(mm, ww, "m.", x.double(), torch.arange(T), eps)
    want = run(m, wd)
    for key in ("size", "keep_first"):                # one key more or one key less would show
        for delta in (-1, 1):
            if m.get("mask") and m["mask"][key] + delta >= (1 if key == "size" else 0):
                other = dict(m, mask=dict(m["mask"], **{key: m["mask"][key] + delta}))
                assert (run(other, wd) - want).abs().max() > 0.02 * want.abs().max(), (key, delta)
    for name in [n for n in w if n.endswith("norm")] + (["m.g"] if gated else []):
        assert (run(m, dict(wd, **{name: torch.ones_like(wd[name])})) - want).abs().max() > 0.01 * want.abs().max(), name
    if gated:
        assert w["m.g"].shape == (m["heads"] * m["vdim"], W)
    _, kv = _scenario([(0, T)], part.cache_spec())
    got, at = [], 0
    for n in (11, 2, 16):
        batch, _ = _scenario([(at, n)], part.cache_spec())
        got.append(part.forward(x[at:at + n], _context(batch, kv)))
        at += n
    assert_close(torch.cat(got), want, 1e-5)
