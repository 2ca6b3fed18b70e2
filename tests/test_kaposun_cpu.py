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


def _edge_case(part, W, T, at, strength=40.0, seed=3):
    """Weights and inputs of an attention part in which every query scores the key of row `at` far above all others: channel 0
    of the input is 1 in that row only and drives the keys along one direction, channel 1 is 1 in every row and drives the
    queries along the same direction; channel 2 drives all other rows' keys along another (keys are normalised, and small random
    ones would point anywhere)."""
    g = torch.Generator().manual_seed(seed)
    w = {name: (torch.randn(spec.shape, generator=g) * 0.05 + (1.0 if name.endswith("norm") else 0.0)).to(torch.bfloat16)
         for name, spec in part.tensor_specs().items()}
    D = part.head_dim
    q, k = w["m.q"].float(), w["m.k"].float()
    q[:, :3], k[:, :3] = 0.0, 0.0
    q[torch.arange(part.num_heads) * D, 1] = strength
    k[torch.arange(part.num_kv_heads) * D, 0] = strength
    k[torch.arange(part.num_kv_heads) * D + 1, 2] = strength
    w["m.q"], w["m.k"] = q.to(torch.bfloat16), k.to(torch.bfloat16)
    x = torch.randn(T, W, generator=g) * 0.1
    x[:, 0], x[:, 1], x[:, 2] = 0.0, 1.0, 1.0
    x[at, 0], x[at, 2] = 1.0, 0.0
    return w, x


@pytest.mark.parametrize("at,mask,taken", [(0, None, True), (150, (90, 6), True), (149, (90, 6), False), (5, (90, 6), True), (6, (90, 6), False),
                                            (15, (20, 16), True), (16, (20, 16), False)])
def test_one_key_far_away_takes_all_the_weight_or_none(at, mask, taken):
    """Random weights would hide a lost key among hundreds.  Row 239 sees keys 150 .. 239 of a window of 90 and the kept ones."""
    T, W = 240, 24
    m = dict(heads=4, kv_heads=2, dim=8, vdim=6, scale=40.0)
    if mask:
        m["mask"] = {"size": mask[0], "keep_first": mask[1]}
    part = _attention_part(W, m)
    w, x = _edge_case(part, W, T, at)
    part.bind(w, torch.device("cpu"))
    wd = {k: v.double() for k, v in w.items()}
    want = plain.attention(m, wd, "m.", x.double(), torch.arange(T), 1e-5)
    value = (x[at].double() @ wd["m.v"].t()).view(2, 6).repeat_interleave(2, dim=0).reshape(1, -1) @ wd["m.o"].t()
    assert bool((want[239] - value).abs().max() < 1e-3 * want.abs().max()) == taken
    _, kv = _scenario([(0, T)], part.cache_spec(), page_size=16)
    got, start = [], 0
    for n in [131, 2, 67, 32] + [1] * 8:
        batch, _ = _scenario([(start, n)], part.cache_spec(), page_size=16)
        got.append(part.forward(x[start:start + n], _context(batch, kv)))
        start += n
    assert_close(torch.cat(got), want, 1e-5)


# The recurrent mixers: (part, plain function of (weights, rows)).
def _delta_part(W, H, G, D, V, taps, ranks=(6, 5), eps=1e-5):
    from kvcache_b200.parts.recurrent import GatedDeltaMixer
    m = {"heads": H, "kv_heads": G, "dim": D, "vdim": V, "conv": taps}
    part = GatedDeltaMixer(W, H, G, D, V, taps, eps=eps, prefix="m.", dtype="float32", decay_rank=ranks[0], gate_rank=ranks[1])
    return part, lambda w, x: plain.gated_delta(m, w, "m.", x, eps)


def _space_part(W, H, V, N, G, parts, taps, eps=1e-5):
    from kvcache_b200.parts.recurrent import StateSpaceMixer
    m = {"heads": H, "vdim": V, "state": N, "groups": G, "norm_groups": parts, "conv": taps}
    part = StateSpaceMixer(W, H, V, N, G, parts, taps, eps=eps, prefix="m.", dtype="float32")
    return part, lambda w, x: plain.mamba2(m, w, "m.", x, eps)


RECURRENT = {"delta": lambda W: _delta_part(W, 4, 2, 6, 10, 4), "delta, one tap": lambda W: _delta_part(W, 3, 3, 8, 8, 1),
             "delta, long convolution": lambda W: _delta_part(W, 6, 1, 5, 3, 6, (9, 33)), "space": lambda W: _space_part(W, 4, 6, 5, 2, 3, 4),
             "space, one tap": lambda W: _space_part(W, 3, 8, 9, 1, 1, 1), "space, a group a head": lambda W: _space_part(W, 5, 4, 7, 5, 10, 2)}


@pytest.mark.parametrize("which", list(RECURRENT))
def test_recurrent_mixer_alone_in_portions_and_beside_others(which):
    """Whole; one token at a time; portions shorter than the convolution; two requests beside one another in slots whose order is
    not the segments'; a slot that another request held, zeroed as at admission."""
    W, T = 20, 31
    part, reference = RECURRENT[which](W)
    w = _weights(part.tensor_specs(), 5)
    part.bind(w, torch.device("cpu"))
    wd = {k: v.double() for k, v in w.items()}
    x, other = (torch.randn(T, W, generator=torch.Generator().manual_seed(s)) for s in (6, 7))
    want, want_other = reference(wd, x.double()), reference(wd, other.double())
    for name in wd:                                   # every tensor matters
        assert (reference(dict(wd, **{name: wd[name] * 0.5 + 0.3}), x.double()) - want).abs().max() > 1e-3 * want.abs().max(), name
    state = _states(part)

    def run(pieces):
        batch, _ = _scenario([(start, len(rows)) for start, rows, _ in pieces], slots=[slot for _, _, slot in pieces])
        return part.forward(torch.cat([rows for _, rows, _ in pieces]), _context(batch, state=state)).clone()
    assert_close(run([(0, x, 1)]), want, 1e-5, "whole")
    for sizes in ([1] * T, [2, 1, 1, 3, 2, 5, 17]):
        for s in state.values():
            s[1].zero_()
        got, at = [], 0
        for n in sizes:
            got.append(run([(at, x[at:at + n], 1)]))
            at += n
        assert_close(torch.cat(got), want, 1e-5, f"portions {sizes[:3]}")
    for s in state.values():
        s.zero_()
        s[1].fill_(7.0)                               # nobody's: must stay
    first = run([(0, x[:9], 2), (0, other[:1], 0)])
    second = run([(1, other[1:3], 0), (9, x[9:10], 2)])
    third = run([(10, x[10:], 2), (3, other[3:], 0)])
    assert_close(torch.cat([first[:9], second[2:], third[:21]]), want, 1e-5, "beside another request")
    assert_close(torch.cat([first[9:], second[:2], third[21:]]), want_other, 1e-5, "the other request")
    assert all(bool((s[1] == 7.0).all()) for s in state.values())


def test_gated_delta_reads_after_the_decay_and_before_its_own_write():
    """No convolution, one head, key and query the first unit vector: with write strength b and decay a the state along that key
    goes s -> a s + b (v - a s), and the read-out sees it; reading the undecayed state, or before the write, differs."""
    k = TorchKernels(wide=True)
    batch, _ = _scenario([(0, 3)], slots=[0])
    D = Dv = 2
    rows = torch.tensor([[1.0, 0.0, 1.0, 0.0, 5.0, 1.0]] * 3)
    gates = torch.tensor([[0.5, 0.9, 0.25]] * 3)
    memory, out = torch.zeros(1, 1, D, Dv), torch.zeros(3, Dv)
    k.gated_delta_scan(rows, gates, 1.0, batch, memory, out, 1, 1, D, Dv)
    s, want = 0.0, []
    for _ in range(3):
        s = 0.5 * s + 0.25 * (5.0 - 0.5 * s)
        want.append(s)
    assert_close(out[:, 0], torch.tensor(want), 1e-6)


def test_parallel_mixer_in_the_layers_own_product():
    """Two sides with their scales, alone and as part of the layer's one product with the feed-forward; the residual multiplier;
    a layer without feed-forward."""
    from kvcache_b200.parts.base import ScaledDelta
    from kvcache_b200.parts.block import ParallelBlock
    from kvcache_b200.parts.feedforward import PlainMLP
    from kvcache_b200.parts.norm import RMSNorm
    from kvcache_b200.parts.recurrent import ParallelMixer
    T, W, eps = 21, 20, 1e-5
    left = dict(heads=4, kv_heads=2, dim=6, vdim=3, scale=1.1, mask={"size": 5, "keep_first": 2})
    right = {"heads": 2, "kv_heads": 1, "dim": 5, "vdim": 7, "conv": 3}
    m = {"left": left, "right": right, "left_scale": 0.7, "right_scale": 1.6}

    def make():
        from kvcache_b200.parts.recurrent import GatedDeltaMixer
        d = GatedDeltaMixer(W, 2, 1, 5, 7, 3, eps=eps, prefix="l0.mix.right.", dtype="float32", decay_rank=4, gate_rank=3)
        return ParallelMixer(W, _attention_part(W, left, "g", prefix="l0.mix.left."), d, 0.7, 1.6, "float32")
    mlp = PlainMLP(W, 13, activation="gelu", prefix="l0.mlp.", dtype="float32")
    blocks = [ParallelBlock(W, RMSNorm(W, eps, "l0.norm1"), make(), ffn, "float32", gain=0.4) for ffn in (mlp, None)]
    w = _weights(blocks[0].tensor_specs(), 8)
    wd = {k: v.double() for k, v in w.items()}
    x = torch.randn(T, W, generator=torch.Generator().manual_seed(9))
    mixer = make()
    mixer.bind(w, torch.device("cpu"))
    batch, kv = _scenario([(0, T)], mixer.cache_spec(), slots=[1])
    want = plain.mixer_forward("parallel", m, wd, "l0.mix.", x.double(), torch.arange(T), eps)
    assert_close(mixer.forward(x, _context(batch, kv, _states(mixer))), want, 1e-5, "the mixer alone")
    for block, ff in zip(blocks, ({"kind": "dense"}, None)):
        block.bind(w, torch.device("cpu"))
        config = {"layers": [{"type": "parallel", "mixer": m, "mlp": ff}], "norm": {"eps": eps}, "residual_mult": 0.4}
        _, kv = _scenario([(0, T)], mixer.cache_spec(), slots=[1])
        delta = block.forward(x.clone(), None, _context(batch, kv, _states(mixer)))
        assert isinstance(delta, ScaledDelta)
        assert_close(x.double() + delta.delta.double() * delta.scale.double(), plain.layer_forward(config, wd, 0, x.double(), torch.arange(T)), 1e-5)
        assert block.weight_bytes() > 0
    with pytest.raises(ValueError):
        ParallelBlock(W, RMSNorm(W, eps, "n"), make(), object(), "float32")


def test_exact_gelu_feed_forward():
    from kvcache_b200.parts.feedforward import PlainMLP
    T, W, F = 9, 20, 24
    part = PlainMLP(W, F, activation="gelu", prefix="f.", dtype="float32")
    w = _weights(part.tensor_specs(), 5, std=0.6)
    part.bind(w, torch.device("cpu"))
    x = torch.randn(T, W, generator=torch.Generator().manual_seed(6))
    wd = {k: v.double() for k, v in w.items()}
    want = plain.feed_forward(wd, "f.", x.double())
    assert_close(part.forward(x, _context()), want, 1e-6)
    z = x.double() @ wd["f.up"].t()
    tanh_form = 0.5 * z * (1 + torch.tanh((2 / torch.pi) ** 0.5 * (z + 0.044715 * z ** 3)))
    assert (tanh_form @ wd["f.down"].t() - want).abs().max() > 20 * 1e-6 * want.abs().max(), "the other gelu differs by more"
    wide = torch.full((T, F + 7), 3.0)
    part.forward_hidden(x, _context(), wide, 5)
    assert_close(wide[:, 5:5 + F], plain.exact_gelu(z), 1e-6)
    assert bool((wide[:, :5] == 3.0).all()) and bool((wide[:, 5 + F:] == 3.0).all())


def test_residual_stream_after_every_layer_run(tmp_path):
    """Run by run, the passes of the loop among them: a model cut after k layer runs (its final norm with weight 1, its head the
    identity) gives the plain implementation's residual stream after run k, divided by its root mean square."""
    from kvcache_b200.cache import CacheManager
    from kvcache_b200.engine.loading import load_model
    from kvcache_b200.engine.runner import ModelRunner, StepEntry
    folder = make_kaposun_folder(tmp_path, "A")
    config, weights = plain.read_folder(folder)
    tokens = random_tokens(config["vocab"], 37, 3)
    streams = []
    plain.forward(config, weights, tokens, streams)
    assert len(streams) == 5
    for k in range(1, len(streams) + 1):
        model = load_model(folder, "float32", "cpu", max_positions=64)
        model.schedule = model.schedule[:k]
        model._writers = {c.cache: c.layer for c in model.schedule}
        model.final_norm.weight, model.final_norm.eps = torch.ones(model.width), 0.0
        model.head, model.vocab_size = torch.eye(model.width), model.width
        cache = CacheManager(model.cache_entries(), page_size=8, num_pages=16, max_slots=1, max_tokens_per_request=64, dtype="float32", device="cpu")
        runner = ModelRunner(model, cache, TorchKernels(wide=True), max_tokens_per_step=64)
        got = runner.step([StepEntry(cache.admit(), tokens, list(range(len(tokens))))])
        assert_close(got, plain.rms_norm(streams[k - 1], torch.ones(model.width, dtype=torch.float64), 0.0), 1e-5, f"after run {k}")


# ---- the model in the engine ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_and_its_first_tokens(tmp_path, name):
    runner, config, weights = _runner(tmp_path, name)
    tokens = random_tokens(config["vocab"], 75, 1)
    want = plain.forward(config, weights, tokens)
    assert_close(replay_modes.whole(runner, tokens), want, REL)
    assert runner.cache.used_pages() == 0
    for n in (1, 2, 3):
        assert_close(replay_modes.whole(runner, tokens[:n]), want[:n], REL, f"first {n}")


@pytest.mark.parametrize("name", list(CONFIGS))
def test_prefill_against_token_by_token_decoding(tmp_path, name):
    runner, config, weights = _runner(tmp_path, name)
    tokens = random_tokens(config["vocab"], 60, 2)
    want = plain.forward(config, weights, tokens)
    assert_close(replay_modes.last_32_one_by_one(runner, tokens), want[-33:], REL)
    assert_close(replay_modes.portions(runner, tokens, [1] * 60), want, REL, "every token alone")


@pytest.mark.parametrize("name", list(CONFIGS))
def test_portions_down_to_two_tokens(tmp_path, name):
    runner, config, weights = _runner(tmp_path, name)
    tokens = random_tokens(config["vocab"], 101, 3)
    want = plain.forward(config, weights, tokens)
    assert_close(replay_modes.portions(runner, tokens, [2, 17, 3, 31, 2, 16, 8, 22]), want, REL)
    assert_close(replay_modes.portions(runner, tokens, [40, 2, 2, 5, 52]), want, REL)


@pytest.mark.parametrize("name", list(CONFIGS))
def test_mixed_batches_with_pages_and_slots_used_again(tmp_path, name):
    """Unequal requests beside one another against each alone; a and b end and d and e take their pages and slots, which hold
    other requests' keys, states and convolution inputs."""
    runner, config, weights = _runner(tmp_path, name, num_pages=replay_modes.mixed_pool_tokens() // PAGE_SIZE[name])
    seqs = {k: random_tokens(config["vocab"], n, 10 + i) for i, (k, n) in enumerate(replay_modes.MIXED_LENGTHS)}
    got = replay_modes.mixed(runner, seqs)
    for k, tokens in seqs.items():
        assert_close(got[k], plain.forward(config, weights, tokens), REL, k)


def _masks(config):
    return [layer["mixer"]["left"]["mask"] for layer in config["layers"] if layer["type"] == "parallel" and "mask" in layer["mixer"]["left"]]


@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_sharp_attention_at_the_edges_in_prompts_and_decoding(tmp_path, name):
    """With the score scale multiplied the softmax of most heads rests on single keys: a window or a run of kept tokens one token
    too long or too short changes the logits by far more than the tolerance."""
    runner, config, weights = _runner(tmp_path, name, sharpen=12.0, max_tokens_per_step=256, max_tokens_per_request=256)
    tokens = random_tokens(config["vocab"], 120, 5)
    want = plain.forward(config, weights, tokens)
    for key in ("size", "keep_first"):
        for delta in (-1, 1):
            other = copy.deepcopy(config)
            for mask in _masks(other):
                mask[key] = max(1 if key == "size" else 0, mask[key] + delta)
            if other != config:
                assert (plain.forward(other, weights, tokens) - want).abs().max() > 0.01 * want.abs().max(), (key, delta)
    assert_close(replay_modes.portions(runner, tokens, [7, 2, 27, 64, 3, 17]), want, 1e-3)
    assert_close(replay_modes.portions(runner, tokens, [80] + [1] * 40), want, 1e-3, "the window passes over decoded tokens")


def test_positions_are_not_rotated_in_the_window_layers_and_are_in_the_others(tmp_path):
    """A longer context in front of the same tokens: kept as a fact of the plain implementation, so that the engine's agreement
    with it means something."""
    config, weights = plain.read_folder(make_kaposun_folder(tmp_path, "A"))
    bare = copy.deepcopy(config)
    bare["layers"][1]["mixer"].pop("rot")
    unscaled = copy.deepcopy(config)
    unscaled["layers"][1]["mixer"]["rot"].pop("scaling")
    tokens = random_tokens(config["vocab"], 40, 9)
    want = plain.forward(config, weights, tokens)
    for other in (bare, unscaled):
        assert (plain.forward(other, weights, tokens) - want).abs().max() > 100 * REL * want.abs().max()


def test_every_pass_of_a_loop_keeps_its_own_state(tmp_path):
    """C's loop holds recurrent layers: three passes, three states per layer, none of them shared, all moved on by decoding."""
    from kvcache_b200.engine.runner import StepEntry
    runner, config, weights = _runner(tmp_path, "C")
    tokens = random_tokens(config["vocab"], 30, 4)
    slot = runner.cache.admit()
    runner.step([StepEntry(slot, tokens[:29], [])])
    out = runner.step([StepEntry(slot, tokens[29:], [0])]).clone()
    assert_close(out, plain.forward(config, weights, tokens)[-1:], REL)
    passes = [runner.cache.states[i]["right.memory"][slot] for i in (1, 3, 5)]
    assert all((a - b).abs().max() > 1e-2 * a.abs().max() for a, b in zip(passes, passes[1:]))


def test_long_decoding(tmp_path):
    runner, config, weights = _runner(tmp_path, "A", max_tokens_per_step=512, max_tokens_per_request=512)
    tokens = random_tokens(config["vocab"], 220, 6)
    got = replay_modes.portions(runner, tokens, [20] + [1] * 200)
    assert_close(got, plain.forward(config, weights, tokens), REL)


def test_pages_behind_the_window_are_given_back_and_kept_ones_stay(tmp_path):
    """C has only a windowed attention: a long request never holds more pages than its kept tokens, its window and a portion span."""
    from kvcache_b200.engine.runner import StepEntry
    runner, config, weights = _runner(tmp_path, "C", num_pages=24, max_tokens_per_step=64, max_tokens_per_request=512)
    tokens = random_tokens(config["vocab"], 150, 8)
    slot, at, most, got = runner.cache.admit(), 0, 0, []
    for n in [16] * 5 + [1] * 70:
        got.append(runner.step([StepEntry(slot, tokens[at:at + n], list(range(n)))]).clone())
        at += n
        most = max(most, runner.cache.used_pages())
    assert_close(torch.cat(got), plain.forward(config, weights, tokens), REL)
    assert most <= 3 + (5 - 1 + 16 + 3) // 4 + 1 and runner.cache.used_pages() <= 3 + 3
    runner.cache.release(slot)
    assert runner.cache.used_pages() == 0


# ---- generation through the entry point and the scheduler -------------------------------------------------------------
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_greedy_generation_matches_plain(tmp_path, name):
    from kvcache_b200 import LLM, SamplingParams
    folder = make_kaposun_folder(tmp_path, name)
    config, weights = plain.read_folder(folder)
    prompts = [random_tokens(config["vocab"], n, 40 + n) for n in (1, 9, 24, 40)]
    llm = LLM(folder, kernels=TorchKernels(), dtype="float32", device="cpu", page_size=PAGE_SIZE[name], num_pages=40, max_running=3,
              max_tokens_per_step=48, chunk_size=16, use_graphs=False)
    got = llm.generate(prompts, SamplingParams(max_new_tokens=6, ignore_eos=True))
    for prompt, out in zip(prompts, got):
        assert out == plain.greedy(config, weights, prompt, 6)
    assert llm.core.cache.used_pages() == 0 and llm.last_stats.finished == len(prompts)
