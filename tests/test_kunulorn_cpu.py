"""The Kunulorn model in the engine (step function, cache manager, scheduler) on the CPU stand-in kernels against the plain
implementation; its parts alone against the plain functions; its configuration."""
import copy
import dataclasses

import pytest
import torch

import plain_kunulorn as plain
import replay_modes
from helpers import assert_close, make_runner, paged_scenario, random_tokens
from kunulorn_configs import CONFIGS, PAGE_SIZE, config_dict, make_kunulorn_folder
from torch_kernels import TorchKernels

REL = 1e-4


def _runner(tmp_path, name, num_pages=64, sharpen=1.0, **kw):
    folder = make_kunulorn_folder(tmp_path, name, sharpen=sharpen)
    runner = make_runner(folder, TorchKernels(), dtype="float32", device="cpu", page_size=PAGE_SIZE[name], num_pages=num_pages, **kw)
    config, weights = plain.read_folder(folder)
    return runner, config, weights


# ---- configuration --------------------------------------------------------------------------------------------------
def test_config_round_trip():
    from kvcache_b200.config import config_from_dict
    for name in CONFIGS:
        c = config_from_dict(config_dict(name))
        assert config_from_dict(c.to_dict()) == c
    c = config_from_dict(config_dict("A"))
    m = c.layers[0].mixer
    assert (m.heads, m.kv_heads, m.dim, m.vdim, m.scale, m.chunk, m.kv_from) == (4, 2, 12, 20, 0.3, 11, None) and m.rot.dims == 8
    assert c.layers[2].mixer.kv_from == 0 and c.layers[2].mixer.chunk == 19 and c.layers[3].mlp is None
    assert (c.layers[0].mlp.ff, c.layers[0].mlp.limit) == (48, 0.9) and c.embed_scale == 5.5
    r = c.layers[1].mlp
    assert (r.expert_ff, r.experts, r.top, r.weight_scale, r.groups.count, r.groups.keep, r.shared_ff) == (24, 6, 2, 1.7, 3, 2, 40)
    b = config_from_dict(config_dict("B"))
    assert b.layers[0].mixer.chunk is None and b.layers[0].mixer.rot is None and b.embed_scale == 1.0
    assert b.layers[0].mlp.groups is None and b.layers[0].mlp.shared_ff is None and b.layers[0].mlp.weight_scale == 1.0


def test_config_faults_are_all_reported():
    from kvcache_b200.config import ConfigError, config_from_dict
    bad = config_dict("A")
    bad["layers"][0]["mixer"].pop("vdim")
    bad["layers"][0]["mlp"].pop("limit")
    bad["layers"][1]["mixer"]["kv_heads"] = 4
    bad["layers"][1]["mlp"]["router"]["groups"]["count"] = 4
    bad["layers"][2]["mixer"]["kv_from"] = 3
    bad["layers"][2]["mlp"]["router"]["top"] = 5
    bad["layers"][3]["type"] = "convolution"
    bad["layers"][3]["mlp"] = {"kind": "sparse"}
    del bad["norm"]
    with pytest.raises(ConfigError) as info:
        config_from_dict(bad)
    text = str(info.value)
    for piece in ("vdim", "limit", "not a multiple of kv_heads", "not a multiple of groups.count 4", "kv_from 3", "top 5 exceeds the 4 experts",
                  "convolution", "sparse", "norm"):
        assert piece in text, piece
    other = config_dict("A")
    other["layers"][2]["mixer"]["rot"]["base"] = 5.0          # the reader must agree with its source in what is cached
    with pytest.raises(ConfigError, match="must equal those of layer 0"):
        config_from_dict(other)


def test_model_as_data(tmp_path):
    """Cache entries: keys and values with the chunk of their layer; none for a layer that reads another's (its call names the
    other's entry, which keeps what any of its readers sees)."""
    from kvcache_b200.engine.loading import load_model
    model = load_model(make_kunulorn_folder(tmp_path, "A"), "float32", "cpu", max_positions=64)
    entries = model.cache_entries()
    assert len(entries) == 3 and all(e.state is None for e in entries)
    first = entries[0].kv
    # Chunks of 11 and of 19 tokens: neither holds the other, so the entry keeps a window that holds both.
    assert (first.num_kv_heads, first.head_dim, first.v_head_dim, first.window, first.chunk, first.reach) == (2, 12, 20, 19, None, 19)
    assert (entries[1].kv.chunk, entries[1].kv.reach, entries[2].kv.chunk) == (7, -7, 16)
    assert [(c.layer, c.cache, c.writes_cache) for c in model.schedule] == [(0, 0, True), (1, 1, True), (2, 0, False), (3, 2, True)]
    reader = model.blocks[2].mixer
    assert reader.cache_spec() is None and reader.reach == -19 and not {"l2.mix.k", "l2.mix.v", "l2.mix.k.norm", "l2.mix.k.b"} & set(model.tensor_specs())
    assert model.tied and model.embed_scale == 5.5 and model.blocks[3].ffn is None
    d = load_model(make_kunulorn_folder(tmp_path, "D"), "float32", "cpu", max_positions=64)
    assert len(d.cache_entries()) == 1 and d.cache_entries()[0].kv.reach == 0 and d.blocks[0].mixer.reach == -24
    # Equal masks share an entry and a group as they are; bfloat16 caches keys and values in one width where kernels want it.
    e = load_model(make_kunulorn_folder(tmp_path, "E"), "bfloat16", "cpu", max_positions=64)
    assert [(x.kv.head_dim, x.kv.v_head_dim) for x in e.cache_entries()] == [(64, 64), (64, 64), (64, 64)]
    same = config_dict("E")
    same["layers"][2]["mixer"]["mask"]["size"] = 40
    s = load_model(make_kunulorn_folder(tmp_path, "E", seed=1, data=same), "bfloat16", "cpu", max_positions=64)
    assert s.cache_entries()[0].kv.chunk == 40 and s.cache_entries()[0].kv.window is None


def test_reach():
    from kvcache_b200.parts.base import PagedKVSpec, first_seen, reach_code
    assert (reach_code(None, None), reach_code(5, None), reach_code(None, 5)) == (0, 5, -5)
    with pytest.raises(ValueError):
        reach_code(3, 4)
    for p in range(40):
        assert first_seen(p, 0) == 0 and first_seen(p, 7) == max(0, p - 6) and first_seen(p, -7) == p // 7 * 7
    assert PagedKVSpec(1, 8, None, None, 0, 12).reach == -12


# ---- mechanisms alone ---------------------------------------------------------------------------------------------------
def _context(batch=None, kv=None):
    from kvcache_b200.engine.workspace import Workspace
    from kvcache_b200.parts.base import LayerContext
    return LayerContext(batch=batch, kernels=TorchKernels(wide=True), workspace=Workspace("cpu"), kv=kv)


def _weights(specs, seed, std=0.3):
    g = torch.Generator().manual_seed(seed)
    return {name: (torch.randn(spec.shape, generator=g) * std + (1.0 if name.endswith("norm") else 0.0)).to(torch.bfloat16)
            for name, spec in specs.items()}


def _scenario(segments, spec, page_size=4, writes=True):
    from kvcache_b200.parts.base import PagedKVView
    batch, kv = paged_scenario(segments, num_kv_heads=spec.num_kv_heads, head_dim=spec.head_dim, page_size=page_size, dtype=torch.float32,
                               device="cpu", fill_history=False)
    return batch, PagedKVView(spec=spec, k_pages=kv.k_pages, v_pages=torch.zeros(*kv.k_pages.shape[:-1], spec.v_head_dim),
                              block_table=kv.block_table, page_size=page_size, writes=writes)


def _part(W, m, prefix="m.", eps=1e-5, **kw):
    from kvcache_b200.parts.attention import GQAAttention
    from kvcache_b200.parts.position import RotaryHalf
    rot = m.get("rot")
    return GQAAttention(W, m["heads"], m["kv_heads"], m["dim"], qkv_bias=True, out_bias=True, window=None, prefix=prefix, dtype="float32",
                        position=None if rot is None else RotaryHalf(rot["dims"], rot["base"], 512), chunk=(m.get("mask") or {}).get("size"),
                        scale=m["scale"], value_dim=m["vdim"], names=("q", "k", "v", "o"), qk_norm_eps=eps, qk_norm_scope="all",
                        rotary_layout="interleaved", pad_values=True, **kw)


def _sum(delta):
    """What a norm would add to the stream: the delta and its bias."""
    return delta.delta + delta.bias


def test_centred_norm_and_a_bias_on_the_delta():
    from kvcache_b200.parts.base import BiasedDelta, ScaledDelta
    from kvcache_b200.parts.norm import LayerNorm, RMSNorm
    W, eps = 24, 1e-5
    g = torch.Generator().manual_seed(1)
    norm = LayerNorm(W, eps, "n")
    w = {"n": (torch.randn(W, generator=g) * 0.2 + 1.0).to(torch.bfloat16)}
    norm.bind(w, torch.device("cpu"))
    assert norm.fold_params() is None and norm.init_kinds() == {"n": "ones_plus_normal"}
    h, delta, bias = torch.randn(5, W, generator=g) + 3.0, torch.randn(5, W, generator=g), torch.randn(W, generator=g)
    for handed, added in ((BiasedDelta(delta, bias), delta + bias), (ScaledDelta(delta, bias), delta * bias), (delta, delta), (None, 0.0 * delta)):
        stream, out = h.clone(), torch.zeros(5, W)
        norm.add_norm(stream, handed, out, _context())
        assert_close(stream, h.double() + added.double(), 1e-6, "the add")
        assert_close(out, plain.centred_norm(h.double() + added.double(), w["n"].double(), eps), 1e-5, "the norm")
    # A mean far from zero shows the difference to a norm that does not take it off; the other norm takes a bias as well.
    rms = RMSNorm(W, eps, "n")
    rms.bind(w, torch.device("cpu"))
    stream, out = h.clone(), torch.zeros(5, W)
    rms.add_norm(stream, BiasedDelta(delta, bias), out, _context())
    assert_close(stream, h + delta + bias, 1e-6)
    assert (out.double() - plain.centred_norm(stream.double(), w["n"].double(), eps)).abs().max() > 0.5
    gathered = torch.zeros(2, W)
    norm.add_norm(h.clone(), BiasedDelta(delta, bias), gathered, _context(), rows=torch.tensor([4, 1], dtype=torch.int32))
    assert_close(gathered, plain.centred_norm((h + delta + bias).double(), w["n"].double(), eps)[[4, 1]], 1e-5, "gathered rows")


SIZES = [dict(heads=4, kv_heads=2, dim=12, vdim=20, scale=1.0, mask={"size": 7}, rot={"base": 777.0, "dims": 8}),
         dict(heads=3, kv_heads=1, dim=8, vdim=4, scale=2.0, mask={"size": 4}, rot={"base": 50.0, "dims": 8}),
         dict(heads=2, kv_heads=2, dim=6, vdim=6, scale=2.0, mask={"size": 1}, rot=None),
         dict(heads=5, kv_heads=5, dim=10, vdim=3, scale=1.5, mask=None, rot={"base": 1000.0, "dims": 2})]


@pytest.mark.parametrize("m", SIZES)
def test_attention_part_alone(m):
    """Sharp scores, whole and cut in two: the norm over a token's whole projection with its weight, neighbours turned (only part
    of a head in some cases), the chunk's first and last key, biases on all four products."""
    T, W, eps = 29, 40, 1e-5
    part = _part(W, m)
    w = _weights(part.tensor_specs(), 3)
    part.bind(w, torch.device("cpu"))
    assert set(w) == {"m." + n for n in ("q", "k", "v", "o", "q.b", "k.b", "v.b", "o.b", "q.norm", "k.norm")}
    assert w["m.q.norm"].shape == (m["heads"] * m["dim"],) and w["m.k.norm"].shape == (m["kv_heads"] * m["dim"],)
    x = torch.randn(T, W, generator=torch.Generator().manual_seed(4))
    wd = {k: v.double() for k, v in w.items()}
    pos = torch.arange(T)
    want, _ = plain.attention(m, wd, "m.", x.double(), pos, eps)
    if m["mask"] and m["mask"]["size"] > 1:       # one key more or one key less would show: the scores are sharp
        for other in (m["mask"]["size"] + 1, m["mask"]["size"] - 1):
            differs, _ = plain.attention(dict(m, mask={"size": other}), wd, "m.", x.double(), pos, eps)
            assert (differs - want).abs().max() > 0.05 * want.abs().max()
    for name in ("q.b", "k.b", "v.b", "o.b", "q.norm", "k.norm"):
        other = dict(wd, **{"m." + name: torch.ones_like(wd["m." + name])})
        differs, _ = plain.attention(m, other, "m.", x.double(), pos, eps)
        if m["mask"] != {"size": 1} or name in ("v.b", "o.b"):
            assert (differs - want).abs().max() > 0.01 * want.abs().max(), name
    batch, kv = _scenario([(0, T)], part.cache_spec())
    assert_close(_sum(part.forward(x, _context(batch, kv))), want, 1e-5)
    second, kv = _scenario([(11, T - 11)], part.cache_spec())
    first, _ = _scenario([(0, 11)], part.cache_spec())
    got = [_sum(part.forward(x[:11], _context(first, kv))), _sum(part.forward(x[11:], _context(second, kv)))]
    assert_close(torch.cat(got), want, 1e-5, "cut in two")


@pytest.mark.parametrize("size", [5, 9, 3, 1, None])
def test_a_layer_reads_the_keys_and_values_another_layer_cached(size):
    """The reader has no projection of keys and values: same cache rows (keys normalised and turned), its own queries, scale
    and mask - a smaller chunk, a larger one, none."""
    T, W, eps = 23, 32, 1e-5
    m1 = dict(heads=4, kv_heads=2, dim=8, vdim=12, scale=2.0, mask={"size": 6}, rot={"base": 50.0, "dims": 4})
    m2 = dict(m1, heads=6, scale=1.3, mask=None if size is None else {"size": size}, kv_from=0)
    owner, reader = _part(W, m1, "a."), _part(W, m2, "b.", own_kv=False)
    owner.keep_for(reader)
    assert reader.cache_spec() is None and not {"b.k", "b.v", "b.k.b", "b.v.b", "b.k.norm"} & set(reader.tensor_specs())
    assert owner.cache_spec().reach == (0 if size is None else max(6, size))
    w = {**_weights(owner.tensor_specs(), 1), **_weights(reader.tensor_specs(), 2)}
    owner.bind(w, torch.device("cpu"))
    reader.bind(w, torch.device("cpu"))
    wd = {k: v.double() for k, v in w.items()}
    x1, x2 = (torch.randn(T, W, generator=torch.Generator().manual_seed(s)) for s in (5, 6))
    pos = torch.arange(T)
    want1, kept = plain.attention(m1, wd, "a.", x1.double(), pos, eps)
    want2, _ = plain.attention(m2, wd, "b.", x2.double(), pos, eps, kept)
    got1, got2, at = [], [], 0
    _, kv = _scenario([(0, T)], owner.cache_spec())
    for n in (9, 1, 13):
        batch, _ = _scenario([(at, n)], owner.cache_spec())
        reading = dataclasses.replace(kv, writes=False)
        got1.append(_sum(owner.forward(x1[at:at + n], _context(batch, kv))))
        got2.append(_sum(reader.forward(x2[at:at + n], _context(batch, reading))))
        at += n
    assert_close(torch.cat(got1), want1, 1e-5, "the owner, with its own chunk over the wider entry")
    assert_close(torch.cat(got2), want2, 1e-5, "the reader")
    with pytest.raises(ValueError):
        reader.forward(x2[:1], _context(batch, kv))


def test_interleaved_order_gives_the_scores_of_neighbouring_pairs():
    """Reordering queries and keys alike and turning halves gives the scores of turning neighbours; turning halves without
    the reordering does not."""
    from kvcache_b200.parts.position import RotaryHalf, interleaved_order
    T, D, dims = 9, 14, 10
    g = torch.Generator().manual_seed(2)
    q, k = torch.randn(T, 1, D, generator=g, dtype=torch.float64), torch.randn(T, 1, D, generator=g, dtype=torch.float64)
    pos = torch.arange(T) * 5
    rope = RotaryHalf(dims, 99.0, 64)
    rope.bind({}, torch.device("cpu"))
    cos, sin = rope.rotation().cos.double()[pos], rope.rotation().sin.double()[pos]
    order = interleaved_order(D, dims)
    assert sorted(order.tolist()) == list(range(D)) and order[dims:].tolist() == list(range(dims, D))

    def halves(t):
        half = dims // 2
        u, v = t[..., :half], t[..., half:dims]
        return torch.cat([u * cos - v * sin, v * cos + u * sin, t[..., dims:]], dim=-1)
    rot = {"base": 99.0, "dims": dims}
    want = plain.rotate_pairs(q, pos, rot)[:, 0] @ plain.rotate_pairs(k, pos, rot)[:, 0].t()
    assert_close(halves(q[:, 0, order]) @ halves(k[:, 0, order]).t(), want, 1e-6)
    assert (halves(q[:, 0]) @ halves(k[:, 0]).t() - want).abs().max() > 0.1


def test_dense_feed_forward_part_alone():
    from kvcache_b200.parts.feedforward import GatedMLP
    T, W, F, limit = 9, 40, 24, 0.7
    part = GatedMLP(W, F, activation="clamped_swiglu", limit=limit, prefix="f.", dtype="float32", names=("gate", "up", "down"))
    w = _weights(part.tensor_specs(), 5)
    part.bind(w, torch.device("cpu"))
    x = torch.randn(T, W, generator=torch.Generator().manual_seed(6))
    wd = {k: v.double() for k, v in w.items()}
    want = plain.dense_ff({"limit": limit}, wd, "f.", x.double())
    assert_close(part.forward(x, _context()), want, 1e-5)
    assert (plain.dense_ff({"limit": 100.0}, wd, "f.", x.double()) - want).abs().max() > 0.1 * want.abs().max()


@pytest.mark.parametrize("E,top,groups,scale,shared", [(12, 3, (4, 2), 1.7, 24), (6, 2, (6, 3), 1.0, None), (5, 5, None, 0.4, 8), (8, 1, (1, 1), 2.0, 16),
                                                       (8, 4, (2, 1), 3.0, None)])
def test_routed_feed_forward_part_alone(E, top, groups, scale, shared):
    """The choice goes by score + correction (strongly negative ones among them, so that a group left out must count as minus
    infinity and not as zero), the weights by the score alone; groups change the choice; the shared result is gated."""
    from kvcache_b200.parts.feedforward import GatedMLP, RoutedMLP
    T, W, F = 17, 40, 24
    sh = None if shared is None else GatedMLP(W, shared, activation="silu", prefix="f.shared.", dtype="float32", names=("gate", "up", "down"))
    part = RoutedMLP(W, F, E, top, activation="swiglu", scores="sigmoid", prefix="f.", dtype="float32", shared=sh, correction="correction",
                     groups=groups, weight_scale=scale, shared_gate=None if shared is None else "shared.sg")
    w = _weights(part.tensor_specs(), 5)
    w["f.correction"] = (torch.randn(E, generator=torch.Generator().manual_seed(8)) * 0.6 - 1.5).to(torch.bfloat16)
    part.bind(w, torch.device("cpu"))
    x = torch.randn(T, W, generator=torch.Generator().manual_seed(6))
    wd = {k: v.double() for k, v in w.items()}
    router = {"experts": E, "top": top, "scale": scale}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    mlp = {"kind": "moe", "router": router, "expert": {"ff": F}}
    if shared is not None:
        mlp["shared"] = {"ff": shared}
    assert_close(part.forward(x, _context()), plain.feed_forward(mlp, wd, "f.", x.double()), 1e-5)
    which, weight = plain.route(mlp, wd, "f.", x.double())
    assert torch.allclose(weight.sum(dim=-1), torch.full((T,), scale, dtype=torch.float64))
    sets = lambda r, weights: [sorted(row.tolist()) for row in plain.route(dict(mlp, router=r), weights, "f.", x.double())[0]]
    if top < E:
        assert sets(router, wd) != sets(router, dict(wd, **{"f.correction": torch.zeros(E, dtype=torch.float64)}))
    if groups is not None and groups[1] < groups[0] and E > groups[0]:       # groups of one expert, no fewer than chosen, change nothing
        assert sets(router, wd) != sets({"experts": E, "top": top, "scale": scale}, wd)
    if shared is not None:
        ungated = dict(wd, **{"f.shared.sg": torch.zeros(1, W, dtype=torch.float64)})
        assert (plain.feed_forward(mlp, ungated, "f.", x.double()) - plain.feed_forward(mlp, wd, "f.", x.double())).abs().max() > 0.05


def test_routing_options_that_do_not_fit_are_refused():
    from kvcache_b200.parts.feedforward import GatedMLP, RoutedMLP
    common = dict(activation="swiglu", prefix="f.", dtype="float32")
    for bad in (dict(scores="chosen", groups=(2, 1)), dict(scores="sigmoid", groups=(3, 1)), dict(scores="sigmoid", groups=(4, 1)),
                dict(scores="all", correction="c"), dict(scores="sigmoid", shared_gate="sg"), dict(scores="other")):
        with pytest.raises(ValueError):
            RoutedMLP(8, 4, 8, 3, **dict(common, **bad))
    with pytest.raises(ValueError):
        RoutedMLP(8, 4, 8, 3, scores="chosen", shared_gate="sg", shared=GatedMLP(8, 4, activation="silu", prefix="s.", dtype="float32"), **common)


def test_pages_behind_a_chunk():
    """A group with chunks holds the pages of the current chunk only; a portion that runs over chunks holds them from the chunk
    of its first token on."""
    from kvcache_b200.cache.pages import GroupPages
    g = GroupPages(num_pages=12, page_size=4, max_slots=1, max_pages_per_request=64, chunk=10)
    assert [g.first_needed_page(p) for p in (0, 9, 10, 19, 20, 29, 30)] == [0, 0, 2, 2, 5, 5, 7]
    at, most = 0, 0
    for n in (3, 6, 1, 1, 7, 2, 25) + (1,) * 40:
        g.extend(0, at, at + n)
        for p in range(at // 10 * 10, at + n):
            assert g.table[0, p // 4] >= 0
        held = len(g.held_pages(0))
        assert held <= g.worst_case_pages(200, 25)
        if n == 1:
            most = max(most, held)
        at += n
    assert most <= 4 and g.worst_case_pages(200, 1) == 4 and g.worst_case_pages(8, 8) == 2
    g.release(0)
    assert g.allocator.num_used == 0


def test_residual_stream_after_every_layer(tmp_path):
    """Layer by layer: a model cut after k layers (its final norm with weight 1, its head the identity) gives the plain
    implementation's residual stream after layer k, centred and divided."""
    folder = make_kunulorn_folder(tmp_path, "A")
    config, weights = plain.read_folder(folder)
    tokens = random_tokens(config["vocab"], 37, 3)
    streams = []
    plain.forward(config, weights, tokens, streams)
    from kvcache_b200.cache import CacheManager
    from kvcache_b200.engine.loading import load_model
    from kvcache_b200.engine.runner import ModelRunner, StepEntry
    for k in range(1, len(streams) + 1):
        model = load_model(folder, "float32", "cpu", max_positions=64)
        model.schedule = model.schedule[:k]
        model._writers = {c.cache: c.layer for c in model.schedule if c.writes_cache}
        model.final_norm.weight = torch.ones(model.width)
        model.final_norm.eps = 0.0
        model.head = torch.eye(model.width)
        model.vocab_size, real = model.width, model.vocab_size
        cache = CacheManager(model.cache_entries(), page_size=8, num_pages=16, max_slots=1, max_tokens_per_request=64, dtype="float32", device="cpu")
        assert real == config["vocab"]
        runner = ModelRunner(model, cache, TorchKernels(wide=True), max_tokens_per_step=64)
        got = runner.step([StepEntry(cache.admit(), tokens, list(range(len(tokens))))])
        assert_close(got, plain.centred_norm(streams[k - 1], torch.ones(model.width, dtype=torch.float64), 0.0), 1e-5, f"after layer {k}")


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
    tokens = random_tokens(config["vocab"], 70, 2)
    want = plain.forward(config, weights, tokens)
    assert_close(replay_modes.last_32_one_by_one(runner, tokens), want[-33:], REL)
    assert_close(replay_modes.portions(runner, tokens, [1] * 70), want, REL, "every token alone")


@pytest.mark.parametrize("name", list(CONFIGS))
def test_portions_down_to_two_tokens(tmp_path, name):
    runner, config, weights = _runner(tmp_path, name)
    tokens = random_tokens(config["vocab"], 101, 3)
    want = plain.forward(config, weights, tokens)
    assert_close(replay_modes.portions(runner, tokens, [2, 17, 3, 31, 2, 16, 8, 22]), want, REL)
    assert_close(replay_modes.portions(runner, tokens, [40, 2, 2, 5, 52]), want, REL)


@pytest.mark.parametrize("name", list(CONFIGS))
def test_mixed_batches_with_pages_and_slots_used_again(tmp_path, name):
    """Unequal requests beside one another against each alone; a and b end and d and e take their pages, which hold other
    requests' rows."""
    page = PAGE_SIZE[name]
    runner, config, weights = _runner(tmp_path, name, num_pages=replay_modes.mixed_pool_tokens() // page)
    seqs = {k: random_tokens(config["vocab"], n, 10 + i) for i, (k, n) in enumerate(replay_modes.MIXED_LENGTHS)}
    got = replay_modes.mixed(runner, seqs)
    for k, tokens in seqs.items():
        assert_close(got[k], plain.forward(config, weights, tokens), REL, k)


@pytest.mark.parametrize("name", ["A", "C"])
def test_sharp_attention_at_the_chunks_edges_in_prompts_and_decoding(tmp_path, name):
    """With the score scale multiplied the softmax of most heads rests on single keys: a chunk one token too long or too short
    (of the layer that owns the keys, or of one that reads them), chunks counted from a portion's start, or a key lost at a
    page border changes the logits by far more than the tolerance."""
    runner, config, weights = _runner(tmp_path, name, sharpen=12.0, max_tokens_per_step=256, max_tokens_per_request=256)
    tokens = random_tokens(config["vocab"], 150, 5)
    want = plain.forward(config, weights, tokens)
    for index, layer in enumerate(config["layers"]):
        for delta in (-1, 1):
            size = layer["mixer"]["mask"]["size"] + delta
            if size < 1:
                continue
            other = copy.deepcopy(config)
            other["layers"][index]["mixer"]["mask"]["size"] = size
            assert (plain.forward(other, weights, tokens) - want).abs().max() > 0.01 * want.abs().max(), (index, delta)
    assert_close(replay_modes.portions(runner, tokens, [7, 2, 57, 64, 3, 17]), want, 1e-3)
    assert_close(replay_modes.last_32_one_by_one(runner, tokens), want[-33:], 1e-3)
    assert_close(replay_modes.portions(runner, tokens, [100] + [1] * 50), want, 1e-3, "chunks begin among decoded tokens")


def edge_key_case(part, W, T, at, strength=40.0, seed=3):
    """Weights and inputs of an attention part in which every query scores the key of row `at` far above all others: channel 0
    of the input is 1 in that row only and drives the keys along one direction, channel 1 is 1 in every row and drives the
    queries along the same direction."""
    g = torch.Generator().manual_seed(seed)
    w = {name: (torch.randn(spec.shape, generator=g) * 0.05 + (1.0 if name.endswith("norm") else 0.0)).to(torch.bfloat16)
         for name, spec in part.tensor_specs().items()}
    D = part.head_dim
    q, k = w["m.q"].float(), w["m.k"].float()
    q[:, :2], k[:, :2] = 0.0, 0.0
    for h in range(part.num_heads):
        q[h * D, 1] = strength
    for h in range(part.num_kv_heads):
        k[h * D, 0] = strength
    w["m.q"], w["m.k"] = q.to(torch.bfloat16), k.to(torch.bfloat16)
    x = torch.randn(T, W, generator=g) * 0.1
    x[:, 0], x[:, 1] = 0.0, 1.0
    x[at, 0] = 1.0
    return w, x


@pytest.mark.parametrize("at,size,taken", [(0, None, True), (128, 128, True), (127, 128, False), (200, 100, True), (199, 100, False)])
def test_one_key_at_the_edge_of_a_chunk_takes_all_the_weight_or_none(at, size, taken):
    """Random weights would hide a lost key among hundreds: here one key takes all the weight of the queries that see it - the
    first key of the last rows' chunk, many pages back - and none where it is the last key of the chunk before."""
    T, W = 256, 24
    m = dict(heads=4, kv_heads=2, dim=8, vdim=6, scale=40.0, mask=None if size is None else {"size": size}, rot=None)
    part = _part(W, m)
    w, x = edge_key_case(part, W, T, at)
    part.bind(w, torch.device("cpu"))
    wd = {k: v.double() for k, v in w.items()}
    want, (_, values) = plain.attention(m, wd, "m.", x.double(), torch.arange(T), 1e-5)
    the_value = values[at].repeat_interleave(2, dim=0).reshape(1, -1)
    near = (want[250:] - plain.linear(the_value, wd["m.o"], wd["m.o.b"])).abs().max() < 1e-3 * want.abs().max()
    assert bool(near) == taken
    _, kv = _scenario([(0, T)], part.cache_spec(), page_size=16)
    got, start = [], 0
    for n in [131, 2, 67, 48] + [1] * 8:
        batch, _ = _scenario([(start, n)], part.cache_spec(), page_size=16)
        got.append(_sum(part.forward(x[start:start + n], _context(batch, kv))))
        start += n
    assert_close(torch.cat(got), want, 1e-5)


def test_long_decoding(tmp_path):
    runner, config, weights = _runner(tmp_path, "A", max_tokens_per_step=512, max_tokens_per_request=512)
    tokens = random_tokens(config["vocab"], 300, 6)
    got = replay_modes.portions(runner, tokens, [20] + [1] * 280)
    assert_close(got, plain.forward(config, weights, tokens), REL)


def test_pages_behind_every_chunk_are_given_back(tmp_path):
    """C has only chunked layers: a long request never holds more pages than its widest chunk and a portion span."""
    runner, config, weights = _runner(tmp_path, "C", num_pages=24, max_tokens_per_step=64, max_tokens_per_request=512)
    from kvcache_b200.engine.runner import StepEntry
    tokens = random_tokens(config["vocab"], 200, 8)
    want = plain.forward(config, weights, tokens)
    slot, at, most = runner.cache.admit(), 0, 0
    got = []
    for n in [16] * 5 + [1] * 120:
        got.append(runner.step([StepEntry(slot, tokens[at:at + n], list(range(n)))]).clone())
        at += n
        most = max(most, runner.cache.used_pages())
    assert_close(torch.cat(got), want, REL)
    assert most <= (12 - 1 + 16 + 3) // 4 + 1
    runner.cache.release(slot)
    assert runner.cache.used_pages() == 0


# ---- generation through the entry point and the scheduler -------------------------------------------------------------
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_greedy_generation_matches_plain(tmp_path, name):
    from kvcache_b200 import LLM, SamplingParams
    folder = make_kunulorn_folder(tmp_path, name)
    config, weights = plain.read_folder(folder)
    prompts = [random_tokens(config["vocab"], n, 40 + n) for n in (1, 9, 24, 40)]
    llm = LLM(folder, kernels=TorchKernels(), dtype="float32", device="cpu", page_size=PAGE_SIZE[name], num_pages=40, max_running=3,
              max_tokens_per_step=48, chunk_size=16, use_graphs=False)
    got = llm.generate(prompts, SamplingParams(max_new_tokens=6, ignore_eos=True))
    for prompt, out in zip(prompts, got):
        assert out == plain.greedy(config, weights, prompt, 6)
    assert llm.core.cache.used_pages() == 0 and llm.last_stats.finished == len(prompts)
