"""The Kunulorn model through the engine on the GPU, in float32 and bfloat16, against the plain implementation, and every CUDA
operator (or operator option) it brought alone against the plain PyTorch statement of the same operator
(tests/torch_kernels.py)."""
import copy
import dataclasses
import json
import os
import subprocess
import sys

import numpy as np

import pytest
import torch

import plain_kunulorn as plain
import replay_modes
from helpers import assert_close, batch_to, clone_kv, make_runner, paged_scenario, random_tokens
from kunulorn_configs import CONFIGS, PAGE_SIZE, config_dict, make_kunulorn_folder
from torch_kernels import TorchKernels

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {torch.float32: 2e-5, torch.bfloat16: 2e-2}


def _spread(config, weights, tokens, want):
    """What rounding alone does to each position's logits: the plain implementation with every product's rows and results
    rounded to bfloat16, against itself without."""
    with plain.rounding(torch.bfloat16):
        return (plain.forward(config, weights, tokens) - want).abs().max(dim=1).values


def assert_model_close(got, want, dtype, what="", spread=None, rel=None):
    """float32: within `rel` of the largest logit.  bfloat16: no position beyond 4 times the largest error that rounding alone
    makes in the plain implementation (`spread`; floor: 1 % of the largest logit), the median position within 2 % - a lost
    key or a token in the wrong chunk moves positions by as much as the logits themselves."""
    if dtype == "float32":
        return assert_close(got, want, rel or 1e-4, what)
    got, want = got.detach().double().cpu(), want.double()
    assert got.shape == want.shape and torch.isfinite(got).all(), what
    scale = float(want.abs().max())
    err = (got - want).abs().max(dim=1).values
    limit = 4.0 * max(float(spread.max()), 0.01 * scale)
    assert float(err.max()) <= limit, f"{what}: error {float(err.max()):.3e} of {scale:.3e}, limit {limit:.3e}"
    assert float(err.median()) <= 0.02 * scale, f"{what}: median error {float(err.median()):.3e} of {scale:.3e}"


@pytest.fixture(scope="module")
def kernels():
    from kvcache_b200.kernels.api import CudaKernels
    return CudaKernels(DEV)


def _rand(*shape, dtype=torch.float32, seed=0, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(dtype)


def _used(k, before):
    return {name for name, count in k.launch_counts.items() if count > before.get(name, 0)}


# ---- operators alone ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("W,T", [(23, 5), (24, 5), (200, 9), (896, 300), (2050, 3), (2052, 260), (8200, 2), (48, 400)])
def test_centred_norm_with_a_bias_on_the_delta(kernels, dtype, W, T):
    """h += delta + bias (or with a scale as well, or with neither) inside the launch that normalises the next rows, with and
    without taking the mean off: the scalar, the vector and the warp-per-row forms, in place and for gathered rows.  The
    stream's mean is large against its spread, where squares taken before the mean is off would lose the variance."""
    h, delta = _rand(T, W, seed=1) + 30.0, _rand(T, W, dtype=dtype, seed=2)
    bias, scale, weight = _rand(W, seed=5), _rand(W, seed=3), _rand(W, seed=4) + 1.0
    for rows in (None, torch.tensor([T - 1, 0, T // 2], dtype=torch.int32)):
        n = T if rows is None else len(rows)
        for b, s, d in ((bias, None, delta), (bias, scale, delta), (None, None, delta), (None, None, None)):
            for centred in (True, False):
                h_ref, out_ref = h.clone(), torch.zeros(n, W, dtype=dtype)
                TorchKernels(wide=True).add_rmsnorm(h_ref, d, weight, 1e-5, out_ref, rows, delta_scale=s, delta_bias=b, centred=centred)
                h_dev, out = h.clone().to(DEV), torch.zeros(n, W, dtype=dtype, device=DEV)
                on = lambda t: None if t is None else t.to(DEV)
                kernels.add_rmsnorm(h_dev, on(d), on(weight), 1e-5, out, on(rows), delta_scale=on(s), delta_bias=on(b), centred=centred)
                assert_close(h_dev, h_ref, 1e-6, "the stream")
                assert_close(out, out_ref, TOL[dtype], f"the normalised rows, centred {centred}")


def _kv_scenario(segments, Hkv, D, Dv, page, dtype, chunk=None, window=None, seed=2, fill=True, drop_chunk=None):
    """`drop_chunk`: pages that lie wholly before the first row's chunk of this size are taken out of the block table, as a
    chunked cache entry gives them back."""
    from kvcache_b200.parts.base import PagedKVSpec, PagedKVView
    batch, kv = paged_scenario(segments, num_kv_heads=Hkv, head_dim=D, page_size=page, dtype=dtype, device="cpu", seed=seed, fill_history=fill)
    values = _rand(*kv.k_pages.shape[:-1], Dv, dtype=dtype, seed=seed + 1) if fill else torch.zeros(*kv.k_pages.shape[:-1], Dv, dtype=dtype)
    table = kv.block_table.clone()
    if drop_chunk:
        for i, (start, _) in enumerate(segments):
            table[i, :start // drop_chunk * drop_chunk // page] = -1
    return batch, PagedKVView(spec=PagedKVSpec(Hkv, D, window, None if Dv == D else Dv, 0, chunk), k_pages=kv.k_pages, v_pages=values,
                              block_table=table, page_size=page, writes=True)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("Hq,Hkv,D,Dv,Dk,Dvs,dims", [(4, 2, 12, 20, 12, 20, 8), (3, 1, 10, 6, 10, 6, 10), (4, 2, 64, 48, 64, 64, 32), (14, 2, 64, 64, 64, 64, 64),
                                                     (2, 1, 32, 64, 64, 64, 32), (5, 5, 16, 24, 24, 24, 0), (40, 8, 128, 128, 128, 128, 64),
                                                     (2, 2, 48, 32, 48, 48, 16)])
def test_append_with_a_norm_over_the_whole_projection(kernels, dtype, Hq, Hkv, D, Dv, Dk, Dvs, dims):
    """Biases, the norm over a token's whole query (key) projection with weights, rotation of part of a head, keys and values
    stored wider than they are - single rows, a step of hundreds of rows (several rows a block), and rows of queries alone
    for a layer that reads another's keys; bfloat16 sizes in steps of 8 take the kernel that moves 16 bytes a thread."""
    page, table = 8, 700
    angles = torch.arange(table, dtype=torch.float64)[:, None] * (100.0 ** (-torch.arange(max(dims // 2, 1), dtype=torch.float64) * 2.0 / max(dims, 1)))[None, :]
    cos, sin = (torch.cos(angles).float(), torch.sin(angles).float()) if dims else (None, None)
    on = lambda t: None if t is None else t.to(DEV)
    for segments in ([(0, 9), (130, 3), (63, 2), (5, 1)], [(0, 301), (600, 1), (17, 2)]):
        batch, kv = _kv_scenario(segments, Hkv, Dk, Dvs, page, dtype, fill=False)
        kv.k_pages.fill_(7.0)
        kv.v_pages.fill_(7.0)                                    # stale rows: the zeros after a key or value must be written
        T = batch.num_tokens
        P = (Hq + Hkv) * D + Hkv * Dv
        qkv, bias = _rand(T, P, dtype=dtype, seed=3), _rand(P, seed=4)
        q_norm, k_norm = _rand(Hq * D, seed=5) + 1.0, _rand(Hkv * D, seed=6) + 1.0
        for b in (bias, None):
            ref_kv, dev_kv = clone_kv(kv), clone_kv(kv, DEV)
            ref_q, got_q = torch.zeros(T, Hq * Dk, dtype=dtype), torch.zeros(T, Hq * Dk, dtype=dtype, device=DEV)
            args = dict(norm_eps=1e-5, key_dim=D, value_dim=Dv, norm_scope="all")
            TorchKernels(wide=True).qkv_rope_append(qkv, b, cos, sin, batch, ref_kv, ref_q, Hq, q_norm=q_norm, k_norm=k_norm, **args)
            kernels.qkv_rope_append(on(qkv), on(b), on(cos), on(sin), batch_to(batch, DEV), dev_kv, got_q, Hq, q_norm=on(q_norm),
                                    k_norm=on(k_norm), **args)
            kernels.check_errors()
            assert_close(got_q, ref_q, TOL[dtype], "queries")
            assert_close(dev_kv.k_pages, ref_kv.k_pages, TOL[dtype], "keys")
            assert_close(dev_kv.v_pages, ref_kv.v_pages, TOL[dtype], "values")
            reading, reading_dev = dataclasses.replace(ref_kv, writes=False), dataclasses.replace(dev_kv, writes=False)
            only, b_only = qkv[:, :Hq * D].contiguous(), None if b is None else b[:Hq * D].contiguous()
            ref_q2, got_q2 = torch.zeros_like(ref_q), torch.zeros_like(got_q)
            TorchKernels(wide=True).qkv_rope_append(only, b_only, cos, sin, batch, reading, ref_q2, Hq, q_norm=q_norm, queries_only=True, **args)
            kernels.qkv_rope_append(on(only), on(b_only), on(cos), on(sin), batch_to(batch, DEV), reading_dev, got_q2, Hq, q_norm=on(q_norm),
                                    queries_only=True, **args)
            kernels.check_errors()
            assert_close(got_q2, ref_q2, TOL[dtype], "queries alone")
            assert torch.equal(dev_kv.k_pages.cpu(), reading_dev.k_pages.cpu())
    from kvcache_b200.kernels.api import KernelError
    with pytest.raises(KernelError):
        kernels.qkv_rope_append(on(only), None, None, None, batch_to(batch, DEV), dev_kv, got_q2, Hq, q_norm=on(q_norm), queries_only=True, **args)


def test_append_in_bfloat16_gives_a_row_the_same_bits_alone_and_among_many(kernels):
    Hq, Hkv, D, page = 14, 2, 64, 16
    batch, kv = _kv_scenario([(0, 300)], Hkv, D, D, page, torch.bfloat16, fill=False)
    qkv, bias = _rand(300, (Hq + 2 * Hkv) * D, dtype=torch.bfloat16, seed=3).to(DEV), _rand((Hq + 2 * Hkv) * D, seed=4).to(DEV)
    qn, kn = (_rand(n * D, seed=5).to(DEV) + 1.0 for n in (Hq, Hkv))
    together, kv_a = torch.zeros(300, Hq * D, dtype=torch.bfloat16, device=DEV), clone_kv(kv, DEV)
    kernels.qkv_rope_append(qkv, bias, None, None, batch_to(batch, DEV), kv_a, together, Hq, q_norm=qn, k_norm=kn, norm_eps=1e-5, norm_scope="all")
    part, _ = _kv_scenario([(100, 7)], Hkv, D, D, page, torch.bfloat16, fill=False)
    kv_b = clone_kv(kv, DEV)
    alone = torch.zeros(7, Hq * D, dtype=torch.bfloat16, device=DEV)
    kernels.qkv_rope_append(qkv[100:107].contiguous(), bias, None, None, batch_to(part, DEV), kv_b, alone, Hq, q_norm=qn, k_norm=kn, norm_eps=1e-5,
                            norm_scope="all")
    kernels.check_errors()
    assert torch.equal(alone, together[100:107])
    for p in range(100, 107):
        at = int(kv.block_table[0, p // page]), slice(None), p % page
        assert torch.equal(kv_a.k_pages[at], kv_b.k_pages[at]) and torch.equal(kv_a.v_pages[at], kv_b.v_pages[at])


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("Hq,Hkv,D,Dv,chunk", [(4, 2, 16, 8, 11), (3, 3, 6, 10, 1), (8, 2, 64, 64, 64), (5, 1, 40, 72, 48), (2, 2, 200, 200, 130), (20, 1, 32, 32, 96)])
def test_attention_within_chunks(kernels, dtype, Hq, Hkv, D, Dv, chunk):
    """Prompts, portions that begin inside a chunk and run over several, single tokens at a chunk's first, second and last
    place, pages of chunks that are over gone from the block table; float32, and bfloat16 sizes the tensor-core kernels do not
    take, on the generic kernel.  Then the same cache entry read by a layer with another chunk and by one without."""
    from kvcache_b200.engine.workspace import Workspace
    c = chunk
    segments = [(0, 70), (c * 3, 1), (c * 3 + 1, 1), (c * 4 - 1, 1), (150, 30), (0, 1), (c + c // 2, 2 * c + 3)]
    batch, kv = _kv_scenario(segments, Hkv, D, Dv, 8, dtype, chunk=c, drop_chunk=c)
    T = batch.num_tokens
    q = _rand(T, Hq * D, dtype=dtype, seed=5, scale=0.6)
    ref, got = torch.zeros(T, Hq * Dv, dtype=dtype), torch.zeros(T, Hq * Dv, dtype=dtype, device=DEV)
    TorchKernels(wide=True).paged_attention(q, batch, kv, ref, Hq, 0.4)
    kernels.paged_attention(q.to(DEV), batch_to(batch, DEV), clone_kv(kv, DEV), got, Hq, 0.4, Workspace(DEV))
    kernels.check_errors()
    assert_close(got, ref, TOL[dtype])
    batch, kv = _kv_scenario(segments, Hkv, D, Dv, 8, dtype)
    for reach in (-max(1, c - 1), -(c + 5), 0, 9):
        TorchKernels(wide=True).paged_attention(q, batch, kv, ref, Hq, 0.4, reach=reach)
        kernels.paged_attention(q.to(DEV), batch_to(batch, DEV), clone_kv(kv, DEV), got, Hq, 0.4, Workspace(DEV), reach=reach)
        kernels.check_errors()
        assert_close(got, ref, TOL[dtype], f"read with reach {reach}")


@pytest.mark.parametrize("path", ["default", "clusters without TMA", "scratch decode", "tensor memory from 128 rows, tiles shared out"])
@pytest.mark.parametrize("Hq,Hkv,D,chunk", [(4, 2, 64, 64), (8, 2, 64, 1000), (2, 1, 128, 192), (6, 2, 32, 48), (16, 1, 64, 300), (4, 4, 48, 640), (3, 1, 96, 37)])
def test_tensor_core_attention_within_chunks(kernels, path, Hq, Hkv, D, chunk):
    """bfloat16 with values as wide as keys: the tensor-memory and mma.sync kernels for portions, the TMA-cluster, cluster and
    scratch-merge kernels for single tokens - chunks that end inside a tile of rows, inside a tile of keys and at their edges,
    several units a tile, short requests beside long ones; no generic kernel may run."""
    from kvcache_b200.engine.workspace import Workspace
    from kvcache_b200.kernels.api import CudaKernels
    from kvcache_b200.parts.base import PagedKVSpec
    k, min_tiles = kernels, 16
    if path != "default":
        k = CudaKernels(DEV)
    if path == "clusters without TMA":
        k.tc_attention_min_rows, k.decode_merge = None, "cluster"
    elif path == "scratch decode":
        k.tc_attention_min_rows, k.decode_merge = None, "ticket"
    elif path != "default":
        k.tc_attention_min_rows, min_tiles = 128, 2
        k.tc_unit_min_tiles = min_tiles
    dtype = torch.bfloat16
    last = 2560 // chunk * chunk
    segments = [(0, 700), (2500, 1), (last, 1), (last - 1, 1), (1500, 300), (900, 1), (63, 1), (64, 1), (0, 1), (3, 2), (1100, 130)]
    batch, kv = paged_scenario(segments, num_kv_heads=Hkv, head_dim=D, page_size=16, dtype=dtype, device="cpu", seed=11, tc_min_key_tiles=min_tiles)
    kv = dataclasses.replace(kv, spec=PagedKVSpec(Hkv, D, None, None, 0, chunk))
    for i, (start, _) in enumerate(segments):
        kv.block_table[i, :start // chunk * chunk // 16] = -1
    T = batch.num_tokens
    q = _rand(T, Hq * D, dtype=dtype, seed=5, scale=0.5)
    ref, got = torch.zeros(T, Hq * D, dtype=dtype), torch.zeros(T, Hq * D, dtype=dtype, device=DEV)
    TorchKernels(wide=True).paged_attention(q, batch, kv, ref, Hq, 0.2)
    before = dict(k.launch_counts)
    k.paged_attention(q.to(DEV), batch_to(batch, DEV), clone_kv(kv, DEV), got, Hq, 0.2, Workspace(DEV))
    k.check_errors()
    used = _used(k, before)
    assert not used & {"attention_sink", "attention_generic"}, used
    if D in (64, 128) and path in ("default", "tensor memory from 128 rows, tiles shared out"):
        assert used == {"attention_tc", "flash_decode_tma"}, used
    assert_close(got, ref, TOL[dtype])


@pytest.mark.parametrize("D,chunk,requests", [(64, 96, 20), (128, 64, 17)])
def test_rotation_and_append_fused_into_decode_attention_within_chunks(kernels, D, chunk, requests):
    """A plain layer (no norms, no gate) with chunks takes the fused decode kernel: the new key's stage is found among the
    chunk's stages, also where the new token opens a chunk."""
    from kvcache_b200.engine.workspace import Workspace
    from kvcache_b200.parts.base import PagedKVSpec
    Hq, Hkv, dtype = 4, 2, torch.bfloat16
    segments = [(chunk * (3 + i % 5) + (0, 1, chunk - 1, 17)[i % 4], 1) for i in range(requests)]
    batch, kv = paged_scenario(segments, num_kv_heads=Hkv, head_dim=D, page_size=16, dtype=dtype, device="cpu", seed=3)
    kv = dataclasses.replace(kv, spec=PagedKVSpec(Hkv, D, None, None, 0, chunk))
    qkv, bias = _rand(requests, (Hq + 2 * Hkv) * D, dtype=dtype, seed=4), _rand((Hq + 2 * Hkv) * D, seed=5)
    ref_q, ref, ref_kv = torch.zeros(requests, Hq * D, dtype=dtype), torch.zeros(requests, Hq * D, dtype=dtype), clone_kv(kv)
    TorchKernels(wide=True).qkv_rope_append(qkv, bias, None, None, batch, ref_kv, ref_q, Hq)
    TorchKernels(wide=True).paged_attention(ref_q, batch, ref_kv, ref, Hq, 0.1)
    got, dev_kv = torch.zeros(requests, Hq * D, dtype=dtype, device=DEV), clone_kv(kv, DEV)
    assert kernels.rope_append_attention(qkv.to(DEV), bias.to(DEV), None, None, batch_to(batch, DEV), dev_kv, got, Hq, 0.1, Workspace(DEV))
    kernels.check_errors()
    assert_close(got, ref, 2e-2)
    assert_close(dev_kv.k_pages, ref_kv.k_pages, 1e-2)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows", [1, 70, 500])
def test_one_key_at_the_edge_of_a_chunk_takes_all_the_weight(kernels, dtype, rows):
    """One head's query matches the first key of its chunk and nothing else: the head's result is that key's value.  The key
    just before, the last of the chunk before, matches still more strongly and must not count - for a single token and in
    portions that begin before the chunk and end in it."""
    from kvcache_b200.engine.workspace import Workspace
    Hq, Hkv, D, page, chunk = 4, 2, 64, 16, 400
    pos = 3 * chunk - 2
    segments = [(pos + 1 - rows, rows), (5, 3)]
    row = rows - 1
    for inside, outside in ((2 * chunk, 2 * chunk - 1), (2 * chunk + 63, 2 * chunk - 64)):
        batch, kv = _kv_scenario(segments, Hkv, D, D, page, dtype, chunk=chunk, seed=6)
        key = lambda p: kv.k_pages[int(kv.block_table[0, p // page]), 1, p % page]
        T = batch.num_tokens
        q = (_rand(T, Hq * D, seed=7) * 0.01).to(dtype)
        q.view(T, Hq, D)[row, 3] = (key(inside).float() * 2.0).to(dtype)
        key(outside).copy_((key(inside).float() * 1.5).to(dtype))
        got = torch.zeros(T, Hq * D, dtype=dtype, device=DEV)
        kernels.paged_attention(q.to(DEV), batch_to(batch, DEV), clone_kv(kv, DEV), got, Hq, 1.0, Workspace(DEV))
        kernels.check_errors()
        value = kv.v_pages[int(kv.block_table[0, inside // page]), 1, inside % page]
        assert_close(got.view(T, Hq, D)[row, 3], value, 2e-2 if dtype == torch.bfloat16 else 1e-4, f"key {inside}")


@pytest.mark.parametrize("T,E,top,groups,extra", [(9, 12, 3, (4, 2), 1), (1, 6, 2, (6, 3), 2), (130, 64, 8, (8, 3), 8), (33, 5, 5, None, 0), (700, 256, 8, (8, 4), 8),
                                                  (40, 48, 40, (2, 2), 1), (7, 1000, 6, (500, 4), 3), (5, 3, 1, (1, 1), 1), (64, 128, 1, (16, 1), 0)])
def test_routing_by_sigmoid_scores_within_groups(kernels, T, E, top, groups, extra):
    """The chosen experts (as sets with their weights, in the order of their choice scores), with strongly negative choice
    scores, further columns beside the router's, and corrections that turn choices; without a correction as well."""
    logits = _rand(T, E + extra, seed=1, scale=2.0)
    correction = _rand(E, seed=2, scale=0.7) - 1.5
    for c in (correction, None):
        ref_c, ref_s = torch.zeros(T, top, dtype=torch.int32), torch.zeros(T, top)
        TorchKernels().route_sigmoid(logits, E, c, groups, 1.7, ref_c, ref_s)
        got_c, got_s = torch.zeros(T, top, dtype=torch.int32, device=DEV), torch.zeros(T, top, device=DEV)
        kernels.route_sigmoid(logits.to(DEV), E, None if c is None else c.to(DEV), groups, 1.7, got_c, got_s)
        same = (got_c.cpu() == ref_c).all(dim=1)
        assert int((~same).sum()) <= T // 100                    # a tie in float32 may fall either way
        assert_close(got_s.cpu()[same], ref_s[same], 1e-5)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,E,top,W,F", [(9, 5, 2, 40, 24), (70, 16, 2, 192, 64), (400, 8, 3, 128, 32), (3, 3, 3, 60, 16), (5, 4, 2, 33, 8)])
def test_routed_experts_on_a_gated_base(kernels, dtype, T, E, top, W, F):
    """The shared result times sigmoid of one logit a row, added to the routed sum: on CUDA cores (float32), mma.sync tiles,
    and from 1,024 pairs the tensor-memory kernel."""
    from kvcache_b200.engine.workspace import Workspace
    x = _rand(T, W, dtype=dtype, seed=1)
    w_up, w_down = _rand(E, 2 * F, W, dtype=dtype, seed=2, scale=0.2), _rand(E, W, F, dtype=dtype, seed=3, scale=0.2)
    logits, base = _rand(T, E + 3, seed=4), _rand(T, W, dtype=dtype, seed=5, scale=4.0)
    chosen, share = torch.zeros(T, top, dtype=torch.int32), torch.zeros(T, top)
    TorchKernels().route_sigmoid(logits, E, None, None, 1.0, chosen, share)
    on = lambda t: t.to(DEV)
    ref, got = torch.zeros(T, W, dtype=dtype), torch.zeros(T, W, dtype=dtype, device=DEV)
    TorchKernels(wide=True).routed_experts(x, w_up, w_down, chosen, share, ref, "swiglu", base=base, base_gate=(logits, E))
    kernels.routed_experts(on(x), on(w_up), on(w_down), on(chosen), on(share), got, "swiglu", Workspace(DEV), base=on(base), base_gate=(on(logits), E))
    kernels.check_errors()
    assert_close(got, ref, TOL[dtype] * 2)
    ungated = torch.zeros_like(ref)
    TorchKernels(wide=True).routed_experts(x, w_up, w_down, chosen, share, ungated, "swiglu", base=base)
    assert float((ungated.double() - ref.double()).abs().max()) > 0.1 * float(ref.double().abs().max())


@pytest.mark.parametrize("M,I,K,expected", [(8, 256, 192, "gemm_skinny"), (24, 256, 192, "gemm_wstream"), (100, 256, 192, "gemm_library"),
                                            (1024, 4864, 128, "gemm_tcgen05"), (2000, 2432, 72, "gemm_tcgen05")])
def test_clamped_gated_product(kernels, M, I, K, expected):
    """The clamped activation in the epilogues of the products over interleaved gate/up rows, the tensor-memory product (pairs
    of SMs, its edge tiles included) among them; both clamps active."""
    from kvcache_b200.engine.workspace import Workspace
    x, w = _rand(M, K, dtype=torch.bfloat16, seed=1), _rand(2 * I, K, dtype=torch.bfloat16, seed=2, scale=0.15)
    ref, got = torch.zeros(M, I, dtype=torch.bfloat16), torch.zeros(M, I, dtype=torch.bfloat16, device=DEV)
    before = dict(kernels.launch_counts)
    kernels.gate_up_act(x.to(DEV), w.to(DEV), got, Workspace(DEV), True, activation="clamped_swiglu", limit=1.1)
    kernels.check_errors()
    assert expected in _used(kernels, before)
    TorchKernels().gate_up_act(x, w, ref, None, True, activation="clamped_swiglu", limit=1.1)
    assert_close(got, ref, 2e-2)
    silu = torch.zeros_like(got)
    kernels.gate_up_act(x.to(DEV), w.to(DEV), silu, Workspace(DEV), True)
    TorchKernels().gate_up_act(x, w, ref, None, True)
    assert_close(silu, ref, 2e-2, "the plain gated form beside it")


# ---- the model in the engine ------------------------------------------------------------------------------------------
def _runner(tmp_path, kernels, name, dtype, num_pages=64, sharpen=1.0, data=None, **kw):
    folder = make_kunulorn_folder(tmp_path, name, sharpen=sharpen, dtype=torch.bfloat16, data=data, all_experts=dtype == "bfloat16")
    runner = make_runner(folder, kernels, dtype=dtype, device=DEV, page_size=PAGE_SIZE[name], num_pages=num_pages, **kw)
    config, weights = plain.read_folder(folder)
    return runner, config, weights


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_four_ways_of_cutting(tmp_path, kernels, name, dtype):
    page = PAGE_SIZE[name]
    runner, config, weights = _runner(tmp_path, kernels, name, dtype, num_pages=max(replay_modes.mixed_pool_tokens(), 128) // page)
    tokens = random_tokens(config["vocab"], 101, 3)
    want = plain.forward(config, weights, tokens)
    spread = _spread(config, weights, tokens, want)
    assert_model_close(replay_modes.whole(runner, tokens), want, dtype, "whole", spread)
    for n in (1, 2, 3):
        assert_model_close(replay_modes.whole(runner, tokens[:n]), want[:n], dtype, f"first {n}", spread)
    assert_model_close(replay_modes.last_32_one_by_one(runner, tokens), want[-33:], dtype, "decode", spread)
    assert_model_close(replay_modes.portions(runner, tokens, [2, 17, 3, 31, 2, 16, 8, 22]), want, dtype, "portions", spread)
    seqs = {k: random_tokens(config["vocab"], n, 10 + i) for i, (k, n) in enumerate(replay_modes.MIXED_LENGTHS)}
    got = replay_modes.mixed(runner, seqs)
    for k, toks in seqs.items():
        alone = plain.forward(config, weights, toks)
        assert_model_close(got[k], alone, dtype, f"mixed {k}", _spread(config, weights, toks, alone))
    assert runner.cache.used_pages() == 0
    kernels.check_errors()


def test_the_tensor_core_kernels_serve_sizes_in_steps_of_16(tmp_path, kernels):
    """Configuration E in bfloat16: no attention call of a step goes through a generic kernel."""
    runner, config, weights = _runner(tmp_path, kernels, "E", "bfloat16", num_pages=64)
    tokens = random_tokens(config["vocab"], 120, 3)
    before = dict(kernels.launch_counts)
    replay_modes.portions(runner, tokens, [80, 39, 1])
    used = _used(kernels, before)
    assert {"flash_prefill", "flash_decode_tma", "norm_rope_append", "route_sigmoid"} <= used, used
    assert not used & {"attention_generic", "attention_sink"}, used


@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_float32_rows_do_not_depend_on_the_batch_or_the_cut(tmp_path, kernels, name):
    """In float32 a position's logits are bit for bit the same alone, beside other requests, and in portions."""
    runner, config, _ = _runner(tmp_path, kernels, name, "float32")
    from kvcache_b200.engine.runner import StepEntry
    a, b = random_tokens(config["vocab"], 40, 1), random_tokens(config["vocab"], 23, 2)
    alone = replay_modes.whole(runner, a)
    sa, sb = runner.cache.admit(), runner.cache.admit()
    first = runner.step([StepEntry(sb, b[:20], []), StepEntry(sa, a[:17], list(range(17)))]).clone()
    second = runner.step([StepEntry(sa, a[17:], list(range(23))), StepEntry(sb, b[20:21], [0])]).clone()
    assert torch.equal(torch.cat([first, second[:23]]), alone)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "D", "E"])
def test_long_prompts(tmp_path, kernels, name, dtype):
    """A prompt of several hundred tokens whole (the tensor-memory kernels), in two long portions and beside another request;
    then decoded tokens behind it."""
    runner, config, weights = _runner(tmp_path, kernels, name, dtype, num_pages=200, max_tokens_per_step=700, max_tokens_per_request=700)
    from kvcache_b200.engine.runner import StepEntry
    tokens, other = random_tokens(config["vocab"], 600, 11), random_tokens(config["vocab"], 90, 12)
    want = plain.forward(config, weights, tokens)
    spread = _spread(config, weights, tokens, want) if dtype == "bfloat16" else None
    assert_model_close(replay_modes.whole(runner, tokens), want, dtype, "whole", spread)
    assert_model_close(replay_modes.portions(runner, tokens, [290, 310]), want, dtype, "two portions", spread)
    assert_model_close(replay_modes.portions(runner, tokens, [560] + [1] * 40), want, dtype, "decoded behind a long prompt", spread)
    sa, sb = runner.cache.admit(), runner.cache.admit()
    got = runner.step([StepEntry(sb, other[:60], []), StepEntry(sa, tokens[:333], list(range(333)))]).clone()
    more = runner.step([StepEntry(sa, tokens[333:], list(range(267))), StepEntry(sb, other[60:], [29])]).clone()
    assert_model_close(torch.cat([got, more[:267]]), want, dtype, "beside another request", spread)
    kernels.check_errors()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "C", "E"])
def test_sharp_attention_at_the_edges(tmp_path, kernels, name, dtype):
    """Sharpened scores make single keys carry the softmax: a chunk one token off (of the layer that owns keys or of one that
    reads them), or a key lost at a page border, in a portion's first rows or behind decoded tokens, shows.  bfloat16, whose
    rounding of much larger scores would itself change which key wins, is sharpened less (its single keys are met at kernel level)."""
    sharpen, rel = (12.0, 1e-3) if dtype == "float32" else (3.0, None)
    runner, config, weights = _runner(tmp_path, kernels, name, dtype, sharpen=sharpen, num_pages=96, max_tokens_per_step=320, max_tokens_per_request=320)
    tokens = random_tokens(config["vocab"], 300, 5)
    want = plain.forward(config, weights, tokens)
    if dtype == "float32":
        for index, layer in enumerate(config["layers"]):
            for delta in (-1, 1):
                size = layer["mixer"]["mask"]["size"] + delta
                if size < 1:
                    continue
                other = copy.deepcopy(config)
                other["layers"][index]["mixer"]["mask"]["size"] = size
                assert (plain.forward(other, weights, tokens) - want).abs().max() > 5 * rel * want.abs().max(), (index, delta)
    spread = _spread(config, weights, tokens, want) if dtype == "bfloat16" else None
    assert_model_close(replay_modes.portions(runner, tokens, [7, 2, 57, 64, 3, 135, 32]), want, dtype, "portions", spread, rel)
    assert_model_close(replay_modes.portions(runner, tokens, [230] + [1] * 70), want, dtype, "chunks begin among decoded tokens", spread, rel)
    kernels.check_errors()


def test_pages_behind_the_chunks_are_given_back(tmp_path, kernels):
    """A pool too small for the whole request is enough for a model of chunked layers: pages of chunks that are over go back
    and are used again, and the logits are the whole prompt's."""
    runner, config, weights = _runner(tmp_path, kernels, "C", "float32", num_pages=40, max_tokens_per_step=128, max_tokens_per_request=512)
    from kvcache_b200.engine.runner import StepEntry
    tokens = random_tokens(config["vocab"], 300, 7)
    slot = runner.cache.admit()
    got = [runner.step([StepEntry(slot, tokens[:50], list(range(50)))]).clone()]
    for i in range(50, 300):
        got.append(runner.step([StepEntry(slot, tokens[i:i + 1], [0])]).clone())
    runner.cache.release(slot)
    assert runner.cache.used_pages() == 0
    assert_close(torch.cat(got), plain.forward(config, weights, tokens), 1e-4)
    kernels.check_errors()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "E"])
def test_long_decoding_under_graphs_matches_plain(tmp_path, kernels, name, dtype):
    """200 tokens decoded one by one, two requests at a time, replayed from CUDA graphs: chunks begin and end while the same
    launches are replayed."""
    from kvcache_b200.engine.runner import StepEntry
    runner, config, weights = _runner(tmp_path, kernels, name, dtype, num_pages=80, max_slots=2)
    runner.use_graphs = True
    seqs = [random_tokens(config["vocab"], 230, 7), random_tokens(config["vocab"], 215, 8)]
    slots = [runner.cache.admit(), runner.cache.admit()]
    runner.step([StepEntry(slots[0], seqs[0][:30], []), StepEntry(slots[1], seqs[1][:15], [])])
    rows, last = ([], []), None
    for i in range(200):
        entries = [StepEntry(slots[0], [seqs[0][30 + i]], [0], (0.0, 0, i)), StepEntry(slots[1], [seqs[1][15 + i]], [0], (0.0, 0, i))]
        last, tokens = runner.step(entries, sample=True)
        for r in range(2):
            rows[r].append(last[r:r + 1].clone())
    assert runner.graph_replays >= 190
    kernels.check_errors()
    for r in range(2):
        want = plain.forward(config, weights, seqs[r])
        assert_model_close(torch.cat(rows[r]), want[-200:], dtype, f"request {r}", _spread(config, weights, seqs[r], want))
        assert int(tokens[r]) == int(torch.argmax(last[r]))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_entry_point(tmp_path, kernels, dtype):
    """Through `LLM`, the scheduler and CUDA graphs: prompts cut into chunks beside decoding requests, more requests than
    run at once."""
    from kvcache_b200 import LLM, SamplingParams
    folder = make_kunulorn_folder(tmp_path, "A", dtype=torch.bfloat16, all_experts=dtype == "bfloat16")
    config, weights = plain.read_folder(folder)
    prompts = [random_tokens(config["vocab"], n, 40 + n) for n in (1, 9, 24, 40, 63)]
    llm = LLM(folder, kernels=kernels, dtype=dtype, device=DEV, page_size=8, num_pages=80, max_running=3, max_tokens_per_step=48,
              chunk_size=16, use_graphs=True)
    got = llm.generate(prompts, SamplingParams(max_new_tokens=8, ignore_eos=True))
    assert llm.core.cache.used_pages() == 0
    for prompt, out in zip(prompts, got):
        logits = plain.forward(config, weights, list(prompt) + out)
        for i, token in enumerate(out):
            row = logits[len(prompt) - 1 + i]
            best = torch.topk(row, 2).values
            if float(best[0] - best[1]) > (1e-3 if dtype == "float32" else 0.05) * float(row.abs().max()):
                assert token == int(torch.argmax(row)), (len(prompt), i)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_program(tmp_path, dtype):
    """bin/trace_run as a user runs it, on a Kunulorn folder: mixed steps, requests that pause, pages and slots used again."""
    folder = make_kunulorn_folder(tmp_path, "A", dtype=torch.bfloat16, all_experts=dtype == "bfloat16")
    config, weights = plain.read_folder(folder)
    seqs = {k: random_tokens(config["vocab"], n, 20 + i) for i, (k, n) in enumerate([("a", 70), ("b", 33), ("c", 64), ("d", 50)])}
    plan = [([("a", 40), ("b", 2)], []), ([("b", 1), ("c", 64)], ["c"]), ([("a", 1), ("b", 30)], ["b"]), ([("d", 50), ("a", 29)], ["a", "d"])]
    done = {k: 0 for k in seqs}
    lines, expected = [], []
    for step, (parts, end) in enumerate(plan):
        entries = []
        for k, n in parts:
            entries.append({"id": k, "tokens": seqs[k][done[k]:done[k] + n], "want": list(range(n))})
            expected.append((step, k, done[k], n))
            done[k] += n
        lines.append(json.dumps({"step": step, "entries": entries, "end": end}))
    out = os.path.join(str(tmp_path), "out")
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", out,
                           "--max-tokens", "192", "--max-live", "3"], input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(len(plan))]
    want = {k: plain.forward(config, weights, seqs[k]) for k in seqs}
    spread = {k: _spread(config, weights, seqs[k], want[k]) for k in seqs}
    for step in range(len(plan)):
        got = torch.from_numpy(np.fromfile(os.path.join(out, f"{step}.f32"), dtype="<f4").reshape(-1, config["vocab"]))
        at = 0
        for s, k, lo, n in expected:
            if s == step:
                assert_model_close(got[at:at + n], want[k][lo:lo + n], dtype, f"step {step} {k}", spread[k])
                at += n
