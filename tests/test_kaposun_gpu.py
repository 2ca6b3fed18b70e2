"""The Kaposun model through the engine on the GPU, in float32 and bfloat16, against the plain implementation, and every CUDA
operator it brought alone against the plain PyTorch statement of the same operator (tests/torch_kernels.py)."""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_kaposun as plain
import replay_modes
from helpers import assert_close, batch_to, clone_kv, make_runner, paged_scenario, random_tokens
from kaposun_configs import CONFIGS, PAGE_SIZE, make_kaposun_folder
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


def assert_model_close(got, want, dtype, what="", spread=None, rel=1e-4):
    """float32: within `rel` of the largest logit.  bfloat16: the errors are held, as a distribution, to 4 times what rounding
    alone does in the plain implementation (`spread`: its per-position errors over the whole sequence): the k-th largest error
    against the k-th largest of the spread (floor: 1 % of the largest logit) except for the largest 2 % of them (at least one),
    and no position beyond 30 %."""
    if dtype == "float32":
        return assert_close(got, want, rel, what)
    got, want = got.detach().double().cpu(), want.double()
    assert got.shape == want.shape and torch.isfinite(got).all(), what
    scale = float(want.abs().max())
    floor = 0.01 * scale
    err = (got - want).abs().max(dim=1).values
    assert float(err.max()) <= 0.3 * scale, f"{what}: error {float(err.max()):.3e} of {scale:.3e}"
    if len(err) < 16:
        assert float(err.max()) <= max(4.0 * float(spread.max()), 4.0 * floor), f"{what}: error {float(err.max()):.3e}, spread {float(spread.max()):.3e}"
        return
    e, sp = torch.sort(err, descending=True).values, torch.sort(spread, descending=True).values
    like = sp[(torch.arange(len(e)) * len(sp) // len(e))]
    over = e > 4.0 * torch.clamp(like, min=floor)
    over[:max(1, len(e) // 50)] = False
    assert not bool(over.any()), f"{what}: the {int(over.nonzero()[0])}-th largest error {float(e[over][0]):.3e} against {float(like[over][0]):.3e}"


@pytest.fixture(scope="module")
def kernels():
    from kvcache_b200.kernels.api import CudaKernels
    return CudaKernels(DEV)


def _rand(*shape, dtype=torch.float32, seed=0, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(dtype)


def _segments_batch(segments, slots):
    batch, _ = paged_scenario(segments, num_kv_heads=1, head_dim=4, page_size=4, dtype=torch.float32, device="cpu", fill_history=False)
    batch.seg_slot.copy_(torch.tensor(slots, dtype=torch.int32))
    return batch


# ---- operators alone ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("kind", ["gelu", "relu2", "tanh"])
@pytest.mark.parametrize("cols,wide,at", [(129, 129, 0), (64, 200, 8), (61, 90, 13), (4, 4, 0)])
def test_activation_into_columns_of_wider_rows(kernels, dtype, kind, cols, wide, at):
    x = _rand(37, cols, dtype=dtype, seed=4, scale=2.0)
    ref, got = torch.full((37, wide), 5.0).to(dtype), torch.full((37, wide), 5.0).to(dtype).to(DEV)
    TorchKernels(wide=True).activation_into(x, kind, ref, at)
    kernels.activation_into(x.to(DEV), kind, got, at)
    assert_close(got, ref, TOL[dtype])
    assert bool((got[:, :at] == 5.0).all()) and bool((got[:, at + cols:] == 5.0).all())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("kind", ["gelu", "relu2"])
@pytest.mark.parametrize("M", [1, 3, 8, 13, 16, 17, 40, 300])
@pytest.mark.parametrize("N,K,wide,at", [(192, 128, 400, 104), (50, 96, 50, 0), (45, 40, 77, 11), (4864, 896, 6656, 1792)])
def test_product_with_an_activation(kernels, dtype, kind, M, N, K, wide, at):
    """Into columns of wider rows: in the product's epilogue for few rows (bfloat16, K in steps of 32), else in two launches."""
    from kvcache_b200.engine.workspace import Workspace
    x, w = _rand(M, K, dtype=dtype, seed=1), _rand(N, K, dtype=dtype, seed=2, scale=0.2)
    ref, got = torch.full((M, wide), 5.0).to(dtype), torch.full((M, wide), 5.0).to(dtype).to(DEV)
    TorchKernels(wide=True).linear_act(x, w, kind, ref, at)
    before = kernels.launches
    kernels.linear_act(x.to(DEV), w.to(DEV), kind, got, at, Workspace(DEV))
    if dtype == torch.bfloat16 and K % 32 == 0:
        assert kernels.launches - before == (1 if M <= 16 else 2)
    assert_close(got, ref, TOL[dtype])
    assert bool((got[:, :at] == 5.0).all()) and bool((got[:, at + N:] == 5.0).all())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("per_channel", [True, False, None])
@pytest.mark.parametrize("H,Dv,xs,g_col,wide,at", [(3, 16, 16, 8, 80, 16), (4, 5, 9, 3, 40, 7), (14, 64, 64, 1152, 6656, 0), (2, 48, 64, 0, 96, 0)])
def test_head_gate_per_head_and_per_channel(kernels, dtype, per_channel, H, Dv, xs, g_col, wide, at):
    T = 23
    x, g = _rand(T, H * xs, dtype=dtype, seed=1), _rand(T, g_col + H * Dv + 8, dtype=dtype, seed=2, scale=2.0)
    gate = None if per_channel is None else (g, g_col)
    ref, got = torch.full((T, wide), 5.0).to(dtype), torch.full((T, wide), 5.0).to(dtype).to(DEV)
    extra = {"x_head_stride": xs, "per_channel": bool(per_channel)}
    TorchKernels(wide=True).head_gate(x, gate, H, Dv, 0.7, ref, at, **extra)
    kernels.head_gate(x.to(DEV), None if gate is None else (g.to(DEV), g_col), H, Dv, 0.7, got, at, **extra)
    assert_close(got, ref, TOL[dtype])
    assert bool((got[:, :at] == 5.0).all()) and bool((got[:, at + H * Dv:] == 5.0).all())


SEGMENTS, SLOTS = [(0, 19), (50, 1), (7, 6), (3, 1), (9, 2)], [2, 0, 3, 5, 1]
LONG_SEGMENTS, LONG_SLOTS = [(0, 101), (9, 1), (4, 2), (30, 1), (3, 50)], [1, 3, 0, 2, 5]      # tiles of rows that hold several segments
SINGLES, SINGLE_SLOTS = [(4, 1), (0, 1), (77, 1)], [3, 1, 4]


def _delta_case(segments, H, G, D, Dv, taps, seed=1, pad=3, z_pad=5):
    """(T, proj, weights..., tail): rows with the columns of a delta mixer's projections; every slot's state holds something."""
    T, C = sum(n for _, n in segments), 2 * G * D + H * Dv
    return dict(proj=_rand(T, C + H + pad, seed=seed), conv_w=_rand(taps, C, seed=seed + 1), tail=_rand(6, taps - 1, C, seed=seed + 2),
                z=_rand(T, H * D + z_pad, seed=seed + 3, scale=2.0), dt_bias=_rand(H * D, seed=seed + 4), rate=_rand(H, seed=seed + 5).exp())


def _to(case, device):
    return {k: v.clone().to(device) for k, v in case.items()}


@pytest.mark.parametrize("H,G,D,Dv,taps", [(4, 2, 8, 12, 4), (3, 3, 33, 5, 2), (6, 1, 64, 64, 1), (2, 2, 128, 48, 5), (1, 1, 256, 16, 3), (2, 1, 200, 130, 4), (16, 16, 64, 64, 4)])
@pytest.mark.parametrize("segments,slots", [(SEGMENTS, SLOTS), (SINGLES, SINGLE_SLOTS), (LONG_SEGMENTS, LONG_SLOTS)])
def test_gated_delta_inputs(kernels, H, G, D, Dv, taps, segments, slots):
    """Convolutions over portions (shorter and longer than the taps) and single tokens, unit queries and keys, decays, write
    strengths; the convolutions' state afterwards, other slots untouched."""
    batch = _segments_batch(segments, slots)
    T, C = batch.num_tokens, 2 * G * D + H * Dv
    case = _delta_case(segments, H, G, D, Dv, taps)
    ref, got = _to(case, "cpu"), _to(case, DEV)
    outs = []
    for k, c, b, dev in ((TorchKernels(wide=True), ref, batch, "cpu"), (kernels, got, batch_to(batch, DEV), DEV)):
        rows, gates = torch.zeros(T, C, device=dev), torch.zeros(T, H * D + H, device=dev)
        k.gated_delta_inputs(c["proj"], C, c["conv_w"], c["tail"], c["z"], c["dt_bias"], c["rate"], 1e-6, b, rows, gates, H, G, D, Dv)
        outs.append((rows, gates))
    assert_close(outs[1][0], outs[0][0], 1e-5, "rows")
    assert_close(outs[1][1], outs[0][1], 1e-5, "gates")
    assert torch.equal(got["tail"].cpu(), ref["tail"]) and torch.equal(got["proj"].cpu(), case["proj"])
    untouched = [s for s in range(6) if s not in slots]
    assert torch.equal(got["tail"].cpu()[untouched], case["tail"][untouched])


@pytest.mark.parametrize("H,C,taps,col", [(4, 100, 4, 7), (3, 128, 1, 0), (30, 300, 2, 64), (2, 17, 6, 3)])
@pytest.mark.parametrize("segments,slots", [(SEGMENTS, SLOTS), (SINGLES, SINGLE_SLOTS), (LONG_SEGMENTS, LONG_SLOTS)])
def test_state_space_inputs(kernels, H, C, taps, col, segments, slots):
    batch = _segments_batch(segments, slots)
    T = batch.num_tokens
    case = dict(proj=_rand(T, col + C + H + 5, seed=1, scale=2.0), conv_w=_rand(taps, C, seed=2), conv_b=_rand(C, seed=3), tail=_rand(6, taps - 1, C, seed=4),
                dt_bias=_rand(H, seed=5), rate=_rand(H, seed=6).exp())
    ref, got = _to(case, "cpu"), _to(case, DEV)
    outs = []
    for k, c, b, dev in ((TorchKernels(wide=True), ref, batch, "cpu"), (kernels, got, batch_to(batch, DEV), DEV)):
        rows, gates = torch.zeros(T, C, device=dev), torch.zeros(T, 2 * H, device=dev)
        k.state_space_inputs(c["proj"], col, col + C, c["conv_w"], c["conv_b"], c["tail"], c["dt_bias"], c["rate"], b, rows, gates, H)
        outs.append((rows, gates))
    assert_close(outs[1][0], outs[0][0], 1e-5, "rows")
    assert_close(outs[1][1], outs[0][1], 1e-5, "gates")
    assert torch.equal(got["tail"].cpu(), ref["tail"])


def _delta_rows(T, H, G, D, Dv, seed=1):
    rows = _rand(T, 2 * G * D + H * Dv, seed=seed)
    qk = rows[:, :2 * G * D].view(T, 2 * G, D)
    rows[:, :2 * G * D] = (qk / qk.norm(dim=-1, keepdim=True)).reshape(T, -1)
    gates = torch.cat([torch.exp(-torch.rand(T, H * D, generator=torch.Generator().manual_seed(seed + 1)) * 0.3),
                       torch.rand(T, H, generator=torch.Generator().manual_seed(seed + 2))], dim=1)
    return rows, gates


def _space_rows(T, H, G, N, Dv, seed=1):
    gates = torch.cat([torch.exp(-torch.rand(T, H, generator=torch.Generator().manual_seed(seed + 1)) * 0.3),
                       torch.rand(T, H, generator=torch.Generator().manual_seed(seed + 2))], dim=1)
    return _rand(T, H * Dv + 2 * G * N, seed=seed), gates


def _run_scan(k, kind, rows, gates, batch, memory, sizes):
    from kvcache_b200.engine.workspace import Workspace
    out = torch.zeros(rows.shape[0], sizes[0] * sizes[3], device=rows.device)
    if kind == "delta":
        k.gated_delta_scan(rows, gates, 0.3, batch, memory, out, *sizes, Workspace(out.device))
    else:
        k.state_space_scan(rows, gates, batch, memory, out, *sizes)
    return out


@pytest.mark.parametrize("kind", ["delta", "space"])
@pytest.mark.parametrize("H,G,D,Dv", [(4, 2, 8, 12), (1, 1, 33, 40), (6, 3, 64, 64), (2, 2, 128, 128), (3, 1, 200, 20), (5, 5, 6, 70), (2, 1, 100, 300)])
def test_scans(kernels, kind, H, G, D, Dv):
    """Prompts, portions that continue a state, single tokens, states of other slots untouched; then every row alone, which must
    give the same bits as the rows together."""
    batch = _segments_batch(SEGMENTS, SLOTS)
    T = batch.num_tokens
    rows, gates = (_delta_rows if kind == "delta" else _space_rows)(T, H, G, D, Dv)
    memory = _rand(6, H, D, Dv, seed=3)
    ref_mem, got_mem, one_mem = memory.clone(), memory.clone().to(DEV), memory.clone().to(DEV)
    sizes = (H, G, D, Dv)
    want = _run_scan(TorchKernels(wide=True), kind, rows, gates, batch, ref_mem, sizes)
    got = _run_scan(kernels, kind, rows.to(DEV), gates.to(DEV), batch_to(batch, DEV), got_mem, sizes)
    assert_close(got, want, 2e-5, "read-out")
    assert_close(got_mem, ref_mem, 2e-5, "states")
    assert torch.equal(got_mem[4].cpu(), memory[4])
    at = 0
    for (start, n), slot in zip(SEGMENTS, SLOTS):
        for i in range(n):
            single = batch_to(_segments_batch([(start + i, 1)], [slot]), DEV)
            one = _run_scan(kernels, kind, rows[at:at + 1].to(DEV), gates[at:at + 1].to(DEV), single, one_mem, sizes)
            assert torch.equal(one, got[at:at + 1])
            at += 1
    assert torch.equal(one_mem, got_mem)


@pytest.mark.parametrize("kind", ["delta", "space"])
@pytest.mark.parametrize("H,G,D,Dv", [(4, 2, 64, 64), (1, 1, 33, 40), (2, 1, 128, 64), (3, 3, 8, 12), (2, 2, 200, 48), (2, 2, 128, 128), (2, 1, 100, 45),
                                       (3, 1, 70, 5), (1, 1, 256, 33)])
@pytest.mark.parametrize("shorter", [False, True])
def test_scans_of_long_portions(kernels, kind, H, G, D, Dv, shorter):
    """Portions for the scan that spreads a column over many lanes and for the one in chunks: many tiles of tokens, from an empty
    state and from a filled one, lengths that are no multiple of a tile or a group, beside single tokens and short portions;
    against the plain recurrence, and every segment alone, which must give the same bits (in the forms without chunks)."""
    segments, slots = [(0, 120 if shorter else 300), (50, 1), (100, 97 if shorter else 257), (3, 1), (0, 64), (5, 2)], [2, 0, 3, 5, 1, 4]
    batch = _segments_batch(segments, slots)
    T = batch.num_tokens
    rows, gates = (_delta_rows if kind == "delta" else _space_rows)(T, H, G, D, Dv)
    memory = _rand(7, H, D, Dv, seed=3)
    memory[2].zero_()
    ref_mem, got_mem = memory.clone(), memory.clone().to(DEV)
    sizes = (H, G, D, Dv)
    want = _run_scan(TorchKernels(wide=True), kind, rows, gates, batch, ref_mem, sizes)
    got = _run_scan(kernels, kind, rows.to(DEV), gates.to(DEV), batch_to(batch, DEV), got_mem, sizes)
    kernels.check_errors()
    assert_close(got, want, 1e-4, "read-out")
    assert_close(got_mem, ref_mem, 1e-4, "states")
    assert torch.equal(got_mem[6].cpu(), memory[6])
    if kind == "space" or D > kernels.DELTA_WIDE_ABOVE or shorter:
        at, alone_mem = 0, memory.clone().to(DEV)
        for (start, n), slot in zip(segments, slots):
            if n >= kernels.SCAN_WIDE_MIN_ROWS:
                alone = batch_to(_segments_batch([(start, n)], [slot]), DEV)
                assert torch.equal(_run_scan(kernels, kind, rows[at:at + n].to(DEV), gates[at:at + n].to(DEV), alone, alone_mem, sizes), got[at:at + n])
                assert torch.equal(alone_mem[slot], got_mem[slot])
            at += n


@pytest.mark.parametrize("D", [64, 96])
def test_forms_of_the_delta_scan_agree(kernels, D):
    """In one piece, in chunks, spread over lanes: the same read-outs and states up to rounding."""
    H, G, Dv = 2, 1, 40
    segments = [(0, 300), (4, 70)]
    rows, gates = (t.to(DEV) for t in _delta_rows(370, H, G, D, Dv))
    batch = batch_to(_segments_batch(segments, [1, 0]), DEV)
    saved, results = (kernels.DELTA_WIDE_ABOVE, kernels.SCAN_CHUNK, kernels.SCAN_WIDE_MIN_ROWS), []
    try:
        for above, chunk, rows_wide in ((0, 64, 48), (256, 64, 48), (256, 0, 1 << 30)):
            kernels.DELTA_WIDE_ABOVE, kernels.SCAN_CHUNK, kernels.SCAN_WIDE_MIN_ROWS = above, chunk, rows_wide
            memory = _rand(2, H, D, Dv, seed=3).to(DEV)
            results.append((_run_scan(kernels, "delta", rows, gates, batch, memory, (H, G, D, Dv)), memory))
    finally:
        kernels.DELTA_WIDE_ABOVE, kernels.SCAN_CHUNK, kernels.SCAN_WIDE_MIN_ROWS = saved
    for out, memory in results[1:]:
        assert_close(out, results[0][0], 1e-5)
        assert_close(memory, results[0][1], 1e-5)


@pytest.mark.parametrize("kind", ["delta", "space"])
@pytest.mark.parametrize("fast", [False, True])
def test_scans_of_a_very_long_portion_with_slow_and_with_fast_decays(kernels, kind, fast):
    """Decays that hardly forget (early tokens reach the last read-outs) and decays that underflow within a few tokens."""
    H, G, D, Dv = 2, 2, 64, 64
    segments, slots = [(10, 1613), (0, 130), (5, 1)], [1, 0, 2]
    batch = _segments_batch(segments, slots)
    T = batch.num_tokens
    rows, gates = (_delta_rows if kind == "delta" else _space_rows)(T, H, G, D, Dv)
    keep = gates[:, :H * D] if kind == "delta" else gates[:, :H]
    keep.copy_(keep ** (150.0 if fast else 0.01))
    memory = _rand(3, H, D, Dv, seed=3)
    ref_mem, got_mem = memory.clone(), memory.clone().to(DEV)
    want = _run_scan(TorchKernels(wide=True), kind, rows, gates, batch, ref_mem, (H, G, D, Dv))
    got = _run_scan(kernels, kind, rows.to(DEV), gates.to(DEV), batch_to(batch, DEV), got_mem, (H, G, D, Dv))
    kernels.check_errors()
    assert_close(got, want, 2e-4, "read-out")
    assert_close(got_mem, ref_mem, 2e-4, "states")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,Dv,parts,x_wide,g_col,wide,at", [(4, 6, 3, 30, 2, 40, 5), (28, 64, 1, 2048, 0, 5760, 0), (5, 33, 15, 165, 0, 165, 0), (8, 1600, 2, 12800, 0, 12800, 0)])
def test_gate_part_norm(kernels, dtype, H, Dv, parts, x_wide, g_col, wide, at):
    T, W = 11, H * Dv
    o, x, g = _rand(T, W, seed=1), _rand(T, x_wide, seed=2), _rand(T, g_col + W + 3, seed=3, scale=2.0)
    skip, weight = _rand(H, seed=4), 1 + _rand(W, seed=5, scale=0.3)
    ref, got = torch.full((T, wide), 5.0).to(dtype), torch.full((T, wide), 5.0).to(dtype).to(DEV)
    TorchKernels(wide=True).gate_part_norm(o, x, skip, (g, g_col), weight, 1e-5, 0.8, ref, at, H, Dv, parts)
    kernels.gate_part_norm(o.to(DEV), x.to(DEV), skip.to(DEV), (g.to(DEV), g_col), weight.to(DEV), 1e-5, 0.8, got, at, H, Dv, parts)
    assert_close(got, ref, TOL[dtype])
    assert bool((got[:, :at] == 5.0).all()) and bool((got[:, at + W:] == 5.0).all())


def test_sizes_that_do_not_fit_are_refused(kernels):
    from kvcache_b200.kernels.api import KernelError
    batch = batch_to(_segments_batch([(0, 2)], [0]), DEV)
    rows, gates = (t.to(DEV) for t in _delta_rows(2, 2, 1, 8, 8))
    out = torch.zeros(2, 16, device=DEV)
    with pytest.raises(KernelError):
        kernels.gated_delta_scan(rows, gates, 1.0, batch, torch.zeros(1, 2, 8, 9, device=DEV), out, 2, 1, 8, 8, None)
    with pytest.raises(KernelError):
        kernels.gated_delta_scan(rows, gates.double(), 1.0, batch, torch.zeros(1, 2, 8, 8, device=DEV), out, 2, 1, 8, 8, None)
    with pytest.raises(KernelError):
        kernels.gate_part_norm(out, out, torch.zeros(2, device=DEV), (out, 0), torch.ones(16, device=DEV), 1e-5, 1.0, out.clone(), 0, 2, 8, 3)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("decoded", [True, False])
@pytest.mark.parametrize("D,Dv,page,window,keep,last,portion", [(32, 48, 8, 25, 16, 200, 11), (64, 64, 16, 300, 144, 2000, 400), (128, 128, 32, 100, 64, 1500, 130),
                                                                 (48, 48, 16, 64, 3, 700, 33), (64, 64, 16, 1, 1, 300, 20)])
def test_one_key_at_an_edge_takes_all_the_weight(kernels, dtype, decoded, D, Dv, page, window, keep, last, portion):
    """Without a sink: the query of one head matches the window's first key, then the last kept key, and the head's result is
    that key's value, also where a key just outside the edge matches still more strongly."""
    from kvcache_b200.engine.workspace import Workspace
    from kvcache_b200.parts.base import PagedKVSpec, PagedKVView
    Hq, Hkv = 4, 2
    segments = [(last, 1), (5, 1)] if decoded else [(last - portion + 1, portion), (0, 6)]
    row, pos = (0, last) if decoded else (portion - 2, last - 1)
    for inside, outside in ((pos - window + 1, pos - window), (keep - 1, keep)):
        for head, strong_outside in ((1, False), (2, True)):
            batch, kv = paged_scenario(segments, num_kv_heads=Hkv, head_dim=D, page_size=page, dtype=dtype, device="cpu", seed=6, window=window)
            kv = PagedKVView(spec=PagedKVSpec(Hkv, D, window, None if Dv == D else Dv, keep), k_pages=kv.k_pages,
                             v_pages=_rand(*kv.k_pages.shape[:-1], Dv, dtype=dtype, seed=7), block_table=kv.block_table, page_size=page, writes=True)
            T, hk = batch.num_tokens, head // 2
            at = lambda pool, p: pool[int(kv.block_table[0, p // page]), hk, p % page]
            q = (_rand(T, Hq * D, seed=7) * 0.01).to(dtype)
            q.view(T, Hq, D)[row, head] = (at(kv.k_pages, inside).float() * 2.0).to(dtype)
            if strong_outside:
                at(kv.k_pages, outside).copy_((at(kv.k_pages, inside).float() * 1.5).to(dtype))
            got = torch.zeros(T, Hq * Dv, dtype=dtype, device=DEV)
            kernels.paged_attention(q.to(DEV), batch_to(batch, DEV), clone_kv(kv, DEV), got, Hq, 1.0, Workspace(DEV))
            kernels.check_errors()
            assert_close(got.view(T, Hq, Dv)[row, head], at(kv.v_pages, inside), TOL[torch.bfloat16] if dtype == torch.bfloat16 else 1e-4, f"key {inside}, head {head}")


# ---- the model in the engine ------------------------------------------------------------------------------------------
def _runner(tmp_path, kernels, name, dtype, num_pages=64, sharpen=1.0, data=None, **kw):
    folder = make_kaposun_folder(tmp_path, name, sharpen=sharpen, dtype=torch.bfloat16, data=data)
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


@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_float32_rows_do_not_depend_on_the_batch_or_the_cut(tmp_path, kernels, name):
    """In float32 a position's logits are bit for bit the same alone, beside other requests, and in (short) portions."""
    runner, config, _ = _runner(tmp_path, kernels, name, "float32")
    from kvcache_b200.engine.runner import StepEntry
    a, b = random_tokens(config["vocab"], 40, 1), random_tokens(config["vocab"], 23, 2)
    alone = replay_modes.whole(runner, a)
    sa, sb = runner.cache.admit(), runner.cache.admit()
    first = runner.step([StepEntry(sb, b[:20], []), StepEntry(sa, a[:17], list(range(17)))]).clone()
    second = runner.step([StepEntry(sa, a[17:], list(range(23))), StepEntry(sb, b[20:21], [0])]).clone()
    assert torch.equal(torch.cat([first, second[:23]]), alone)


@pytest.mark.parametrize("name", ["A", "C", "E"])
def test_long_prompts(tmp_path, kernels, name):
    """float32: a prompt of several hundred tokens whole, in two long portions and beside another request; then decoded tokens
    behind it."""
    from kvcache_b200.engine.runner import StepEntry
    runner, config, weights = _runner(tmp_path, kernels, name, "float32", num_pages=160, max_tokens_per_step=700, max_tokens_per_request=700)
    tokens, other = random_tokens(config["vocab"], 500, 11), random_tokens(config["vocab"], 90, 12)
    want = plain.forward(config, weights, tokens)
    assert_close(replay_modes.whole(runner, tokens), want, 2e-4, "whole")
    assert_close(replay_modes.portions(runner, tokens, [261, 239]), want, 2e-4, "two portions")
    assert_close(replay_modes.portions(runner, tokens, [470] + [1] * 30), want, 2e-4, "decoded behind a long prompt")
    sa, sb = runner.cache.admit(), runner.cache.admit()
    got = runner.step([StepEntry(sb, other[:60], []), StepEntry(sa, tokens[:333], list(range(333)))]).clone()
    more = runner.step([StepEntry(sa, tokens[333:], list(range(167))), StepEntry(sb, other[60:], [29])]).clone()
    assert_close(torch.cat([got, more[:167]]), want, 2e-4, "beside another request")
    assert_close(more[167:], plain.forward(config, weights, other)[-1:], 2e-4, "the other request")
    kernels.check_errors()


def test_a_long_prompt_in_bfloat16(tmp_path, kernels):
    """E through the tensor-core kernels: chunked scans, tensor-memory attention over a window with kept tokens."""
    runner, config, weights = _runner(tmp_path, kernels, "E", "bfloat16", num_pages=160, max_tokens_per_step=700, max_tokens_per_request=700)
    tokens = random_tokens(config["vocab"], 500, 11)
    want = plain.forward(config, weights, tokens)
    spread = _spread(config, weights, tokens, want)
    before = dict(kernels.launch_counts)
    assert_model_close(replay_modes.whole(runner, tokens), want, "bfloat16", "whole", spread)
    used = {n for n, c in kernels.launch_counts.items() if c > before.get(n, 0)}
    assert "attention_tc" in used and not used & {"attention_generic", "attention_sink", "gemm_simt"}, used
    assert_model_close(replay_modes.portions(runner, tokens, [261, 2, 197] + [1] * 40), want, "bfloat16", "portions and decoded", spread)
    kernels.check_errors()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "E"])
def test_sharp_attention_at_the_edges(tmp_path, kernels, name, dtype):
    """Sharpened scores make single keys carry the softmax: a window or a run of kept tokens one token off, or a key lost at a
    page border, shows.  bfloat16 is sharpened less (its single keys are met at kernel level)."""
    sharpen, rel = (12.0, 1e-3) if dtype == "float32" else (2.0, None)
    runner, config, weights = _runner(tmp_path, kernels, name, dtype, sharpen=sharpen, num_pages=96, max_tokens_per_step=320, max_tokens_per_request=320)
    tokens = random_tokens(config["vocab"], 240, 5)
    want = plain.forward(config, weights, tokens)
    if dtype == "float32":
        for key, delta in (("size", -1), ("size", 1), ("keep_first", -1), ("keep_first", 1)):
            other = copy.deepcopy(config)
            for layer in other["layers"]:
                mask = layer["mixer"].get("left", {}).get("mask")
                if mask:
                    mask[key] = max(1 if key == "size" else 0, mask[key] + delta)
            if other != config:
                assert (plain.forward(other, weights, tokens) - want).abs().max() > 5 * rel * want.abs().max(), (key, delta)
    spread = _spread(config, weights, tokens, want) if dtype == "bfloat16" else None
    assert_model_close(replay_modes.portions(runner, tokens, [7, 2, 57, 64, 3, 75, 32]), want, dtype, "portions", spread, rel)
    assert_model_close(replay_modes.portions(runner, tokens, [180] + [1] * 60), want, dtype, "the window passes over decoded tokens", spread, rel)
    kernels.check_errors()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "E"])
def test_long_decoding_under_graphs_matches_plain(tmp_path, kernels, name, dtype):
    """200 tokens decoded one by one, two requests at a time, replayed from CUDA graphs: every state (matrices, the convolutions'
    inputs, pages, kept first tokens, those of every pass of the loop) moves exactly once a step."""
    from kvcache_b200.engine.runner import StepEntry
    runner, config, weights = _runner(tmp_path, kernels, name, dtype, num_pages=80, max_slots=2)
    runner.use_graphs = True
    seqs = [random_tokens(config["vocab"], 230, 7), random_tokens(config["vocab"], 215, 8)]
    slots = [runner.cache.admit(), runner.cache.admit()]
    runner.step([StepEntry(slots[0], seqs[0][:30], []), StepEntry(slots[1], seqs[1][:15], [])])
    last = None
    for i in range(200):
        entries = [StepEntry(slots[0], [seqs[0][30 + i]], [0], (0.0, 0, i)), StepEntry(slots[1], [seqs[1][15 + i]], [0], (0.0, 0, i))]
        last, tokens = runner.step(entries, sample=True)
    assert runner.graph_replays >= 190
    kernels.check_errors()
    for r in range(2):
        want = plain.forward(config, weights, seqs[r])
        assert_model_close(last[r:r + 1], want[-1:], dtype, f"request {r}", _spread(config, weights, seqs[r], want))
        assert int(tokens[r]) == int(torch.argmax(last[r]))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions_under_graphs(tmp_path, kernels, dtype):
    """A portion's shape that comes again and again is replayed: the convolutions' state moves on in a launch of its own, which
    the graph must hold."""
    from kvcache_b200.engine.runner import StepEntry
    runner, config, weights = _runner(tmp_path, kernels, "A", dtype)
    runner.use_graphs = True
    tokens = random_tokens(config["vocab"], 140, 4)
    want = plain.forward(config, weights, tokens)
    spread = _spread(config, weights, tokens, want)
    for _ in range(2):
        slot, got = runner.cache.admit(), []
        for at in range(0, 140, 14):
            got.append(runner.step([StepEntry(slot, tokens[at:at + 14], list(range(14)))]).clone())
        runner.cache.release(slot)
        assert_model_close(torch.cat(got), want, dtype, "portions of 14", spread)
    assert runner.graph_replays >= 8
    kernels.check_errors()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_entry_point(tmp_path, kernels, dtype):
    """Through `LLM`, the scheduler and CUDA graphs: prompts cut into chunks beside decoding requests, more requests than run at
    once."""
    from kvcache_b200 import LLM, SamplingParams
    folder = make_kaposun_folder(tmp_path, "A", dtype=torch.bfloat16)
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
    """bin/trace_run as a user runs it, on a Kaposun folder: mixed steps, requests that pause, pages and slots used again."""
    folder = make_kaposun_folder(tmp_path, "A", dtype=torch.bfloat16)
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
