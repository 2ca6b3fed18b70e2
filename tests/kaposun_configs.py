"""Tiny Kaposun configurations for the tests: they differ from one another in every size, in the order and kinds of layers, in
windows, kept tokens, rotation, loops and scales; values that tend to coincide or to be 1 (one key/value head, as many as query
heads, values as wide as keys, narrower and wider ones, one group, one part of the norm, more parts than heads, a convolution of
one tap, two, five, delta-rule heads that share queries and keys, a layer without feed-forward, a window of one token, no window,
no kept tokens, more of them than the window is wide, no rotation, only part of a head turned, no scaling, a residual multiplier
of 1, no loop, a loop over the last layers, over all, once) each occur somewhere."""
from __future__ import annotations

import copy
import os

import torch


def _attention(heads, kv_heads, dim, vdim, scale, rot=None, mask=None):
    out = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if rot is not None:
        out["rot"] = {"base": rot[0], "dims": rot[1]}
        if len(rot) > 2:
            out["rot"]["scaling"] = {"factor": rot[2]}
    if mask is not None:
        out["mask"] = {"size": mask[0], "keep_first": mask[1]}
    return out


def _delta(heads, kv_heads, dim, vdim, conv, ranks):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "decay_rank": ranks[0], "gate_rank": ranks[1]}


def _full(*args, ff=None, **kw):
    return _layer("attention", _attention(*args, **kw), ff)


def _parallel(left, right, scales, ff=None):
    return _layer("parallel", {"left": left, "right": right, "left_scale": scales[0], "right_scale": scales[1]}, ff)


def _space(heads, vdim, state, groups, parts, conv, ff=None):
    return _layer("mamba2", {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": parts, "conv": conv}, ff)


def _layer(kind, mixer, ff):
    return {"type": kind, "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


# A: every kind of layer; values wider and narrower than keys, delta-rule heads that share keys, a window that is no multiple of a
# page, a loop over the first layers.
KAP_A = {
    "architecture": "Kaposun", "vocab": 203, "width": 72, "norm": {"eps": 1e-5}, "residual_mult": 0.6,
    "layers": [
        _parallel(_attention(4, 2, 12, 20, 0.3, mask=(11, 3)), _delta(4, 2, 10, 14, 4, (6, 9)), (0.7, 1.4), ff=56),
        _full(6, 3, 10, 6, 0.35, rot=(5000.0, 6, 3.0), ff=40),
        _space(6, 8, 10, 3, 2, 3, ff=24),
    ],
    "loop": {"start": 0, "stop": 2, "times": 2},
}
# B: no loop, no scaling, one key/value head, one group, one part, a window of one token that keeps one, a layer without
# feed-forward, a convolution of one tap, a residual multiplier of 1.
KAP_B = {
    "architecture": "Kaposun", "vocab": 331, "width": 96, "norm": {"eps": 3e-5}, "residual_mult": 1.0,
    "layers": [
        _space(3, 20, 7, 1, 1, 1, ff=32),
        _parallel(_attention(5, 1, 16, 16, 0.25, mask=(1, 1)), _delta(3, 1, 12, 12, 2, (5, 5)), (1.0, 1.0)),
        _full(3, 3, 24, 24, 0.2, rot=(300.0, 24), ff=64),
    ],
}
# C: recurrent layers and a window with more kept tokens than it is wide; the loop runs over the last layers; wide convolutions;
# parts of the norm that cross heads.
KAP_C = {
    "architecture": "Kaposun", "vocab": 150, "width": 40, "norm": {"eps": 1e-6}, "residual_mult": 0.45,
    "layers": [
        _space(4, 6, 5, 2, 8, 5, ff=28),
        _parallel(_attention(2, 2, 8, 4, 0.4, mask=(5, 9)), _delta(6, 3, 6, 4, 5, (3, 7)), (1.7, 0.6), ff=20),
        _space(1, 33, 12, 1, 3, 2),
    ],
    "loop": {"start": 1, "stop": 3, "times": 3},
}
# D: a left side without a window, one without kept tokens, whole-head rotation, one delta-rule head, a loop over everything.
KAP_D = {
    "architecture": "Kaposun", "vocab": 400, "width": 120, "norm": {"eps": 1e-5}, "residual_mult": 0.8,
    "layers": [
        _parallel(_attention(8, 4, 20, 28, 0.2), _delta(1, 1, 30, 40, 3, (11, 4)), (0.9, 0.8), ff=88),
        _parallel(_attention(4, 1, 14, 10, 0.3, mask=(24, 0)), _delta(2, 2, 18, 7, 1, (8, 8)), (1.1, 0.5), ff=16),
        _full(8, 2, 18, 18, 0.25, rot=(80.0, 18, 7.5)),
    ],
    "loop": {"start": 0, "stop": 3, "times": 1},
}
# E: sizes in steps of 16 as real models have them (in bfloat16 the tensor-core kernels): values narrower and wider than keys,
# windows over a few pages, kept tokens within one page and over a page's end.
KAP_E = {
    "architecture": "Kaposun", "vocab": 300, "width": 128, "norm": {"eps": 1e-6}, "residual_mult": 0.7,
    "layers": [
        _full(4, 2, 64, 48, 0.11, rot=(50000.0, 32, 4.0), ff=192),
        _parallel(_attention(2, 1, 32, 64, 0.17, mask=(40, 5)), _delta(4, 2, 32, 48, 4, (32, 16)), (1.2, 0.9), ff=192),
        _space(8, 32, 64, 2, 4, 4, ff=160),
        _parallel(_attention(4, 4, 64, 64, 0.125, mask=(100, 20)), _delta(2, 2, 64, 64, 4, (24, 24)), (1.0, 1.3), ff=192),
    ],
    "loop": {"start": 1, "stop": 2, "times": 2},
}
CONFIGS = {"A": KAP_A, "B": KAP_B, "C": KAP_C, "D": KAP_D, "E": KAP_E}
PAGE_SIZE = {"A": 8, "B": 16, "C": 4, "D": 16, "E": 16}


def config_dict(name: str, **changes) -> dict:
    out = copy.deepcopy(CONFIGS[name])
    out.update(changes)
    return out


def enliven(tensors: dict, seed: int = 0) -> dict:
    """Random weights with which every mechanism moves the logits: convolution weights of the size of 1, slow and fast decays
    (log rates around -2, step biases around -1), skips and biases that matter.  Works on a folder's tensors by their names."""
    g = torch.Generator().manual_seed(seed + 77)
    out = {}
    for name, t in tensors.items():
        last = name.rsplit(".", 1)[-1]
        draw = lambda mean, std: (torch.randn(t.shape, generator=g) * std + mean).to(t.dtype)
        if last == "conv":
            t = draw(0.0, 0.7)
        elif last == "A_log":
            t = draw(-1.5, 1.0)
        elif last == "dt_bias":
            t = draw(-1.0, 1.0)
        elif last == "D":
            t = draw(0.5, 0.5)
        elif name.endswith("conv.b"):
            t = draw(0.0, 0.3)
        out[name] = t
    return out


def make_kaposun_folder(tmp_path, name: str, seed: int = 0, dtype=torch.float32, sharpen: float = 1.0, std: float = 0.1,
                        data: dict = None) -> str:
    """A random-weights folder for configuration `name` (or for `data`), enlivened.  `sharpen` multiplies every attention's score
    scale, so that the softmax picks out single keys and a wrong or missing key shows in the logits."""
    import kvcache_b200  # registers the architectures  # noqa: F401
    from kvcache_b200.config import config_from_dict
    from kvcache_b200.weights import write_random_model
    from kvcache_b200.weights.safetensors_io import write_safetensors
    from safetensors.torch import load_file
    data = config_dict(name, initializer_range=std) if data is None else dict(copy.deepcopy(data), initializer_range=std)
    for layer in data["layers"]:
        m = layer["mixer"]
        for side in (m, m.get("left")):
            if side is not None and "scale" in side:
                side["scale"] *= sharpen
    folder = os.path.join(str(tmp_path), f"kap_{name}_{seed}_{sharpen}")
    write_random_model(folder, config_from_dict(data), seed, dtype)
    path = os.path.join(folder, "model.safetensors")
    tensors = {k: v.clone() for k, v in load_file(path).items()}
    write_safetensors(path, enliven(tensors, seed), metadata={"format": "pt"})
    return folder
