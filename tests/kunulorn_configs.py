"""Tiny Kunulorn configurations for the tests: they differ from one another in every size, in the order and kinds of layers,
in chunk sizes, rotation, limits and routing; values that tend to coincide or to be 1 (one key/value head, as many as query
heads, values as wide as keys, narrower and wider ones, one expert chosen, all chosen, one group, groups of one expert, no
groups, no shared expert, a layer without feed-forward, a chunk of one token, of one page, none at all, no rotation, only part
of a head turned, an embedding scale and a weight scale of 1, a layer that reads the keys of a layer that is not the first,
with a smaller chunk, a larger one, one that fits no multiple) each occur somewhere."""
from __future__ import annotations

import copy
import os

import torch


def _attention(heads, kv_heads, dim, vdim, scale, chunk, rot, kv_from=None):
    out = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if chunk is not None:
        out["mask"] = {"size": chunk}
    if rot is not None:
        out["rot"] = {"base": rot[0], "dims": rot[1]}
    if kv_from is not None:
        out["kv_from"] = kv_from
    return out


def _moe(experts, top, ff, shared=None, groups=None, scale=None):
    router = {"experts": experts, "top": top}
    if scale is not None:
        router["scale"] = scale
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    out = {"kind": "moe", "expert": {"ff": ff}, "router": router}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def _dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def _layer(mixer, mlp):
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


# A: every kind of layer; values wider than keys, part of a head turned; the reader's chunk is larger than the owner's and no
# multiple of it.
KUN_A = {
    "architecture": "Kunulorn", "vocab": 211, "width": 72, "norm": {"eps": 1e-6}, "embedding": {"scale": 5.5},
    "layers": [
        _layer(_attention(4, 2, 12, 20, 0.3, 11, (10000.0, 8)), _dense(48, 0.9)),
        _layer(_attention(6, 3, 8, 8, 0.35, 7, (300.0, 8)), _moe(6, 2, 24, 40, (3, 2), 1.7)),
        _layer(_attention(4, 2, 12, 20, 0.25, 19, (10000.0, 8), kv_from=0), _moe(6, 2, 24, 40, (3, 2), 1.7)),
        _layer(_attention(2, 2, 10, 6, 0.4, 16, (77.0, 6)), None),
    ],
}
# B: no chunks and no rotation, one key/value head, values as wide as keys, all experts chosen, one chosen, no groups, groups of
# one expert, no shared expert, scales of 1.
KUN_B = {
    "architecture": "Kunulorn", "vocab": 331, "width": 96, "norm": {"eps": 3e-5},
    "layers": [
        _layer(_attention(5, 1, 24, 24, 0.2, None, None), _moe(3, 3, 40)),
        _layer(_attention(3, 3, 16, 16, 0.25, None, (500.0, 4)), _moe(4, 1, 16, 16, (4, 2), 1.0)),
        _layer(_attention(2, 1, 40, 8, 0.15, 32, (500.0, 40)), _dense(24, 7.0)),
    ],
}
# C: the source of the shared keys is not the first layer; its readers have chunks of other sizes (one of a single token); a
# chunk of one token, chunks of one page.
KUN_C = {
    "architecture": "Kunulorn", "vocab": 150, "width": 40, "norm": {"eps": 1e-5}, "embedding": {"scale": 3.0},
    "layers": [
        _layer(_attention(1, 1, 14, 10, 0.4, 1, (100.0, 6)), _moe(2, 1, 56, 24, (1, 1), 0.8)),
        _layer(_attention(6, 2, 8, 12, 0.5, 12, (3000.0, 4)), None),
        _layer(_attention(6, 2, 8, 12, 0.3, 8, (3000.0, 4), kv_from=1), _dense(32, 0.5)),
        _layer(_attention(6, 2, 8, 12, 0.6, 1, (3000.0, 4), kv_from=1), _dense(32, 0.5)),
        _layer(_attention(6, 2, 8, 12, 0.3, 4, (3000.0, 4), kv_from=1), _moe(4, 2, 20, 12, (2, 1), 3.0)),
    ],
}
# D: a reader without chunks (the entry keeps every key), chunks across pages, many small groups, negative choice scores.
KUN_D = {
    "architecture": "Kunulorn", "vocab": 500, "width": 120, "norm": {"eps": 1e-5}, "embedding": {"scale": 11.0},
    "layers": [
        _layer(_attention(8, 4, 20, 28, 0.2, 24, (50.0, 12)), _moe(12, 3, 24, 72, (6, 3), 2.5)),
        _layer(_attention(8, 4, 20, 28, 0.3, None, (50.0, 12), kv_from=0), _dense(40, 1.3)),
    ],
}
# E: sizes in steps of 16 as real models have them (in bfloat16 the tensor-core kernels): values narrower than keys (cached as
# wide as the keys), keys narrower than values, chunks across pages and of a few pages, shared keys.
KUN_E = {
    "architecture": "Kunulorn", "vocab": 300, "width": 128, "norm": {"eps": 1e-6}, "embedding": {"scale": 8.0},
    "layers": [
        _layer(_attention(4, 2, 64, 48, 0.11, 40, (50000.0, 32)), _dense(192, 1.2)),
        _layer(_attention(2, 1, 32, 64, 0.17, 96, (50000.0, 32)), _moe(8, 2, 32, 64, (4, 2), 1.5)),
        _layer(_attention(4, 2, 64, 48, 0.13, 64, (50000.0, 32), kv_from=0), _moe(8, 2, 32, 64, (4, 2), 1.5)),
        _layer(_attention(4, 4, 64, 64, 0.125, 128, (50000.0, 64)), _dense(192, 1.2)),
    ],
}
CONFIGS = {"A": KUN_A, "B": KUN_B, "C": KUN_C, "D": KUN_D, "E": KUN_E}
PAGE_SIZE = {"A": 8, "B": 16, "C": 4, "D": 16, "E": 16}


def config_dict(name: str, **changes) -> dict:
    out = copy.deepcopy(CONFIGS[name])
    out.update(changes)
    return out


def make_kunulorn_folder(tmp_path, name: str, seed: int = 0, dtype=torch.float32, sharpen: float = 1.0, std: float = 0.08,
                         all_experts: bool = False, data: dict = None) -> str:
    """A random-weights folder for configuration `name` (or for `data`).  `sharpen` multiplies every attention's score scale, so
    that the softmax picks out single keys and a wrong or missing key shows in the logits.  `all_experts`: every routed layer
    chooses all its experts (and keeps all groups) - for comparisons in bfloat16, where rounding may turn a close call between
    two experts the other way than the plain implementation's float64 does."""
    import kvcache_b200  # registers the architectures  # noqa: F401
    from kvcache_b200.config import config_from_dict
    from kvcache_b200.weights import write_random_model
    data = config_dict(name, initializer_range=std) if data is None else dict(copy.deepcopy(data), initializer_range=std)
    for layer in data["layers"]:
        layer["mixer"]["scale"] *= sharpen
        if all_experts and layer["mlp"] is not None and layer["mlp"]["kind"] == "moe":
            router = layer["mlp"]["router"]
            router["top"] = router["experts"]
            if "groups" in router:
                router["groups"]["keep"] = router["groups"]["count"]
    folder = os.path.join(str(tmp_path), f"kun_{name}_{seed}_{sharpen}_{int(all_experts)}")
    write_random_model(folder, config_from_dict(data), seed, dtype)
    return folder
