"""Plain, slow implementation of the Kunulorn decoder: whole sequences, no cache, one function for each mechanism, float64
by default.  It shares no code with `kvcache_b200` (it reads the model folder with the `safetensors` package and `json`)
and states every formula directly.

The design, in this file's notation.  W = width, residual stream x[T, W].

* embedding: x_t = s embed[tok_t], s = embedding.scale.
* centred norm: N(x; w) = (x - mu) / sqrt(mean((x - mu)^2) + eps) * w, mu = mean(x); no bias.
* layer: x += mixer(N(x; norm1)); x += ff(N(x; norm2)) (the second only if the layer has a feed-forward).
* attention: q = Wq h + bq, k = Wk h + bk, v = Wv h + bv (kv_heads keys and values; query head h uses number
  h div (heads / kv_heads)).  All of a token's q numbers together are divided by sqrt(mean(q^2) + eps) and multiplied by a
  weight of that size; k likewise with its own.  Then, per head, the neighbours (2 t, 2 t + 1) of the first rot.dims numbers
  are turned by the angle p base^(-2 t / dims).  s_ij = scale q_i . k_j over the keys j <= i of i's chunk,
  i div size = j div size; softmax; out = Wo concat + bo.  A layer with `kv_from` = j takes layer j's k (normalised and
  turned) and v of the same tokens and has only q, its norm and the output matrix of its own, with its own chunk size.
* dense feed-forward: g = min(Wgate h, L), u = max(-L, min(L, Wup h)); Wdown (g sigmoid(1.702 g) (u + 1)).
* routed feed-forward: s = sigmoid(Wrouter h), c = s + correction.  The experts form `count` runs of equal length; a run's
  value is the sum of its two largest c; the `keep` runs with the largest values stay, and among their experts the `top`
  with the largest c are chosen; weights = scale s / (sum of the chosen s + 1e-20).  expert(h) = Wdown (silu(Wgate h)
  (Wup h)); a shared expert of the same form, times sigmoid(Wsg h) (one number per token), is added for every token.
* logits = embed N(x; final.norm) (the table without s).
"""
from __future__ import annotations

import contextlib
import json
import os
from typing import Dict, List, Optional, Sequence

import torch
from safetensors import safe_open


def read_folder(folder: str, dtype: torch.dtype = torch.float64):
    with open(os.path.join(folder, "config.json"), "r", encoding="utf-8") as fh:
        config = json.load(fh)
    weights: Dict[str, torch.Tensor] = {}
    with safe_open(os.path.join(folder, "model.safetensors"), framework="pt", device="cpu") as f:
        for name in f.keys():
            weights[name] = f.get_tensor(name).to(dtype)
    return config, weights


_ROUND_TO: Optional[torch.dtype] = None


@contextlib.contextmanager
def rounding(dtype: torch.dtype = torch.bfloat16):
    """Within the block every matrix product rounds its input rows and its result to `dtype` (the arithmetic stays as
    wide as the weights): what rounding alone does to a position's logits."""
    global _ROUND_TO
    saved, _ROUND_TO = _ROUND_TO, dtype
    try:
        yield
    finally:
        _ROUND_TO = saved


def linear(x: torch.Tensor, weight: torch.Tensor, bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    if _ROUND_TO is None:
        y = x @ weight.t()
    else:
        y = (x.to(_ROUND_TO).to(weight.dtype) @ weight.t()).to(_ROUND_TO).to(weight.dtype)
    return y if bias is None else y + bias


# ---- norms ------------------------------------------------------------------------------------------------------------
def centred_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * weight


def whole_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    """Over all of a token's numbers at once, before they are split into heads."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * weight


# ---- attention --------------------------------------------------------------------------------------------------------
def rotate_pairs(x: torch.Tensor, positions: torch.Tensor, rot: Optional[dict]) -> torch.Tensor:
    """x [T, heads, D]: of each head's first rot.dims numbers, neighbours (2 t, 2 t + 1) are turned by p base^(-2 t / dims)."""
    if not rot:
        return x
    dims, base = int(rot["dims"]), float(rot["base"])
    out = x.clone()
    for t in range(dims // 2):
        angle = positions.to(torch.float64) * base ** (-2.0 * t / dims)
        c, s = torch.cos(angle)[:, None].to(x.dtype), torch.sin(angle)[:, None].to(x.dtype)
        u, v = x[..., 2 * t], x[..., 2 * t + 1]
        out[..., 2 * t], out[..., 2 * t + 1] = u * c - v * s, v * c + u * s
    return out


def first_in_chunk(i: int, size: Optional[int]) -> int:
    return 0 if not size else i - i % size


def attention_kv(m: dict, w: Dict[str, torch.Tensor], p: str, h: torch.Tensor, positions: torch.Tensor, eps: float):
    """What a layer keeps per token: keys [T, kv_heads, dim], normalised and turned, and values [T, kv_heads, vdim]."""
    T = h.shape[0]
    G, dim, vdim = (int(m[k]) for k in ("kv_heads", "dim", "vdim"))
    k = whole_norm(linear(h, w[p + "k"], w[p + "k.b"]), w[p + "k.norm"], eps).view(T, G, dim)
    v = linear(h, w[p + "v"], w[p + "v.b"]).view(T, G, vdim)
    return rotate_pairs(k, positions, m.get("rot")), v


def attention(m: dict, w: Dict[str, torch.Tensor], p: str, h: torch.Tensor, positions: torch.Tensor, eps: float, kept=None):
    """`kept`: (keys, values) of the layer named by `kv_from`, or None for a layer with its own.  Returns (out, (keys, values))."""
    T = h.shape[0]
    H, G, dim, vdim = (int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
    size = int(m["mask"]["size"]) if m.get("mask") else None
    k, v = kept if kept is not None else attention_kv(m, w, p, h, positions, eps)
    q = whole_norm(linear(h, w[p + "q"], w[p + "q.b"]), w[p + "q.norm"], eps).view(T, H, dim)
    q = rotate_pairs(q, positions, m.get("rot"))
    out = torch.zeros(T, H, vdim, dtype=h.dtype)
    for i in range(T):
        lo = first_in_chunk(i, size)
        for head in range(H):
            g = head // (H // G)
            s = (k[lo:i + 1, g] @ q[i, head]) * float(m["scale"])
            out[i, head] = torch.softmax(s, dim=0) @ v[lo:i + 1, g]
    return linear(out.reshape(T, H * vdim), w[p + "o"], w[p + "o.b"]), (k, v)


# ---- feed-forwards ----------------------------------------------------------------------------------------------------
def dense_ff(mlp: dict, w: Dict[str, torch.Tensor], p: str, h: torch.Tensor) -> torch.Tensor:
    limit = float(mlp["limit"])
    g = torch.clamp(linear(h, w[p + "gate"]), max=limit)
    u = torch.clamp(linear(h, w[p + "up"]), min=-limit, max=limit)
    return linear(g * torch.sigmoid(1.702 * g) * (u + 1.0), w[p + "down"])


def gated_expert(w: Dict[str, torch.Tensor], p: str, h: torch.Tensor) -> torch.Tensor:
    g = linear(h, w[p + "gate"])
    return linear(g * torch.sigmoid(g) * linear(h, w[p + "up"]), w[p + "down"])


def choose(scores: torch.Tensor, correction: torch.Tensor, router: dict) -> List[int]:
    """The experts one token uses, from its scores [experts]."""
    c = scores + correction
    allowed = list(range(len(c)))
    groups = router.get("groups")
    if groups:
        size = len(c) // int(groups["count"])
        value = [float(torch.topk(c[g * size:(g + 1) * size], min(2, size)).values.sum()) for g in range(int(groups["count"]))]
        best = sorted(range(len(value)), key=lambda g: -value[g])[:int(groups["keep"])]
        allowed = [e for e in allowed if e // size in best]
    return sorted(allowed, key=lambda e: -float(c[e]))[:int(router["top"])]


def route(mlp: dict, w: Dict[str, torch.Tensor], p: str, h: torch.Tensor):
    """(chosen experts [T, top], their weights [T, top])."""
    s = torch.sigmoid(h @ w[p + "router"].t())
    which = torch.tensor([choose(row, w[p + "correction"], mlp["router"]) for row in s])
    chosen = torch.gather(s, 1, which)
    return which, chosen / (chosen.sum(dim=-1, keepdim=True) + 1e-20) * float(mlp["router"]["scale"])


def routed_ff(mlp: dict, w: Dict[str, torch.Tensor], p: str, h: torch.Tensor) -> torch.Tensor:
    which, share = route(mlp, w, p, h)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for s in range(which.shape[1]):
            out[t] += share[t, s] * gated_expert(w, f"{p}e{int(which[t, s])}.", h[t:t + 1])[0]
    if mlp.get("shared"):
        out = out + torch.sigmoid(h @ w[p + "shared.sg"].t()) * gated_expert(w, p + "shared.", h)
    return out


def feed_forward(mlp: dict, w: Dict[str, torch.Tensor], p: str, h: torch.Tensor) -> torch.Tensor:
    return dense_ff(mlp, w, p, h) if mlp["kind"] == "dense" else routed_ff(mlp, w, p, h)


# ---- the model --------------------------------------------------------------------------------------------------------
def layer_forward(config: dict, w: Dict[str, torch.Tensor], i: int, x: torch.Tensor, positions: torch.Tensor, kept: dict) -> torch.Tensor:
    """One layer on the whole sequence.  `kept`: {layer: (keys, values)} of the layers that ran before."""
    layer, eps, p = config["layers"][i], float(config["norm"]["eps"]), f"l{i}."
    source = layer["mixer"].get("kv_from")
    delta, kept[i] = attention(layer["mixer"], w, p + "mix.", centred_norm(x, w[p + "norm1"], eps), positions, eps,
                               None if source is None else kept[int(source)])
    x = x + delta
    if layer.get("mlp"):
        x = x + feed_forward(layer["mlp"], w, p + "mlp.", centred_norm(x, w[p + "norm2"], eps))
    return x


def forward(config: dict, w: Dict[str, torch.Tensor], tokens: Sequence[int], trace: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of every place of one sequence; `trace` receives the residual stream after every layer."""
    positions = torch.arange(len(tokens))
    x = w["embed"][list(tokens)] * float((config.get("embedding") or {}).get("scale", 1.0))
    kept: dict = {}
    for i in range(len(config["layers"])):
        x = layer_forward(config, w, i, x, positions, kept)
        if trace is not None:
            trace.append(x.clone())
    return linear(centred_norm(x, w["final.norm"], float(config["norm"]["eps"])), w["embed"])


def greedy(config: dict, w: Dict[str, torch.Tensor], prompt: Sequence[int], new_tokens: int) -> List[int]:
    tokens = list(prompt)
    for _ in range(new_tokens):
        tokens.append(int(torch.argmax(forward(config, w, tokens)[-1])))
    return tokens[len(prompt):]
