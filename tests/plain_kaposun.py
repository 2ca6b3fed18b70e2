"""Plain, slow implementation of the Kaposun decoder: whole sequences, no cache, one function for each mechanism, float64 by
default.  It shares no code with `kvcache_b200` (it reads the model folder with the `safetensors` package and `json`) and
states every formula directly.

The design, in this file's notation.  W = width, residual stream x[T, W], N(x; w) = x / sqrt(mean(x^2) + eps) * w.

* embedding: x_t = embed[tok_t]; logits = embed N(x; final.norm).
* layer: h = N(x; norm1); x += m (mixer(h) + ff(h)), m = residual_mult; a layer may have no ff.
* loop: layers start .. stop - 1 run `times` times before the rest (the same weights; every pass starts its states empty).
* ff(h) = Wdown g(Wup h), g(z) = z Phi(z) with the normal distribution function Phi.
* attention: q, k, v = Wq h, Wk h, Wv h; all of a token's q numbers together are divided by sqrt(mean(q^2) + eps) and
  multiplied by a weight of that size, k likewise; then the pairs (i, i + dims / 2) of the first rot.dims numbers of a head are
  turned by p base^(-2 i / dims) / factor.  s_ij = scale q_i . k_j, j <= i, softmax, Wo.
* parallel: left_scale left(h) + right_scale right(h).
  left: attention without rotation over the keys with i - j < size or j < keep_first; its heads times sigmoid(Wg h), then Wo.
  right: the gated delta rule.  q, k (kv_heads x dim) and v (heads x vdim) pass a causal convolution per channel and silu;
  q and k become unit vectors per head, q also times dim^(-1/2); b = sigmoid(Wb h) per head;
  a = exp(-exp(A_log_h) softplus(Wa2 Wa1 h + dt_bias)) per head and key channel.  S~ = diag(a) S; S = S~ + k (b (v - S~^T k))^T;
  o = S^T q; each head's o over its root mean square, times norm, times sigmoid(Wg2 Wg1 h), then Wo.
* mamba2: Win h = [z | x | B | C | dt]; x, B, C pass a causal convolution with bias and silu; d = softplus(dt + dt_bias);
  S = exp(-exp(A_log_h) d) S + d B x^T, y = S^T C + D_h x; y silu(z) in norm_groups equal parts, each over its root mean
  square, times norm, then Wo.
"""
from __future__ import annotations

import contextlib
import json
import math
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


def linear(x: torch.Tensor, weight: torch.Tensor) -> torch.Tensor:
    if _ROUND_TO is None:
        return x @ weight.t()
    return (x.to(_ROUND_TO).to(weight.dtype) @ weight.t()).to(_ROUND_TO).to(weight.dtype)


# ---- norms and pointwise functions --------------------------------------------------------------------------------------
def rms_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * weight


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def exact_gelu(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


# ---- attention ----------------------------------------------------------------------------------------------------------
def rotate_halves(x: torch.Tensor, positions: torch.Tensor, rot: Optional[dict]) -> torch.Tensor:
    """x [T, heads, D]: numbers i and i + dims / 2 of each head are turned by p f_i, f_i = base^(-2 i / dims) / factor."""
    if not rot:
        return x
    dims, base = int(rot["dims"]), float(rot["base"])
    factor = float(rot["scaling"]["factor"]) if rot.get("scaling") else 1.0
    out = x.clone()
    for i in range(dims // 2):
        angle = positions.to(torch.float64) * (base ** (-2.0 * i / dims) / factor)
        c, s = torch.cos(angle)[:, None].to(x.dtype), torch.sin(angle)[:, None].to(x.dtype)
        u, v = x[..., i], x[..., i + dims // 2]
        out[..., i], out[..., i + dims // 2] = u * c - v * s, v * c + u * s
    return out


def sees(i: int, j: int, mask: Optional[dict]) -> bool:
    if j > i:
        return False
    return not mask or i - j < int(mask["size"]) or j < int(mask.get("keep_first", 0))


def attention_heads(m: dict, w: Dict[str, torch.Tensor], p: str, h: torch.Tensor, positions: torch.Tensor, eps: float) -> torch.Tensor:
    """The concatenated heads [T, heads * vdim], before gate and output matrix."""
    T = h.shape[0]
    H, G, dim, vdim = (int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
    q = rms_norm(linear(h, w[p + "q"]), w[p + "q.norm"], eps).view(T, H, dim)
    k = rms_norm(linear(h, w[p + "k"]), w[p + "k.norm"], eps).view(T, G, dim)
    v = linear(h, w[p + "v"]).view(T, G, vdim)
    q, k = rotate_halves(q, positions, m.get("rot")), rotate_halves(k, positions, m.get("rot"))
    out = torch.zeros(T, H, vdim, dtype=h.dtype)
    for i in range(T):
        js = [j for j in range(i + 1) if sees(i, j, m.get("mask"))]
        for head in range(H):
            g = head // (H // G)
            out[i, head] = torch.softmax((k[js, g] @ q[i, head]) * float(m["scale"]), dim=0) @ v[js, g]
    return out.reshape(T, H * vdim)


def attention(m, w, p, h, positions, eps):
    return linear(attention_heads(m, w, p, h, positions, eps), w[p + "o"])


def gated_attention(m, w, p, h, positions, eps):
    heads = attention_heads(m, w, p, h, positions, eps) * torch.sigmoid(linear(h, w[p + "g"]))
    return linear(heads, w[p + "o"])


# ---- recurrent mixers ---------------------------------------------------------------------------------------------------
def short_convolution(x: torch.Tensor, weight: torch.Tensor, bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    """silu(bias + sum_n weight[:, n] x_{t - (taps - 1) + n}), x zero before the start; x [T, channels], weight [channels, taps]."""
    T, taps = x.shape[0], weight.shape[1]
    y = torch.zeros_like(x) if bias is None else bias.expand_as(x).clone()
    for t in range(T):
        for n in range(taps):
            at = t - (taps - 1) + n
            if at >= 0:
                y[t] = y[t] + weight[:, n] * x[at]
    return silu(y)


def delta_decays(m: dict, w: Dict[str, torch.Tensor], p: str, h: torch.Tensor) -> torch.Tensor:
    T, H, dim = h.shape[0], int(m["heads"]), int(m["dim"])
    z = (linear(linear(h, w[p + "a1"]), w[p + "a2"]) + w[p + "dt_bias"]).view(T, H, dim)
    return torch.exp(-torch.exp(w[p + "A_log"])[None, :, None] * softplus(z))


def gated_delta(m: dict, w: Dict[str, torch.Tensor], p: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, dim, vdim = (int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
    q = unit(short_convolution(linear(h, w[p + "q"]), w[p + "q.conv"]).view(T, G, dim)) * dim ** -0.5
    k = unit(short_convolution(linear(h, w[p + "k"]), w[p + "k.conv"]).view(T, G, dim))
    v = short_convolution(linear(h, w[p + "v"]), w[p + "v.conv"]).view(T, H, vdim)
    beta = torch.sigmoid(linear(h, w[p + "b"]))
    decay = delta_decays(m, w, p, h)
    gate = torch.sigmoid(linear(linear(h, w[p + "g1"]), w[p + "g2"])).view(T, H, vdim)
    out = torch.zeros(T, H, vdim, dtype=h.dtype)
    for head in range(H):
        g = head // (H // G)
        S = torch.zeros(dim, vdim, dtype=h.dtype)
        for t in range(T):
            S = decay[t, head][:, None] * S
            u = beta[t, head] * (v[t, head] - S.t() @ k[t, g])
            S = S + torch.outer(k[t, g], u)
            out[t, head] = S.t() @ q[t, g]
    out = rms_norm(out, w[p + "norm"], eps) * gate
    return linear(out.reshape(T, H * vdim), w[p + "o"])


def grouped_norm(y: torch.Tensor, weight: torch.Tensor, groups: int, eps: float) -> torch.Tensor:
    """Each of `groups` equal parts of a row over its own root mean square, then the weight."""
    parts = y.view(y.shape[0], groups, -1)
    return (parts / torch.sqrt((parts * parts).mean(dim=-1, keepdim=True) + eps)).reshape(y.shape) * weight


def mamba2(m: dict, w: Dict[str, torch.Tensor], p: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, V, N, G = (int(m[k]) for k in ("heads", "vdim", "state", "groups"))
    inner = H * V
    z, xbc, dt = torch.split(linear(h, w[p + "in"]), [inner, inner + 2 * G * N, H], dim=1)
    xbc = short_convolution(xbc, w[p + "conv"], w[p + "conv.b"])
    x, B, C = xbc[:, :inner].reshape(T, H, V), xbc[:, inner:inner + G * N].reshape(T, G, N), xbc[:, inner + G * N:].reshape(T, G, N)
    dt = softplus(dt + w[p + "dt_bias"])
    y = torch.zeros(T, H, V, dtype=h.dtype)
    for head in range(H):
        g = head // (H // G)
        S = torch.zeros(N, V, dtype=h.dtype)
        for t in range(T):
            S = torch.exp(-torch.exp(w[p + "A_log"][head]) * dt[t, head]) * S + dt[t, head] * torch.outer(B[t, g], x[t, head])
            y[t, head] = S.t() @ C[t, g] + w[p + "D"][head] * x[t, head]
    y = grouped_norm(y.reshape(T, inner) * silu(z), w[p + "norm"], int(m["norm_groups"]), eps)
    return linear(y, w[p + "o"])


def mixer_forward(kind: str, m: dict, w: Dict[str, torch.Tensor], p: str, h: torch.Tensor, positions: torch.Tensor, eps: float) -> torch.Tensor:
    if kind == "attention":
        return attention(m, w, p, h, positions, eps)
    if kind == "mamba2":
        return mamba2(m, w, p, h, eps)
    assert kind == "parallel", kind
    return (float(m["left_scale"]) * gated_attention(m["left"], w, p + "left.", h, positions, eps)
            + float(m["right_scale"]) * gated_delta(m["right"], w, p + "right.", h, eps))


# ---- the model ----------------------------------------------------------------------------------------------------------
def feed_forward(w: Dict[str, torch.Tensor], p: str, h: torch.Tensor) -> torch.Tensor:
    return linear(exact_gelu(linear(h, w[p + "up"])), w[p + "down"])


def layer_forward(config: dict, w: Dict[str, torch.Tensor], i: int, x: torch.Tensor, positions: torch.Tensor) -> torch.Tensor:
    layer, eps, p = config["layers"][i], float(config["norm"]["eps"]), f"l{i}."
    h = rms_norm(x, w[p + "norm1"], eps)
    delta = mixer_forward(layer["type"], layer["mixer"], w, p + "mix.", h, positions, eps)
    if layer.get("mlp"):
        delta = delta + feed_forward(w, p + "mlp.", h)
    return x + float(config["residual_mult"]) * delta


def layer_order(config: dict) -> List[int]:
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return list(range(n))
    start, stop = int(loop["start"]), int(loop["stop"])
    return list(range(start)) + list(range(start, stop)) * int(loop["times"]) + list(range(stop, n))


def forward(config: dict, w: Dict[str, torch.Tensor], tokens: Sequence[int], trace: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of every place of one sequence; `trace` receives the residual stream after every layer run."""
    positions = torch.arange(len(tokens))
    x = w["embed"][list(tokens)]
    for i in layer_order(config):
        x = layer_forward(config, w, i, x, positions)
        if trace is not None:
            trace.append(x.clone())
    return linear(rms_norm(x, w["final.norm"], float(config["norm"]["eps"])), w["embed"])


def greedy(config: dict, w: Dict[str, torch.Tensor], prompt: Sequence[int], new_tokens: int) -> List[int]:
    tokens = list(prompt)
    for _ in range(new_tokens):
        tokens.append(int(torch.argmax(forward(config, w, tokens)[-1])))
    return tokens[len(prompt):]
