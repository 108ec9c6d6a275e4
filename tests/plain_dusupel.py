"""A plain, slow evaluation of the Dusupel decoder: one function per mechanism, float64 on the CPU, whole sequences at
once, the recurrences token by token, no cache.  It shares no code with ``dryft_b200`` and takes its sizes and constants
from the same ``config.json`` dictionary the library reads (the ranks of the low-rank maps from the tensors' shapes);
``weights`` maps tensor names to tensors.

Notation: ``W`` matrices are ``[out, in]`` and applied as ``x @ W.T``; ``L`` is the number of tokens of the sequence;
positions count from 0.

The design in short.  Two layer norms (with bias) of the same stream, one for the mixer and one for the feed-forward, whose
results join the stream together times a constant: ``x <- x + m (mixer(norm1(x)) + ff(norm2(x)))``.  A stretch of layers runs
several times in a row with the same weights.  Mixers: a gated delta rule with one decay per head and key channel
(``channel_delta``, ``channel_delta_2``), and two mixers side by side -- windowed attention that also keeps the first tokens,
behind short convolutions, with a gate per value -- and a gated delta rule with one decay per head.
"""

from __future__ import annotations

import math
from typing import Callable, Dict, List, Mapping, Optional

import torch

F = torch.float64
_ROUND: Optional[torch.dtype] = None      # set by ``forward(..., rounding=...)``: products read and leave values of this type


def rnd(x: torch.Tensor) -> torch.Tensor:
    return x if _ROUND is None else x.to(_ROUND).to(F)


def mm(h: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """``h @ w.T``; with a rounding type set, of the rounded ``h`` and rounded itself (what a 16-bit product does)."""
    return rnd(rnd(h) @ w.T)


def layer_norm(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor, eps: float) -> torch.Tensor:
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.where(z > 30.0, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


# ----------------------------------------------------------------------------- short convolution
def short_conv(u: torch.Tensor, weight: torch.Tensor) -> torch.Tensor:
    """``u [L, C]``, ``weight [C, taps]``: the last column multiplies the current token, zeros before the start, no bias."""
    L, taps = u.shape[0], weight.shape[1]
    out = torch.zeros_like(u)
    for j in range(taps):
        back = taps - 1 - j
        if back < L:
            out[back:] += u[:L - back] * weight[:, j]
    return out


# ----------------------------------------------------------------------------- rotation
def rotate_halves(v: torch.Tensor, pos: torch.Tensor, rot: Optional[Mapping]) -> torch.Tensor:
    """``v [L, heads, n]``: dims ``i`` and ``i + dims/2`` of the first ``rot.dims`` turn by ``pos * base^(-2i/dims)``."""
    if rot is None:
        return v
    dims = int(rot["dims"])
    half = dims // 2
    f = torch.pow(torch.tensor(float(rot["base"]), dtype=F), -2.0 * torch.arange(half, dtype=F) / dims)
    ang = pos.to(F)[:, None, None] * f
    c, s = torch.cos(ang), torch.sin(ang)
    a, b = v[..., :half], v[..., half:dims]
    return torch.cat([a * c - b * s, b * c + a * s, v[..., dims:]], dim=-1)


# ----------------------------------------------------------------------------- windowed attention that keeps the first tokens
def sees(i: int, j: int, mask: Optional[Mapping]) -> bool:
    if j > i:
        return False
    return mask is None or i - j < int(mask["size"]) or j < int(mask.get("keep_first", 0))


def visible(L: int, mask: Optional[Mapping]) -> torch.Tensor:
    i, j = torch.arange(L)[:, None], torch.arange(L)[None, :]
    near = torch.ones(L, L, dtype=torch.bool) if mask is None else (i - j < int(mask["size"])) | (j < int(mask.get("keep_first", 0)))
    return (j <= i) & near


def masked_softmax_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, seen: torch.Tensor) -> torch.Tensor:
    """``q [L, d]``, ``k [L, d]``, ``v [L, dv]`` of one head."""
    s = ((q @ k.T) * scale).masked_fill(~seen, -math.inf)
    return rnd(torch.softmax(s, dim=-1)) @ v


def gated_window_attention(h: torch.Tensor, p: Mapping, w: Mapping[str, torch.Tensor], pre: str) -> torch.Tensor:
    L = h.shape[0]
    H, G, d, dv = int(p["heads"]), int(p["kv_heads"]), int(p["dim"]), int(p["vdim"])
    pos = torch.arange(L)
    q, k, v = (short_conv(mm(h, w[pre + n]), w[pre + n + ".conv"]) for n in ("q", "k", "v"))
    q = rnd(rotate_halves(q.view(L, H, d), pos, p.get("rot")))
    k = rnd(rotate_halves(k.view(L, G, d), pos, p.get("rot")))
    v = rnd(v.view(L, G, dv))
    seen = visible(L, p.get("mask"))
    out = torch.empty(L, H, dv, dtype=F)
    for hd in range(H):
        g = hd // (H // G)
        out[:, hd] = masked_softmax_attention(q[:, hd], k[:, g], v[:, g], float(p["scale"]), seen)
    return mm(rnd(out.reshape(L, H * dv)) * torch.sigmoid(mm(h, w[pre + "g"])), w[pre + "o"])


# ----------------------------------------------------------------------------- gated delta rule
def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_operands(h: torch.Tensor, p: Mapping, w: Mapping[str, torch.Tensor], pre: str, per_channel: bool):
    """``q, k [L, H, d]`` (unit vectors, q times d^-1/2, each head its own copy), ``v [L, H, dv]``, ``log g [L, H, d or 1]``,
    ``beta [L, H]``."""
    L = h.shape[0]
    H, G, d, dv = int(p["heads"]), int(p["kv_heads"]), int(p["dim"]), int(p["vdim"])
    q, k, v = (silu(short_conv(mm(h, w[pre + n]), w[pre + n + ".conv"])) for n in ("q", "k", "v"))
    q, k = unit(q.view(L, G, d)) * d ** -0.5, unit(k.view(L, G, d))
    q, k = (x.repeat_interleave(H // G, dim=1) for x in (q, k))
    beta = torch.sigmoid(mm(h, w[pre + "b"]))
    if per_channel:
        z = mm(mm(h, w[pre + "a1"]), w[pre + "a2"]) + w[pre + "dt_bias"]
        lg = -torch.exp(w[pre + "A_log"])[:, None] * softplus(z).view(L, H, d)
    else:
        z = mm(h, w[pre + "a"]) + w[pre + "dt_bias"]
        lg = (-torch.exp(w[pre + "A_log"]) * softplus(z))[..., None]
    return q, k, v.view(L, H, dv), lg, beta


def delta_rule(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, lg: torch.Tensor, beta: torch.Tensor,
               S: Optional[torch.Tensor] = None):
    """Token by token: the state decays, ``u = beta (v - S^T k)`` is written along ``k``, and ``S^T q`` is read after the write.
    Returns ``(o [L, H, dv], S [H, d, dv])``."""
    L, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=F) if S is None else S.clone()
    o = torch.empty_like(v)
    for t in range(L):
        S = torch.exp(lg[t])[:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return o, S


def gated_head_norm(o: torch.Tensor, weight: torch.Tensor, gate: torch.Tensor, eps: float) -> torch.Tensor:
    """``o [L, H, dv]`` over each head's root mean square, times a weight shared by the heads, times the gate ``[L, H * dv]``."""
    L, H, dv = o.shape
    n = o / torch.sqrt((o * o).mean(-1, keepdim=True) + eps) * weight
    return n.reshape(L, H * dv) * gate


def delta_mixer(h: torch.Tensor, p: Mapping, w: Mapping[str, torch.Tensor], pre: str, eps: float, per_channel: bool) -> torch.Tensor:
    q, k, v, lg, beta = delta_operands(h, p, w, pre, per_channel)
    o, _ = delta_rule(q, k, v, lg, beta)
    if per_channel:
        gate = torch.sigmoid(mm(mm(h, w[pre + "g1"]), w[pre + "g2"]))
    else:
        gate = silu(mm(h, w[pre + "g"]))
    return mm(gated_head_norm(o, w[pre + "norm"], gate, eps), w[pre + "o"])


def side_by_side_mixer(h, p, w, pre, eps):
    left = gated_window_attention(h, p["left"], w, pre + "left.")
    right = delta_mixer(h, p["right"], w, pre + "right.", eps, per_channel=False)
    return float(p.get("left_scale", 1.0)) * left + float(p.get("right_scale", 1.0)) * right


# ----------------------------------------------------------------------------- feed-forward
def dense_ffn(h: torch.Tensor, w: Mapping[str, torch.Tensor], pre: str) -> torch.Tensor:
    return mm(silu(mm(h, w[pre + "gate"])) * mm(h, w[pre + "up"]), w[pre + "down"])


# ----------------------------------------------------------------------------- the model
def run_order(config: Mapping) -> List[int]:
    n = len(config["layers"])
    loop = config.get("loop")
    if loop is None:
        return list(range(n))
    a, b = int(loop["start"]), int(loop["stop"])
    return list(range(a)) + list(range(a, b)) * int(loop["times"]) + list(range(b, n))


def forward(config: Mapping, weights: Mapping[str, torch.Tensor], tokens: List[int],
            tap: Optional[Callable[[int, torch.Tensor], None]] = None, rounding: Optional[torch.dtype] = None) -> torch.Tensor:
    """Logits ``[L, vocab]`` of one sequence.  ``tap(run, x)`` sees the stream after every layer run."""
    global _ROUND
    _ROUND = rounding
    try:
        return _forward(config, weights, tokens, tap)
    finally:
        _ROUND = None


def _forward(config, weights, tokens, tap):
    w = {k: v.to(F) for k, v in weights.items() if v.is_floating_point()}
    eps, m = float(config["norm"]["eps"]), float(config.get("residual_mult", 1.0))
    x = w["embed"][torch.tensor(tokens, dtype=torch.long)]
    for run, i in enumerate(run_order(config)):
        layer, pre = config["layers"][i], f"l{i}."
        n1 = layer_norm(x, w[pre + "norm1"], w[pre + "norm1.b"], eps)
        if layer["type"] in ("channel_delta", "channel_delta_2"):
            y = delta_mixer(n1, layer["mixer"], w, pre + "mix.", eps, per_channel=True)
        elif layer["type"] == "parallel":
            y = side_by_side_mixer(n1, layer["mixer"], w, pre + "mix.", eps)
        else:
            raise ValueError(layer["type"])
        if layer.get("mlp") is not None:
            if layer["mlp"]["kind"] != "dense":
                raise ValueError(layer["mlp"]["kind"])
            y = y + dense_ffn(layer_norm(x, w[pre + "norm2"], w[pre + "norm2.b"], eps), w, pre + "mlp.")
        x = x + m * y
        if tap is not None:
            tap(run, x)
    return rnd(layer_norm(x, w["final.norm"], w["final.norm.b"], eps)) @ w["head"].T


def greedy(config: Mapping, weights: Mapping[str, torch.Tensor], prompt: List[int], n_new: int) -> List[int]:
    """The best next token, ``n_new`` times, each from a whole evaluation of all tokens so far."""
    ids, out = list(prompt), []
    for _ in range(n_new):
        t = int(torch.argmax(forward(config, weights, ids)[-1]))
        out.append(t)
        ids.append(t)
    return out
