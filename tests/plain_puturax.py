"""A plain, slow evaluation of the Puturax decoder: one function per mechanism, float64 on the CPU, whole sequences at
once, the recurrence token by token, no cache.  It shares no code with ``dryft_b200`` and takes its sizes and constants
from the same ``config.json`` dictionary the library reads; ``weights`` maps tensor names to tensors.

Notation: ``W`` matrices are ``[out, in]`` and applied as ``x @ W.T``; ``L`` is the number of tokens of the sequence;
positions count from 0.

The design in short.  Every sublayer stands between two norms whose stored weights are deviations from one:
``x <- x + norm1b(mixer(norm1(x)))``, then the same for the feed-forward.  Mixers: attention over low-rank latents with a
gate per value; and two mixers side by side, added with fixed factors -- grouped-query attention without rotation (unit
queries, keys and values; queries that grow with the position; squashed scores from which a logarithm of the distance is
taken off; a one in the softmax's denominator; a gate per value) and a linear recurrence with a decay per key channel
whose projections read mixtures of the token's and the previous token's input.  Feed-forwards: an ungated dense one, and
routed experts chosen by groups beside an expert that always runs.
"""

from __future__ import annotations

import math
from typing import Callable, List, Mapping, Optional

import torch

F = torch.float64
_ROUND: Optional[torch.dtype] = None      # set by ``forward(..., rounding=...)``: products read and leave values of this type


def rnd(x: torch.Tensor) -> torch.Tensor:
    return x if _ROUND is None else x.to(_ROUND).to(F)


def mm(h: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """``h @ w.T``; with a rounding type set, of the rounded ``h`` and rounded itself (what a 16-bit product does)."""
    return rnd(rnd(h) @ w.T)


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm1(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return unit_rms(x, eps) * (1.0 + w)


def plain_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return unit_rms(x, eps) * w


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


# ----------------------------------------------------------------------------- rotation
def rotate_half(v: torch.Tensor, pos: torch.Tensor, rot: Optional[Mapping]) -> torch.Tensor:
    """``v [L, ..., n]``: dims ``i`` and ``i + dims/2`` of the first ``rot.dims`` turn by ``pos * base^(-2i/dims)``."""
    if rot is None:
        return v
    dims = int(rot["dims"])
    half = dims // 2
    f = torch.pow(torch.tensor(float(rot["base"]), dtype=F), -2.0 * torch.arange(half, dtype=F) / dims)
    ang = pos.to(F)[:, None] * f[None, :]
    shape = [v.shape[0]] + [1] * (v.dim() - 2) + [half]
    c, s = torch.cos(ang).reshape(shape), torch.sin(ang).reshape(shape)
    a, b = v[..., :half], v[..., half:dims]
    return torch.cat([a * c - b * s, b * c + a * s, v[..., dims:]], dim=-1)


# ----------------------------------------------------------------------------- softmax attention, one head at a time
def weights_of(scores: torch.Tensor, one_in_denominator: bool) -> torch.Tensor:
    """Causal softmax of ``scores [L, L]``; optionally with a one added to the denominator (of the unshifted exponentials)."""
    L = scores.shape[0]
    s = scores.masked_fill(torch.ones(L, L, dtype=torch.bool).triu(1), -math.inf)
    m = s.max(-1, keepdim=True).values
    if one_in_denominator:
        m = torch.clamp(m, min=0.0)
    e = torch.exp(s - m)
    den = e.sum(-1, keepdim=True)
    if one_in_denominator:
        den = den + torch.exp(-m)
    return e / den


def squash(s: torch.Tensor, cap: Optional[float]) -> torch.Tensor:
    return s if cap is None else cap * torch.tanh(s / cap)


def distance_bias(L: int, r1: float, r2: float) -> torch.Tensor:
    """``r1 ln(1 + r2 (i - j))`` for ``j <= i`` (0 elsewhere)."""
    i = torch.arange(L, dtype=F)
    return r1 * torch.log1p(r2 * torch.clamp(i[:, None] - i[None, :], min=0.0))


def temperature(L: int, q_temp: Optional[Mapping]) -> torch.Tensor:
    p = torch.arange(L, dtype=F)
    if q_temp is None:
        return torch.ones(L, dtype=F)
    return 1.0 + float(q_temp["coef"]) * torch.log(torch.floor((p + 1.0) / float(q_temp["every"])) + 1.0)


def biased_attention_mixer(h: torch.Tensor, p: Mapping, w: Mapping[str, torch.Tensor], pre: str, eps: float) -> torch.Tensor:
    L = h.shape[0]
    H, G, d, dv = int(p["heads"]), int(p["kv_heads"]), int(p["dim"]), int(p["vdim"])
    cap = float(p["softcap"]) if p.get("softcap") is not None else None
    q = unit_rms(mm(h, w[pre + "q"]).view(L, H, d), eps) * temperature(L, p.get("q_temp"))[:, None, None]
    k = rnd(unit_rms(mm(h, w[pre + "k"]).view(L, G, d), eps))
    v = rnd(unit_rms(mm(h, w[pre + "v"]).view(L, G, dv), eps))
    gate = torch.sigmoid(mm(h, w[pre + "g"]))
    q = rnd(q)
    out = torch.empty(L, H, dv, dtype=F)
    for hd in range(H):
        g = hd // (H // G)
        s = squash((q[:, hd] @ k[:, g].T) * float(p["scale"]), cap)
        s = s - distance_bias(L, float(w[pre + "r1"][hd]), float(w[pre + "r2"][hd]))
        out[:, hd] = weights_of(s, True) @ v[:, g]
    return mm(out.reshape(L, H * dv) * gate, w[pre + "o"])


# ----------------------------------------------------------------------------- the recurrence
def previous(h: torch.Tensor) -> torch.Tensor:
    """Row t holds the input of token t - 1; zeros for the first."""
    return torch.cat([torch.zeros_like(h[:1]), h[:-1]], dim=0)


def decayed_outer_products(r, k, v, w, u) -> torch.Tensor:
    """One head: ``r, k, w [L, d]``, ``v [L, dv]``, ``u [d]``: the read-out sees the past's state plus the current token's outer
    product weighted by ``u``; then the state decays per key channel and takes the outer product in."""
    L, d = r.shape
    S = torch.zeros(d, v.shape[1], dtype=F)
    o = torch.empty(L, v.shape[1], dtype=F)
    for t in range(L):
        kv = k[t][:, None] * v[t][None, :]
        o[t] = (S + u[:, None] * kv).T @ r[t]
        S = w[t][:, None] * S + kv
    return o


def time_mixing_mixer(h: torch.Tensor, p: Mapping, w: Mapping[str, torch.Tensor], pre: str, eps: float) -> torch.Tensor:
    L = h.shape[0]
    H, d = int(p["heads"]), int(p["dim"])
    hr = rnd(h)
    hp = previous(hr)
    mixed = {n: hr + (hp - hr) * w[pre + "mu." + n] for n in "rkvgw"}
    r, k, v = (mm(mixed[n], w[pre + n]).view(L, H, d) for n in "rkv")
    gate = silu(mm(mixed["g"], w[pre + "g"]))
    z = rnd(torch.tanh(rnd(mixed["w"]) @ w[pre + "w1"].T)) @ w[pre + "w2"].T + w[pre + "w0"]
    decay = torch.exp(-torch.exp(z)).view(L, H, d)
    o = torch.stack([unit_rms(decayed_outer_products(r[:, i], k[:, i], v[:, i], decay[:, i], w[pre + "u"][i]), eps) for i in range(H)], 1)
    return mm(o.reshape(L, H * d) * w[pre + "norm"] * gate, w[pre + "o"])


def side_by_side_mixer(h, p, w, pre, eps):
    left = biased_attention_mixer(h, p["left"], w, pre + "left.", eps)
    right = time_mixing_mixer(h, p["right"], w, pre + "right.", eps)
    return float(p.get("left_scale", 1.0)) * left + float(p.get("right_scale", 1.0)) * right


# ----------------------------------------------------------------------------- mixer: attention over latents
def latent_attention_mixer(h: torch.Tensor, p: Mapping, w: Mapping[str, torch.Tensor], pre: str, eps: float) -> torch.Tensor:
    L = h.shape[0]
    H, d, r, dv, kr = int(p["heads"]), int(p["dim"]), int(p["rot_dim"]), int(p["vdim"]), int(p["kv_rank"])
    pos = torch.arange(L)
    rot = p.get("rot") if r else None
    cq = rnd(plain_norm(mm(h, w[pre + "dq"]), w[pre + "dq.norm"], eps))
    q = mm(cq, w[pre + "uq"]).view(L, H, d + r)
    down = mm(h, w[pre + "dkv"])
    c = rnd(plain_norm(down[:, :kr], w[pre + "dkv.norm"], eps))
    k_rot = rnd(rotate_half(down[:, kr:kr + r], pos, rot))                 # one rotated key part for all heads
    k_plain = mm(c, w[pre + "uk"]).view(L, H, d)
    v = mm(c, w[pre + "uv"]).view(L, H, dv)
    q_rot = rotate_half(q[:, :, d:], pos, rot)
    gate = torch.sigmoid(mm(h, w[pre + "g"]))
    out = torch.empty(L, H, dv, dtype=F)
    for hd in range(H):
        s = (q[:, hd, :d] @ k_plain[:, hd].T + q_rot[:, hd] @ k_rot.T) * float(p["scale"])
        out[:, hd] = rnd(weights_of(s, False)) @ v[:, hd]
    return mm(out.reshape(L, H * dv) * gate, w[pre + "o"])


# ----------------------------------------------------------------------------- feed-forwards
def dense_ffn(h: torch.Tensor, w: Mapping[str, torch.Tensor], pre: str) -> torch.Tensor:
    return mm(torch.clamp(mm(h, w[pre + "up"]), min=0.0) ** 2, w[pre + "down"])


def router_choice(h: torch.Tensor, router: Mapping, w: Mapping[str, torch.Tensor], pre: str):
    """Chosen experts ``[L, top]`` and their weights.  Choices rank ``sigmoid(z) + correction``; a group of neighbours counts the
    sum of its two largest; experts outside the best groups are out of the question, however low the rest."""
    s = torch.sigmoid(rnd(h) @ w[pre + "router"].T)
    choice = s + w[pre + "correction"]
    L, E = s.shape
    groups = router.get("groups") or {"count": 1, "keep": 1}
    n, keep, top = int(groups["count"]), int(groups["keep"]), int(router["top"])
    by_group = choice.view(L, n, E // n)
    rank = torch.sort(by_group, dim=-1, descending=True).values[..., :2].sum(-1)
    best = torch.sort(rank, dim=-1, descending=True, stable=True).indices[:, :keep]
    allowed = torch.zeros(L, n, dtype=torch.bool).scatter_(1, best, True).repeat_interleave(E // n, dim=1)
    idx = torch.sort(choice.masked_fill(~allowed, -math.inf), dim=-1, descending=True, stable=True).indices[:, :top]
    wts = torch.gather(s, 1, idx)
    return idx, wts / (wts.sum(-1, keepdim=True) + 1e-20)


def expert(h: torch.Tensor, w: Mapping[str, torch.Tensor], pre: str) -> torch.Tensor:
    return mm(silu(mm(h, w[pre + "gate"])) * mm(h, w[pre + "up"]), w[pre + "down"])


def moe_ffn(h: torch.Tensor, mlp: Mapping, w: Mapping[str, torch.Tensor], pre: str) -> torch.Tensor:
    idx, wts = router_choice(h, mlp["router"], w, pre)
    out = torch.zeros(h.shape[0], h.shape[1], dtype=F)
    for e in range(int(mlp["router"]["experts"])):
        rows, places = torch.nonzero(idx == e, as_tuple=True)
        if rows.numel():
            out.index_add_(0, rows, wts[rows, places][:, None] * expert(h[rows], w, f"{pre}e{e}."))
    if mlp.get("shared") is not None:
        out = out + expert(h, w, pre + "shared.")
    return out


# ----------------------------------------------------------------------------- the model
def forward(config: Mapping, weights: Mapping[str, torch.Tensor], tokens: List[int],
            tap: Optional[Callable[[int, torch.Tensor], None]] = None, rounding: Optional[torch.dtype] = None,
            number: torch.dtype = torch.float64) -> torch.Tensor:
    """Logits ``[L, vocab]`` of one sequence.  ``tap(layer, x)`` sees the stream after every layer.  ``number``: the type everything is
    evaluated in (float32 shows which rows of a model are ill-conditioned in 32-bit whoever evaluates them)."""
    global _ROUND, F
    _ROUND, F = rounding, number
    try:
        return _forward(config, weights, tokens, tap)
    finally:
        _ROUND, F = None, torch.float64


def _forward(config, weights, tokens, tap):
    w = {k: v.to(F) for k, v in weights.items() if v.is_floating_point()}
    eps = float(config["norm"]["eps"])
    x = w["embed"][torch.tensor(tokens, dtype=torch.long)] * float((config.get("embedding") or {}).get("scale", 1.0))
    for i, layer in enumerate(config["layers"]):
        pre = f"l{i}."
        n = layer_norm1(x, w[pre + "norm1"], eps)
        if layer["type"] == "latent_attention":
            y = latent_attention_mixer(n, layer["mixer"], w, pre + "mix.", eps)
        elif layer["type"] == "parallel":
            y = side_by_side_mixer(n, layer["mixer"], w, pre + "mix.", eps)
        else:
            raise ValueError(layer["type"])
        x = x + layer_norm1(y, w[pre + "norm1b"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            n = layer_norm1(x, w[pre + "norm2"], eps)
            if mlp["kind"] == "dense":
                y = dense_ffn(n, w, pre + "mlp.")
            elif mlp["kind"] == "moe":
                y = moe_ffn(n, mlp, w, pre + "mlp.")
            else:
                raise ValueError(mlp["kind"])
            x = x + layer_norm1(y, w[pre + "norm2b"], eps)
        if tap is not None:
            tap(i, x)
    return rnd(layer_norm1(x, w["final.norm"], eps)) @ w["embed"].T


def greedy(config: Mapping, weights: Mapping[str, torch.Tensor], prompt: List[int], n_new: int) -> List[int]:
    """The best next token, ``n_new`` times, each from a whole evaluation of all tokens so far."""
    ids, out = list(prompt), []
    for _ in range(n_new):
        t = int(torch.argmax(forward(config, weights, ids)[-1]))
        out.append(t)
        ids.append(t)
    return out
