"""A gated delta rule: per head a matrix state that decays, is corrected along the current key and read along the current
query.

With ``H`` heads, ``G`` key heads (head ``h`` reads q and k of group ``h // (H / G)``), key size ``d``, value size ``dv`` and
``h`` the mixer's input:

    q, k, v   = W_q h, W_k h (``G x d``), W_v h (``H x dv``), each through a short causal convolution per channel over ``taps``
                tokens (the last column of the stored ``[channels, taps]`` weight multiplies the current token, no bias, zeros
                before a sequence's start) and silu
    q, k      unit vectors per head, ``x / sqrt(sum(x^2) + 1e-6)``; q also times ``d^(-1/2)``
    beta      = sigmoid(W_b h), one per head
    log g     = -exp(A_log_head) softplus(a + dt_bias):  one per head, or (``channel_decay``) one per head and key channel
    S        <- g S ;  u = beta (v - S^T k) ;  S <- S + k u^T ;  o = S^T q          (S: ``d x dv`` per head, 32-bit)
    out       = W_o ( o / sqrt(mean(o^2) + eps) * w * act(z) ), the mean over a head's ``dv`` values, ``w`` shared by the heads

The decay's pre-activation ``a`` and the gate ``z`` are one product of ``h`` each (``a``, ``g``), or (``low_rank``) go through a
low rank, ``W_a2 (W_a1 h)`` and ``W_g2 (W_g1 h)``, whose ranks are the stored tensors' own.  ``gate_act``: ``silu`` or
``sigmoid``.  Everything that reads ``h`` is one product; both second low-rank products are one more (block by block in one
matrix).  The matrix state (kept transposed, ``csrc/delta.cu``) and the convolution's last inputs (a ring of ``taps`` rows) are
per-sequence state of fixed size, so a prompt, a piece of one and a single token are the same operation: a step of many tokens
walks them by fours, a decode step is one launch behind the products.  What follows the products is 32-bit in both precisions.
``params["names"]`` maps the tensors' roles to their names behind the prefix.
"""

from __future__ import annotations

from typing import Dict, Mapping, Optional

import torch

from ..cache.store import KVNeed, StateNeed
from ..ops import kernels as K
from .base import Runtime, StepContext, TensorInfo, register_mixer
from .linear import linear

_ROLES = {"q": "q_proj.weight", "k": "k_proj.weight", "v": "v_proj.weight", "q_conv": "q_conv.weight", "k_conv": "k_conv.weight",
          "v_conv": "v_conv.weight", "b": "b_proj.weight", "a": "a_proj.weight", "a1": "a1_proj.weight", "a2": "a2_proj.weight",
          "g": "g_proj.weight", "g1": "g1_proj.weight", "g2": "g2_proj.weight", "a_log": "A_log", "dt_bias": "dt_bias",
          "norm": "norm.weight", "o": "o_proj.weight"}


def _names(params: Mapping, prefix: str) -> Dict[str, str]:
    given = params.get("names") or {}
    return {role: prefix + given.get(role, default) for role, default in _ROLES.items()}


def _pad(n: int, to: int) -> int:
    return (n + to - 1) // to * to


@register_mixer("gated_delta")
class GatedDelta:
    @staticmethod
    def tensors(params: Mapping, prefix: str) -> Dict[str, TensorInfo]:
        w, heads, kv, d, dv, taps = (int(params[k]) for k in ("hidden_size", "num_heads", "num_kv_heads", "qk_dim", "v_dim", "taps"))
        nm = _names(params, prefix)
        n_dec = heads * d if params.get("channel_decay", False) else heads
        t = {}
        for role, rows in (("q", kv * d), ("k", kv * d), ("v", heads * dv)):
            t[nm[role]] = TensorInfo((rows, w), "matrix")
            t[nm[role + "_conv"]] = TensorInfo((rows, taps), "vector", False, 1.0 / taps)
        t[nm["b"]] = TensorInfo((heads, w), "matrix")
        if params.get("low_rank", False):
            r = int(params.get("rank") or d)       # random weights only: a checkpoint's tensors carry their own ranks
            t[nm["a1"]], t[nm["a2"]] = TensorInfo((r, w), "matrix", free=(0,)), TensorInfo((n_dec, r), "matrix", free=(1,))
            t[nm["g1"]], t[nm["g2"]] = TensorInfo((r, w), "matrix", free=(0,)), TensorInfo((heads * dv, r), "matrix", free=(1,))
        else:
            t[nm["a"]] = TensorInfo((n_dec, w), "matrix")
            t[nm["g"]] = TensorInfo((heads * dv, w), "matrix")
        t[nm["a_log"]] = TensorInfo((heads,), "vector", False, 0.0)
        t[nm["dt_bias"]] = TensorInfo((n_dec,), "vector", False, -2.0)
        t[nm["norm"]] = TensorInfo((dv,), "vector")
        t[nm["o"]] = TensorInfo((w, heads * dv), "matrix")
        return t

    def __init__(self, params: Mapping, prefix: str, weights, rt: Runtime):
        self.rt = rt
        self.hidden, self.heads, self.kv, self.qk_dim, self.v_dim, self.taps = (
            int(params[k]) for k in ("hidden_size", "num_heads", "num_kv_heads", "qk_dim", "v_dim", "taps"))
        self.eps = float(params["eps"])
        self.channel_decay, self.low_rank = bool(params.get("channel_decay", False)), bool(params.get("low_rank", False))
        act = params.get("gate_act", "silu")
        if self.heads % self.kv or not 1 <= self.taps <= K.CONV_MAX_TAPS or not 1 <= self.qk_dim <= K.DELTA_MAX_DIM or act not in ("silu", "sigmoid"):
            raise ValueError(f"gated_delta: {self.heads} heads over {self.kv} key heads of {self.qk_dim} (at most {K.DELTA_MAX_DIM}), "
                             f"{self.taps} taps (at most {K.CONV_MAX_TAPS}), gate {act!r}")
        self.sigmoid_gate = act == "sigmoid"
        nm = _names(params, prefix)
        hd, hv = self.heads * self.qk_dim, self.heads * self.v_dim
        self.n_dec = hd if self.channel_decay else self.heads
        kd = self.kv * self.qk_dim
        self.channels = 2 * kd + hv
        # one product of the mixer's input: q | k | v | (gate | decay) | beta, or q | k | v | beta | low-rank inputs
        roles, rows = ["q", "k", "v"], [kd, kd, hv]
        if not self.low_rank:
            roles += ["g", "a"]
            rows += [hv, self.n_dec]
        roles.append("b")
        rows.append(self.heads)
        at = {r: sum(rows[:i]) for i, r in enumerate(roles)}
        self.b_col, self.g_col, self.a_col = at["b"], at.get("g"), at.get("a")
        w_in = weights.load_fused([nm[r] for r in roles], rows, self.hidden)
        zeros = lambda n, k, like: torch.zeros((n, k), dtype=like.dtype, device=like.device)
        self.low_col = self.low_cols = 0
        self.w_low: Optional[torch.Tensor] = None
        if self.low_rank:
            ra, rg = int(weights.shape(nm["a1"])[0]), int(weights.shape(nm["g1"])[0])
            low = weights.load_fused([nm["a1"], nm["g1"]], [ra, rg], self.hidden)
            a2, g2 = weights.load_fused([nm["a2"]], [self.n_dec], ra), weights.load_fused([nm["g2"]], [hv], rg)
            self.low_col, self.low_cols = _pad(w_in.shape[0], 8), _pad(ra + rg, 16)
            dt = w_in.dtype if w_in.dtype == low.dtype else torch.float32
            w_in = torch.cat([w_in.to(dt), zeros(self.low_col - w_in.shape[0], self.hidden, w_in).to(dt), low.to(dt),
                              zeros(self.low_cols - ra - rg, self.hidden, low).to(dt)])
            dt = a2.dtype if a2.dtype == g2.dtype else torch.float32
            # [a2 | 0 ; 0 | g2]: both second products in one launch
            self.w_low = zeros(self.n_dec + hv, self.low_cols, a2).to(dt)
            self.w_low[:self.n_dec, :ra] = a2
            self.w_low[self.n_dec:, ra:ra + rg] = g2
        pad = (-w_in.shape[0]) % 8
        self.w_in = torch.cat([w_in, zeros(pad, self.hidden, w_in)]).contiguous() if pad else w_in
        self.w_o = weights.load(nm["o"], "matrix")
        f32 = lambda role: weights.load(nm[role], "vector").to(torch.float32).contiguous()
        self.conv_w = torch.cat([f32("q_conv"), f32("k_conv"), f32("v_conv")]).contiguous()
        self.a_log, self.dt_bias, self.norm_w = f32("a_log"), f32("dt_bias"), f32("norm")
        K.delta_lib()

    def kv_need(self) -> Optional[KVNeed]:
        return None

    def state_need(self):
        need = {"s": StateNeed((self.heads, self.v_dim, K.delta_state_rows(self.qk_dim)), torch.float32)}
        if self.taps > 1:
            need["conv"] = StateNeed((self.taps, self.channels), self.rt.dtype)
        return need

    def forward(self, h: torch.Tensor, ctx: StepContext, cache, state, owns_cache: bool = True) -> torch.Tensor:
        n = h.shape[0]
        proj = linear(h, self.w_in, self.rt)
        if self.low_rank:
            low = proj[:, self.low_col:self.low_col + self.low_cols]
            if n <= 64 or h.dtype == torch.float32:
                low = low.contiguous()          # the library's own products read whole rows
            second = linear(low, self.w_low, self.rt)
            dec, gate = second[:, :self.n_dec], second[:, self.n_dec:]
        else:
            dec, gate = proj[:, self.a_col:self.a_col + self.n_dec], proj[:, self.g_col:self.g_col + self.heads * self.v_dim]
        out = torch.empty((n, self.heads * self.v_dim), dtype=h.dtype, device=h.device)
        ring = state.get("conv")
        sizes = (self.heads, self.kv, self.qk_dim, self.v_dim, self.channel_decay)
        if ctx.decode:
            K.delta_decode(proj, 0, self.b_col, dec, gate, self.conv_w, ring, self.a_log, self.dt_bias, self.norm_w, self.eps,
                           self.sigmoid_gate, ctx.tok_slot, ctx.tok_pos, state["s"], out, *sizes)
        else:
            K.delta_tokens(proj, 0, self.b_col, dec, gate, self.conv_w, ring, self.a_log, self.dt_bias, self.norm_w, self.eps,
                           self.sigmoid_gate, ctx, state["s"], out, *sizes)
        return linear(out, self.w_o, self.rt)
