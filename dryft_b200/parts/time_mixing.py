"""Time mixing: a linear recurrence whose projections read mixtures of the token's and the previous token's input.

With ``h_t`` the mixer's input (``h_0`` of a sequence preceded by zeros), ``H`` heads of ``d`` and, for each of the five names
``r k v g w``, a vector ``mu``:

    m_j   = h_t + (h_(t-1) - h_t) * mu_j
    r, k, v = W_r m_r, W_k m_k, W_v m_v          (``H * d`` each) ;   g = W_g m_g
    w     = exp(-exp(W_w2 tanh(W_w1 m_w) + w0))  a decay per head and key channel
    o_t   = (S + diag(u) k_t v_t^T)^T r_t        the bonus ``u`` weighs the current token only
    S    <- diag(w_t) S + k_t v_t^T
    out   = W_o ( o_t / sqrt(mean(o_t^2) + eps) per head  *  norm  *  silu(g) )

The matrix state ``S`` (32-bit) and the previous token's input are per-sequence state of fixed size, zero when a sequence
starts, so a prompt, a piece of one and a single token are the same operation (``csrc/wkv.cu``): a step of many tokens runs its
chunks side by side, a decode step everything behind the products in one launch.  The mixtures are rounded once as the
products' operands; the low-rank map's tanh likewise in a step of many tokens; decays, state, bonus, read-out, norm and gate
are 32-bit in both precisions.  The rank of the low-rank map is the checkpoint's.
``params["names"]`` maps the tensors' roles to their names behind the prefix.
"""

from __future__ import annotations

from typing import Dict, Mapping, Optional

import torch

from ..cache.store import KVNeed, StateNeed
from ..ops import kernels as K
from .base import Runtime, StepContext, TensorInfo, register_mixer
from .linear import linear

_MIX = ("r", "k", "v", "g", "w")
_ROLES = {**{"mu_" + j: "mu." + j for j in _MIX}, "r": "r_proj.weight", "k": "k_proj.weight", "v": "v_proj.weight", "g": "g_proj.weight",
          "w1": "w_down.weight", "w2": "w_up.weight", "w0": "w_up.bias", "u": "bonus", "norm": "norm.weight", "o": "o_proj.weight"}


def _names(params: Mapping, prefix: str) -> Dict[str, str]:
    given = params.get("names") or {}
    return {role: prefix + given.get(role, default) for role, default in _ROLES.items()}


@register_mixer("time_mixing")
class TimeMixing:
    @staticmethod
    def tensors(params: Mapping, prefix: str) -> Dict[str, TensorInfo]:
        w, heads, d = (int(params[k]) for k in ("hidden_size", "num_heads", "dim"))
        nm, hd = _names(params, prefix), heads * d
        rank = int(params.get("rank") or max(8, d // 2))      # random weights only: a checkpoint's tensors carry their own
        t = {nm["mu_" + j]: TensorInfo((w,), "vector", False, 0.5) for j in _MIX}
        t.update({nm[j]: TensorInfo((hd, w), "matrix") for j in "rkvg"})
        t[nm["w1"]], t[nm["w2"]] = TensorInfo((rank, w), "matrix", free=(0,)), TensorInfo((hd, rank), "matrix", free=(1,))
        t[nm["w0"]] = TensorInfo((hd,), "vector", False, -2.0)
        t[nm["u"]] = TensorInfo((heads, d), "vector", False, 0.5)
        t[nm["norm"]] = TensorInfo((hd,), "vector")
        t[nm["o"]] = TensorInfo((w, hd), "matrix")
        return t

    def __init__(self, params: Mapping, prefix: str, weights, rt: Runtime):
        self.rt = rt
        self.hidden, self.heads, self.dim = (int(params[k]) for k in ("hidden_size", "num_heads", "dim"))
        self.eps = float(params["eps"])
        if not 1 <= self.dim <= K.WKV_MAX_DIM:
            raise ValueError(f"time_mixing: heads of 1 to {K.WKV_MAX_DIM} are served, got {self.dim}")
        nm, hd = _names(params, prefix), self.heads * self.dim
        self.hd = hd
        f32 = lambda role: weights.load(nm[role], "vector").to(torch.float32).reshape(-1).contiguous()
        self.mu = torch.stack([f32("mu_" + j) for j in _MIX]).contiguous()             # [5, hidden]
        self.rank = int(weights.shape(nm["w1"])[0])
        # one matrix, the rows of r | k | v | g | w1: a decode step multiplies all five mixtures in one launch
        self.w_in = weights.load_fused([nm["r"], nm["k"], nm["v"], nm["g"], nm["w1"]], [hd, hd, hd, hd, self.rank], self.hidden)
        self.w_rkvg = self.w_in[:4 * hd].view(4, hd, self.hidden)
        self.w_low = self.w_in[4 * hd:]
        self.w_up = weights.load(nm["w2"], "matrix")
        self.w_o = weights.load(nm["o"], "matrix")
        self.w0, self.bonus, self.norm_w = f32("w0"), f32("u"), f32("norm")
        self.chunked_from = int(params.get("chunked_from", 4 * K.WKV_CHUNK_TOKENS))    # steps of fewer tokens walk them in order
        K.wkv_lib()

    def kv_need(self) -> Optional[KVNeed]:
        return None

    def state_need(self):
        return {"s": StateNeed((self.heads, self.dim, self.dim), torch.float32), "last": StateNeed((self.hidden,), self.rt.dtype)}

    def _products(self, m: torch.Tensor, out_dtype) -> torch.Tensor:
        """``[4, n, H * d]``: the four wide products of the first four mixtures."""
        if m.dtype == torch.float32 or self.w_in.dtype != m.dtype:
            return torch.stack([linear(m[j], self.w_rkvg[j], self.rt, out_dtype=out_dtype) for j in range(4)])
        wt = self.w_rkvg.transpose(1, 2)
        return torch.bmm(m[:4], wt) if out_dtype == m.dtype else torch.bmm(m[:4], wt, out_dtype=out_dtype)

    def forward(self, h: torch.Tensor, ctx: StepContext, cache, state, owns_cache: bool = True) -> torch.Tensor:
        n, dev, hd = h.shape[0], h.device, self.hd
        mix = torch.empty((5, n, self.hidden), dtype=h.dtype, device=dev)
        K.wkv_mix(h, state["last"], self.mu, ctx.tok_slot, mix)
        out = torch.empty((n, hd), dtype=h.dtype, device=dev)
        if ctx.decode:
            if (h.dtype == torch.bfloat16 and self.w_in.dtype == h.dtype and K.gemm_decode_groups_supported(n, self.hidden, hd)
                    and K.fused_rows_supported(n, self.hidden, self.rt.small_m_max, 0, normed=True)):
                p = torch.empty((n, self.w_in.shape[0]), dtype=torch.float32, device=dev)
                K.gemm_decode_groups(mix, self.w_in, p, hd)
                r, k, v, g, low = p.split([hd, hd, hd, hd, self.rank], dim=1)
            else:
                r, k, v, g = self._products(mix, torch.float32)
                low = linear(mix[4], self.w_low, self.rt, out_dtype=torch.float32)
            w_up = self.w_up if self.w_up.dtype == h.dtype else self.w_up.to(h.dtype)
            K.wkv_decode(r, k, v, g, low, w_up, self.w0, self.bonus, self.norm_w, self.eps, h, state["last"], ctx.tok_slot, state["s"], out)
        else:
            r, k, v, g = self._products(mix, h.dtype)
            low = linear(mix[4], self.w_low, self.rt, out_dtype=torch.float32)
            t = torch.empty((n, self.rank), dtype=h.dtype, device=dev)
            K.wkv_tanh(low, t)
            z = linear(t, self.w_up, self.rt, out_dtype=torch.float32)
            K.wkv_tokens(r, k, v, g, z, self.w0, self.bonus, self.norm_w, self.eps, h, state["last"], ctx, state["s"], out,
                         chunked=n >= self.chunked_from)
        return linear(out, self.w_o, self.rt)
