"""Grouped-query attention over a sliding window plus one pooled key and value per block of positions that has left
the window, with a sink in the softmax's denominator.

Per step, with ``h`` the mixer's input:

    q = W_q h (+ b_q), k = W_k h (+ b_k), v = W_v h (+ b_v)           one product (queries only for a run step that reads
                                                                      another step's keys and values)
    q, k: the first ``rotary_dim`` dims of each head rotated by the token's position (position part ``rope``), THEN
          (``unit_norm``) each head divided by its root mean square over ``qk_dim`` (no weight, ``eps`` inside the root)
    k, v -> the cache at the token's position; every token that completes a block of ``pool`` positions leaves the mean
          of the block's cached keys and the mean of its cached values in pooled rows (one row per block)
    the query at position i sees the tokens j with 0 <= i - j < window and the pooled rows of the blocks b with
          b * pool + pool - 1 <= i - window; scores ``(q . k) * scale``; tokens and blocks share one softmax whose
          denominator also holds ``exp(sink_head)`` (``sink``: a number per head without key or value)
    (``head_gate``: head ``h``'s output is multiplied by ``sigmoid(W_g h)_h``, one number per head, ``W_g [heads, hidden]``
          riding in the input product)
    out = W_o (heads concatenated)

``keep_first``: with a ``window``, the sequence's first ``keep_first`` tokens stay visible to every later query (each once, with
their true positions).  ``conv_taps``: q, k and v pass a short causal convolution per channel right behind the projection
(weights ``q_conv`` .. ``[channels, taps]``, no bias, zeros before the sequence's start); its last ``taps - 1`` inputs are
per-sequence state.  ``value_gate``: the concatenated heads are multiplied element by element by ``sigmoid(W_g h)``, ``W_g
[heads * v_dim, hidden]`` riding in the input product.

``proj_norm``: q and k pass an RMS norm over the WHOLE projection (all heads' rows at once, weights ``q_norm [heads * qk_dim]``
and ``k_norm [kv_heads * qk_dim]``, ``eps`` inside the root) before the rotation.  The rotation's layout is the position
part's (``half``: dims ``i`` and ``i + R/2``; ``interleaved``: dims ``2i`` and ``2i + 1``).

``value_norm``: each head's value is divided by its root mean square over ``v_dim`` and cached so.  ``q_temp`` (``coef``, ``every``): the
query of position p is multiplied by ``1 + coef * ln(floor((p + 1) / every) + 1)``.  ``softcap``: a scaled score becomes ``cap *
tanh(score / cap)``.  ``distance_bias``: then ``r1_h * ln(1 + r2_h * (i - j))`` is taken off, two numbers per head (roles ``r1``,
``r2``).  ``unit_sink``: the denominator holds one more exponential of score 0, without key, value or tensor.

Without a ``window`` every earlier token is seen and there are no pooled rows.  A run step that borrows another's cache uses
its own queries, window, pool, scale and sink over the owner's rows; when it summarises the same blocks as the owner it
reads the owner's pooled rows, else it keeps pooled rows of its own (``CacheEntry.fills_pooled``).
Scores, softmax, sums, angles and the unit norm are 32-bit in both precisions (``csrc/pool_attn.cu``).
``params["names"]`` maps the tensors' roles to their names behind the prefix.
"""

from __future__ import annotations

import math
from typing import Dict, Mapping, Optional

import torch

from ..cache.store import CacheEntry, KVNeed, StateNeed
from ..config.spec import PartSpec
from ..ops import kernels as K
from .base import POSITIONS, Runtime, StepContext, TensorInfo, register_mixer
from .linear import linear

_ROLES = {"q": "q_proj.weight", "k": "k_proj.weight", "v": "v_proj.weight", "o": "o_proj.weight", "q_bias": "q_proj.bias",
          "k_bias": "k_proj.bias", "v_bias": "v_proj.bias", "sink": "sink", "q_norm": "q_norm.weight", "k_norm": "k_norm.weight",
          "gate": "g_proj.weight", "q_conv": "q_conv.weight", "k_conv": "k_conv.weight", "v_conv": "v_conv.weight", "r1": "distance.r1", "r2": "distance.r2"}
NO_WINDOW = 1 << 30   # "every earlier token" as a window size


def _names(params: Mapping, prefix: str) -> Dict[str, str]:
    given = params.get("names") or {}
    return {role: prefix + given.get(role, default) for role, default in _ROLES.items()}


@register_mixer("pooled_window_attention")
class PooledWindowAttention:
    @staticmethod
    def tensors(params: Mapping, prefix: str) -> Dict[str, TensorInfo]:
        w, nh, nkv = params["hidden_size"], params["num_heads"], params["num_kv_heads"]
        d, dv = params["qk_dim"], params["v_dim"]
        nm = _names(params, prefix)
        own, bias = params.get("own_kv", True), params.get("bias", False)
        t = {nm["q"]: TensorInfo((nh * d, w), "matrix"), nm["o"]: TensorInfo((w, nh * dv), "matrix")}
        if own:
            t[nm["k"]] = TensorInfo((nkv * d, w), "matrix")
            t[nm["v"]] = TensorInfo((nkv * dv, w), "matrix")
        if bias:
            t[nm["q_bias"]] = TensorInfo((nh * d,), "vector", False, 0.0)
            if own:
                t[nm["k_bias"]] = TensorInfo((nkv * d,), "vector", False, 0.0)
                t[nm["v_bias"]] = TensorInfo((nkv * dv,), "vector", False, 0.0)
        if params.get("sink", False):
            t[nm["sink"]] = TensorInfo((nh,), "vector", False, 0.0)
        if params.get("proj_norm", False):
            t[nm["q_norm"]] = TensorInfo((nh * d,), "vector")
            if own:
                t[nm["k_norm"]] = TensorInfo((nkv * d,), "vector")
        if params.get("head_gate", False):
            t[nm["gate"]] = TensorInfo((nh, w), "matrix")
        if params.get("value_gate", False):
            t[nm["gate"]] = TensorInfo((nh * dv, w), "matrix")
        if params.get("distance_bias", False):
            t[nm["r1"]], t[nm["r2"]] = TensorInfo((nh,), "vector"), TensorInfo((nh,), "vector")    # both positive
        taps = params.get("conv_taps")
        if taps:
            for role, ch in (("q_conv", nh * d), ("k_conv", nkv * d), ("v_conv", nkv * dv)):
                t[nm[role]] = TensorInfo((ch, int(taps)), "vector", False, 1.0 / int(taps))
        return t

    def __init__(self, params: Mapping, prefix: str, weights, rt: Runtime):
        self.rt = rt
        self.hidden = int(params["hidden_size"])
        self.n_heads, self.n_kv = int(params["num_heads"]), int(params["num_kv_heads"])
        self.qk_dim, self.v_dim = int(params["qk_dim"]), int(params["v_dim"])
        self.scale = float(params["scale"])
        self.eps = float(params.get("eps", 0.0))
        self.unit_norm = bool(params.get("unit_norm", False))
        win, pool = params.get("window"), params.get("pool")
        self.size = int(win) if win is not None else NO_WINDOW
        self.pool = int(pool) if (pool is not None and win is not None) else 0
        if self.n_heads % self.n_kv or self.size < 1 or self.pool < 0:
            raise ValueError(f"pooled_window_attention: {self.n_heads} heads over {self.n_kv} kv heads, window {win}, pool {pool}")
        self.group = self.n_heads // self.n_kv
        self.own_kv = bool(params.get("own_kv", True))
        self.q_dim, self.o_dim = self.n_heads * self.qk_dim, self.n_heads * self.v_dim
        nm = _names(params, prefix)
        self.head_gate = bool(params.get("head_gate", False))
        self.value_gate = bool(params.get("value_gate", False))
        if self.head_gate and self.value_gate:
            raise ValueError("pooled_window_attention: a gate per head or a gate per value, not both")
        self.keep = int(params.get("keep_first", 0) or 0) if win is not None else 0
        self.taps = int(params.get("conv_taps") or 0)
        if self.keep < 0 or not 0 <= self.taps <= K.CONV_MAX_TAPS or (self.taps and not self.own_kv):
            raise ValueError(f"pooled_window_attention: {self.keep} kept tokens, {self.taps} taps (at most {K.CONV_MAX_TAPS}; a layer that "
                             "reads another's keys and values has no convolution)")
        names, rows = [nm["q"]], [self.q_dim]
        if self.own_kv:
            names += [nm["k"], nm["v"]]
            rows += [self.n_kv * self.qk_dim, self.n_kv * self.v_dim]
        self.gate_col = sum(rows)
        if self.head_gate:                 # the gate's logits are columns of the input product
            names.append(nm["gate"])
            rows.append(self.n_heads)
        elif self.value_gate:
            names.append(nm["gate"])
            rows.append(self.o_dim)
        self.w_in = weights.load_fused(names, rows, self.hidden) if len(names) > 1 else weights.load(nm["q"], "matrix")
        self.proj_norm = bool(params.get("proj_norm", False))
        self.q_norm_w = weights.load(nm["q_norm"], "vector") if self.proj_norm else None
        self.k_norm_w = weights.load(nm["k_norm"], "vector") if self.proj_norm and self.own_kv else None
        self.w_o = weights.load(nm["o"], "matrix")
        self.conv_w = None
        if self.taps:
            self.conv_w = torch.cat([weights.load(nm[r], "vector") for r in ("q_conv", "k_conv", "v_conv")]).contiguous()
            K.shortconv_lib()
        bias = bool(params.get("bias", False))
        self.q_bias = weights.load(nm["q_bias"], "vector") if bias else None
        self.k_bias = weights.load(nm["k_bias"], "vector") if bias and self.own_kv else None
        self.v_bias = weights.load(nm["v_bias"], "vector") if bias and self.own_kv else None
        self.sink = weights.load(nm["sink"], "vector") if params.get("sink", False) else None
        if params.get("unit_sink", False):
            if self.sink is not None:
                raise ValueError("pooled_window_attention: a sink with a tensor or one of score 0, not both")
            self.sink = torch.zeros(self.n_heads, dtype=torch.float32, device=rt.device)
        self.value_norm = bool(params.get("value_norm", False))
        qt = params.get("q_temp")
        self.q_temp = (float(qt["coef"]), int(qt["every"])) if qt else None
        self.softcap = float(params["softcap"]) if params.get("softcap") is not None else None
        self.dist_bias = None
        if params.get("distance_bias", False):
            self.dist_bias = tuple(weights.load(nm[r], "vector").to(torch.float32).contiguous() for r in ("r1", "r2"))
        if (self.softcap is not None and not self.softcap > 0.0) or (self.q_temp is not None and self.q_temp[1] < 1):
            raise ValueError(f"pooled_window_attention: softcap {self.softcap}, query temperature {self.q_temp}")
        if self.pool and (self.softcap is not None or self.dist_bias is not None):
            raise ValueError("pooled_window_attention: squashed or biased scores do not go with pooled blocks")
        self.side, self.side_out = None, None      # (first column, columns) of rows that ride with the input product
        pos: PartSpec = params.get("position") or PartSpec("none")
        self.position = POSITIONS.get(pos.kind)(pos.params, self.qk_dim, rt)
        self.interleaved = bool(getattr(self.position, "interleaved", False))
        # the per-token preparation with one block a token takes the norm over whole projections and both rotation layouts
        self.prep_by_token = self.proj_norm or self.interleaved
        if self.prep_by_token and self.taps:
            raise ValueError("pooled_window_attention: the convolution does not go with a norm over the whole projection or the interleaved layout")
        if self.prep_by_token and bias:
            raise ValueError("pooled_window_attention: biases do not go with a norm over the whole projection or the interleaved layout")
        if (self.prep_by_token or self.taps) and (self.value_norm or self.q_temp is not None):
            raise ValueError("pooled_window_attention: a value norm or a query temperature does not go with a convolution, a norm over the "
                             "whole projection or the interleaved layout")
        if self.head_gate:
            K.latent_attn_lib()            # the per-head gate kernel lives beside the other gated attention
        self.rot = int(getattr(self.position, "rotary_dim", 0) or 0) if getattr(self.position, "inv_freq", None) is not None else 0
        K.pool_attention_lib(self.qk_dim, self.v_dim, self.group)   # build (or find) the kernels of this head shape now
        self.use_prefill_kernel = rt.is_bf16 and K.pool_attention_prefill_supported(self.qk_dim, self.v_dim, self.group)
        if self.use_prefill_kernel:
            K.pool_attention_prefill_lib(self.qk_dim, self.v_dim, self.group)

    def absorb_rows(self, w: torch.Tensor) -> bool:
        """Rows of another product of the same input join the input product (behind q | k | v, from a column that is a
        multiple of 8); their result is ``side_out`` after every ``forward``."""
        if w.dtype != self.w_in.dtype or w.dim() != 2 or w.shape[1] != self.hidden or self.side is not None:
            return False
        pad = (-self.w_in.shape[0]) % 8
        fill = [torch.zeros((pad, self.hidden), dtype=w.dtype, device=w.device)] if pad else []
        self.side = (self.w_in.shape[0] + pad, w.shape[0])
        self.w_in = torch.cat([self.w_in] + fill + [w])
        return True

    def kv_need(self) -> Optional[KVNeed]:
        if self.size >= NO_WINDOW:
            return KVNeed(self.n_kv, self.qk_dim, None, self.v_dim)
        # rows that must stay: the window's, and those of the block that is still to be summarised
        return KVNeed(self.n_kv, self.qk_dim, max(self.size, self.pool), self.v_dim, None, True, self.pool or None, self.keep)

    def state_need(self):
        if self.taps < 2:
            return None
        # the projected values of the last tokens, in the type the product leaves: row (position % taps) of a ring
        return {"conv": StateNeed((self.taps, self.conv_w.shape[0]), self.rt.dtype)}

    def _n_splits(self, n_rows: int, max_kv: int) -> int:
        """Keys of a row split over enough blocks to fill the device, a block taking at least 128 keys."""
        keys = min(max(1, max_kv), self.size) + self.keep + (max(1, max_kv) // self.pool if self.pool else 0)
        want = math.ceil(2 * self.rt.sm_count / max(1, n_rows * self.n_kv))
        return max(1, min(32, want, (keys + 127) // 128))

    def forward(self, h: torch.Tensor, ctx: StepContext, cache: CacheEntry, state, owns_cache: bool = True) -> torch.Tensor:
        if owns_cache != self.own_kv:
            raise ValueError("pooled_window_attention: a layer without key and value projections must read another run step's cache")
        n, dev = h.shape[0], h.device
        proj = linear(h, self.w_in, self.rt)
        if self.side is not None:
            self.side_out = proj[:, self.side[0]:self.side[0] + self.side[1]]
        q = torch.empty((n, self.n_heads, self.qk_dim), dtype=h.dtype, device=dev)
        pos = self.position
        if self.prep_by_token:
            K.pool_attn_prep_tok(proj, self.q_norm_w, self.k_norm_w, self.eps, pos.inv_freq if self.rot else None,
                                 getattr(pos, "inv_freq_lo", None) if self.rot else None, self.rot, self.interleaved, ctx.tok_slot,
                                 ctx.tok_pos, q, cache.k, cache.v, cache.page_table, self.n_heads, self.n_kv,
                                 self.eps if self.unit_norm else -1.0, owns_cache)
        else:
            freq = (pos.inv_freq, getattr(pos, "inv_freq_lo", None), self.rot) if self.rot else (None, None, 0)
            ring, unit_eps = state["conv"] if self.taps > 1 else None, self.eps if self.unit_norm else -1.0
            if self.taps and not ctx.decode and self.q_bias is None and owns_cache:
                K.pool_attn_prep_run(proj, *freq, ctx, q, cache.k, cache.v, cache.page_table, self.n_heads, self.n_kv, unit_eps, self.conv_w, ring)
            else:
                K.pool_attn_prep(proj, self.q_bias, self.k_bias, self.v_bias, *freq, ctx.tok_slot, ctx.tok_pos, q, cache.k, cache.v,
                                 cache.page_table, self.n_heads, self.n_kv, unit_eps, owns_cache, conv_w=self.conv_w, ring=ring,
                                 store_ring=ctx.decode, v_eps=self.eps if self.value_norm else -1.0, q_temp=self.q_temp)
            if self.taps > 1 and not ctx.decode:
                K.conv_ring_store(proj, 0, ctx.cu_q, ctx.seq_slot, ctx.tok_pos, state["conv"], ctx.n_seqs)
        pooled = None
        if self.pool:
            pc = cache.pooled
            if pc is None:
                raise ValueError("pooled_window_attention: the cache holds no pooled rows for this run step")
            pooled = (pc.k, pc.v, pc.page_table)
            if cache.fills_pooled:
                K.pool_attn_blocks(cache.k, cache.v, cache.page_table, pc.k, pc.v, pc.page_table, ctx.tok_slot, ctx.tok_pos, n,
                                   self.pool, self.group)
        o = torch.empty((n, self.n_heads, self.v_dim), dtype=h.dtype, device=dev)
        gate = proj[:, self.gate_col:self.gate_col + self.o_dim] if self.value_gate else None     # applied inside the attention
        if self.use_prefill_kernel and not ctx.decode and ctx.n_tiles > 0 and cache.k.shape[2] == 64:
            K.pool_attn_prefill(q, cache.k, cache.v, cache.page_table, pooled, self.sink, ctx.tile_tok0, ctx.tile_rows, ctx.tok_slot,
                                ctx.tok_pos, o, ctx.n_tiles, self.scale, self.size, self.pool, keep=self.keep, gate=gate,
                                softcap=self.softcap, dist_bias=self.dist_bias)
        else:
            s = self._n_splits(n, ctx.max_kv)
            part_o = part_ml = None
            if s > 1:
                part_o = torch.empty((n, self.n_heads, s, self.v_dim), dtype=torch.float32, device=dev)
                part_ml = torch.empty((n, self.n_heads, s, 2), dtype=torch.float32, device=dev)
            K.pool_attn_rows(q, cache.k, cache.v, cache.page_table, pooled, self.sink, ctx.tok_slot, ctx.tok_pos, o, self.scale,
                             self.size, self.pool, s, part_o, part_ml, keep=self.keep, gate=gate, softcap=self.softcap,
                             dist_bias=self.dist_bias)
        o = o.view(n, self.o_dim)
        if self.head_gate:
            K.head_gate_rows(o, proj, self.gate_col, o, self.n_heads, self.v_dim)     # in place: an entry reads only itself
        return linear(o, self.w_o, self.rt)
