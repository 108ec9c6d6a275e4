"""Small Dusupel models for the tests: configurations of the tests' own, weights drawn here (not by the product's
random-weights code), written as a model folder the engine loads."""

from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

from mogelix_models import FP32_TOL, assert_close  # noqa: F401  (the tests' common yardstick)
from tevovik_models import prompts, row_errors, write_model  # noqa: F401  (shared helpers of the tests)


def heads(n=4, kv=2, dim=12, vdim=20, conv=3) -> dict:
    return {"heads": n, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}


def delta(m: Optional[dict] = None, ff: Optional[int] = 56, kind="channel_delta", rank=(7, 5)) -> dict:
    """``rank``: of the decay's and the gate's low-rank maps (the tensors carry them, the configuration does not)."""
    return {"type": kind, "mixer": m or heads(), "mlp": None if ff is None else {"kind": "dense", "ff": ff}, "_rank": rank}


def pair(left: Optional[dict] = None, right: Optional[dict] = None, rot: Optional[tuple] = (8, 500.0), mask: Optional[tuple] = (40, 3), scale=None,
         left_scale: Optional[float] = 0.9, right_scale: Optional[float] = 1.3, ff: Optional[int] = 56) -> dict:
    a = dict(left or heads(4, 2, 16, 24, 3))
    a["scale"] = scale if scale is not None else 3.0 / math.sqrt(a["dim"])
    if rot is not None:
        a["rot"] = {"dims": rot[0], "base": rot[1]}
    if mask is not None:
        a["mask"] = {"size": mask[0], "keep_first": mask[1]} if mask[1] is not None else {"size": mask[0]}
    m = {"left": a, "right": dict(right or heads(3, 3, 10, 14, 2))}
    if left_scale is not None:
        m["left_scale"] = left_scale
    if right_scale is not None:
        m["right_scale"] = right_scale
    return {"type": "parallel", "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(layers: List[dict], width=48, vocab=101, eps=1e-5, mult: Optional[float] = 0.6, loop: Optional[tuple] = None) -> dict:
    cfg = {"architecture": "Dusupel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if mult is not None:
        cfg["residual_mult"] = mult
    if loop is not None:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


# Sizes chosen to differ from one another in everything a kernel could take for granted: key sizes that are no multiple of a
# vector or a warp, of three dimensions, up to 200; values wider and narrower than keys; one head per key head, several, all; one tap
# and five (and different counts within a model); ranks that fit no vector and differ; a rotation over part of a head, all of
# it and none; windows below / equal to / above a page, of a single token and none; kept first tokens: none, one, more than a page,
# more than the window; no feed-forward; scales of one and others, left out and given; a stretch of one layer and of several run
# once, twice and three times, from the first layer and from a later one, up to the last layer and short of it; and one model
# whose sizes take the tensor-core kernels.
CONFIGS: Dict[str, dict] = {
    "delta": config([delta()]),
    "pair": config([pair()]),
    "looped": config([delta(heads(2, 2, 8, 8, 4), kind="channel_delta_2", rank=(16, 8)), pair(), delta(heads(4, 1, 20, 12, 4), ff=None),
                      pair(heads(2, 1, 8, 16, 4), heads(4, 2, 36, 24, 4), rot=(8, 90.0), mask=(64, 1), ff=40)],
                     width=64, vocab=157, loop=(1, 3, 2)),
    "sizes": config([pair(heads(6, 2, 10, 18, 1), heads(5, 1, 7, 33, 5), rot=(4, 37.0), mask=(70, 66), left_scale=None, right_scale=None, ff=37),
                     delta(heads(3, 3, 3, 11, 5), ff=29, rank=(1, 3)),
                     pair(heads(3, 1, 12, 7, 5), heads(2, 2, 72, 20, 1), rot=None, mask=(5, 9), left_scale=0.4, right_scale=2.0, ff=None),
                     delta(heads(2, 1, 200, 9, 2), kind="channel_delta_2", ff=None, rank=(11, 2)),
                     pair(heads(2, 2, 6, 6, 2), heads(6, 3, 33, 40, 3), rot=(6, 20.0), mask=None, ff=21)],
                    width=42, vocab=131, eps=3e-4, mult=None, loop=(0, 3, 3)),
    "edges": config([pair(heads(2, 1, 16, 16, 4), heads(2, 1, 16, 16, 4), rot=(16, 1000.0), mask=(1, 0)),
                     pair(heads(2, 1, 16, 16, 4), heads(2, 1, 16, 16, 4), rot=(16, 1000.0), mask=(33, None), left_scale=1.0, right_scale=1.0)],
                    width=56, vocab=77, mult=1.0, loop=(1, 2, 1)),
    "tc": config([pair(heads(4, 2, 64, 64, 4), heads(4, 2, 64, 64, 4), rot=(64, 10000.0), mask=(96, 4), ff=128),
                  delta(heads(4, 4, 128, 64, 4), ff=256, rank=(32, 16))], width=256, vocab=211, loop=(0, 2, 2)),
}


def draw_weights(cfg: dict, seed: int) -> Dict[str, torch.Tensor]:
    """bfloat16 tensors with spreads that make every stage matter (flat scores and logits hide faults): scores spread over
    several units so that single keys, near and far, carry a row; decays from a few tokens to hundreds; writes of very
    different strength; gates on both sides of a half."""
    g = torch.Generator().manual_seed(seed)
    w = cfg["width"]

    def mat(rows, cols, gain=1.0):
        return (torch.randn(rows, cols, generator=g) * gain / math.sqrt(cols)).to(torch.bfloat16)

    def vec(n, mean, spread):
        return (mean + torch.randn(n, generator=g) * spread).to(torch.bfloat16)

    def conv(rows, taps):      # the current token's weight stands out, the others matter
        c = torch.randn(rows, taps, generator=g) * 0.4
        c[:, -1] += 0.8
        return c.to(torch.bfloat16)

    t = {"embed": torch.randn(cfg["vocab"], w, generator=g).to(torch.bfloat16), "head": mat(cfg["vocab"], w, 3.0),
         "final.norm": vec(w, 1.0, 0.2), "final.norm.b": vec(w, 0.0, 0.3)}

    def delta_tensors(p, m, rank):
        H, G, d, dv, taps = (m[k] for k in ("heads", "kv_heads", "dim", "vdim", "conv"))
        for n, rows in (("q", G * d), ("k", G * d), ("v", H * dv)):
            t[p + n], t[p + n + ".conv"] = mat(rows, w, 1.5), conv(rows, taps)
        t[p + "b"] = mat(H, w, 2.0)
        t[p + "A_log"] = vec(H, 0.0, 0.7)
        t[p + "norm"] = vec(dv, 1.0, 0.3)
        t[p + "o"] = mat(w, H * dv, 1.0)
        if rank is None:
            t[p + "a"], t[p + "dt_bias"] = mat(H, w, 1.0), vec(H, -3.0, 1.5)
            t[p + "g"] = mat(H * dv, w, 2.0)
        else:
            t[p + "a1"], t[p + "a2"], t[p + "dt_bias"] = mat(rank[0], w, 1.0), mat(H * d, rank[0], 1.0), vec(H * d, -3.0, 1.5)
            t[p + "g1"], t[p + "g2"] = mat(rank[1], w, 1.5), mat(H * dv, rank[1], 1.5)

    for i, ly in enumerate(cfg["layers"]):
        m, p = ly["mixer"], f"l{i}."
        t[p + "norm1"], t[p + "norm1.b"] = vec(w, 1.0, 0.2), vec(w, 0.0, 0.3)
        if ly["type"] == "parallel":
            a = m["left"]
            H, G, d, dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            for n, rows, gain in (("q", H * d, 1.5), ("k", G * d, 1.5), ("v", G * dv, 1.5)):
                t[p + "mix.left." + n], t[p + "mix.left." + n + ".conv"] = mat(rows, w, gain), conv(rows, a["conv"])
            t[p + "mix.left.g"] = mat(H * dv, w, 2.0)
            t[p + "mix.left.o"] = mat(w, H * dv, 1.0)
            delta_tensors(p + "mix.right.", m["right"], None)
        else:
            delta_tensors(p + "mix.", m, ly["_rank"])
        if ly["mlp"] is not None:
            ff = ly["mlp"]["ff"]
            t[p + "norm2"], t[p + "norm2.b"] = vec(w, 1.0, 0.2), vec(w, 0.0, 0.3)
            t[p + "mlp.gate"], t[p + "mlp.up"], t[p + "mlp.down"] = mat(ff, w, 2.0), mat(ff, w, 2.0), mat(w, ff, 1.0)
    return {k: v.contiguous() for k, v in t.items()}


BF16_TOL = 0.04     # what rounding at every stage does to a typical row of logits of these narrow models (32-bit is the sharp test)
BF16_FAR = 0.1      # ... and to nine rows in ten


def bf16_limits(cfg: dict, tensors: Dict[str, torch.Tensor], tokens: List[int]):
    """(typical row, nine rows in ten): three times what 16-bit rounding alone does to this model's logits, measured with
    the plain evaluation rounding what enters and leaves its matrix products, and no less than the fixed limits above."""
    import plain_dusupel as P

    e = row_errors(P.forward(cfg, tensors, tokens, rounding=torch.bfloat16), P.forward(cfg, tensors, tokens)).double()
    return max(BF16_TOL, 3.0 * float(e.median())), max(BF16_FAR, 3.0 * float(e.quantile(0.9)))
