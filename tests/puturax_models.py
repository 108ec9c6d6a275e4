"""Small Puturax models for the tests: configurations of the tests' own, weights drawn here (not by the product's
random-weights code), written as a model folder the engine loads."""

from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

from mogelix_models import FP32_TOL, assert_close  # noqa: F401  (the tests' common yardstick)
from tevovik_models import prompts, row_errors, write_model  # noqa: F401  (shared helpers of the tests)


def pair(heads=4, kv_heads=2, dim=16, vdim=24, softcap: Optional[float] = 8.0, q_temp: Optional[tuple] = (0.4, 20), scale=None, rec_heads=3,
         rec_dim=16, left_scale: Optional[float] = 0.8, right_scale: Optional[float] = 1.3, mlp="dense") -> dict:
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else 3.0 / dim}
    if softcap is not None:
        left["softcap"] = softcap
    if q_temp is not None:
        left["q_temp"] = {"coef": q_temp[0], "every": q_temp[1]}
    m = {"left": left, "right": {"heads": rec_heads, "dim": rec_dim}}
    if left_scale is not None:
        m["left_scale"] = left_scale
    if right_scale is not None:
        m["right_scale"] = right_scale
    return {"type": "parallel", "mixer": m, "mlp": _mlp(mlp)}


def latent(heads=3, dim=12, rot_dim=6, vdim=10, q_rank=14, kv_rank=20, base=300.0, scale=None, mlp="moe") -> dict:
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
         "scale": scale if scale is not None else 3.0 / math.sqrt(dim + rot_dim)}
    if rot_dim:
        m["rot"] = {"dims": rot_dim, "base": base}
    return {"type": "latent_attention", "mixer": m, "mlp": _mlp(mlp)}


def moe(ff=16, experts=6, top=2, groups: Optional[tuple] = (3, 2), shared: Optional[int] = 20) -> dict:
    r = {"experts": experts, "top": top}
    if groups is not None:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    f = {"kind": "moe", "expert": {"ff": ff}, "router": r}
    if shared is not None:
        f["shared"] = {"ff": shared}
    return f


def _mlp(kind):
    if kind is None or isinstance(kind, dict):
        return kind
    if kind == "dense":
        return {"kind": "dense", "ff": 56}
    if kind == "moe":
        return moe()
    raise ValueError(kind)


def config(layers: List[dict], width=48, vocab=101, eps=1e-5, emb_scale: Optional[float] = 3.0) -> dict:
    cfg = {"architecture": "Puturax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if emb_scale is not None:
        cfg["embedding"] = {"scale": emb_scale}
    return cfg


# The rank of the decay's low-rank map stands in no configuration: the tests' own choice per (heads, dim) of a recurrence.
def rank_of(rec: dict) -> int:
    return {16: 5, 64: 16, 5: 1, 40: 8, 200: 24, 24: 3}.get(rec["dim"], 1 + rec["dim"] % 9)


# Sizes chosen to differ from one another in everything a kernel could take for granted: key sizes that are no multiple of a
# vector or a warp, values wider and narrower than keys, one query head per key head, several and all; scores squashed and not,
# temperatures that step at every token, rarely and never; state heads of 5, 40 and 200; ranks of 1 and others; latents narrower
# and wider than a warp, no rotated key part, values wider than the rotated keys; one expert, every expert chosen, groups of one,
# one group, no groups, no always-on expert; no feed-forward; absent factors; and one model whose sizes take the tensor-core
# kernels and the few-row products that several mixtures share (head rows in whole tiles, a width of 256).
CONFIGS: Dict[str, dict] = {
    "pair": config([pair(mlp="dense")]),
    "latent": config([latent(mlp="moe")], emb_scale=None),
    "mixed": config([latent(mlp="dense"), pair(mlp="moe"), pair(heads=2, kv_heads=1, dim=8, vdim=8, softcap=None, q_temp=None, rec_heads=2, rec_dim=24,
                                                                   mlp=moe(12, 8, 3, (2, 1), 24)), latent(heads=2, dim=8, rot_dim=4, vdim=16, q_rank=6,
                                                                                                          kv_rank=40, mlp=None)], width=64, vocab=157),
    "sizes": config([pair(heads=6, kv_heads=2, dim=10, vdim=20, softcap=3.0, q_temp=(0.7, 1), rec_heads=7, rec_dim=5, left_scale=None, right_scale=None,
                          mlp=moe(7, 1, 1, None, None)),
                     latent(heads=3, dim=12, rot_dim=0, vdim=7, q_rank=9, kv_rank=21, mlp="dense"),
                     pair(heads=2, kv_heads=2, dim=24, vdim=7, softcap=40.0, q_temp=(1.5, 64), rec_heads=1, rec_dim=200, left_scale=0.3, right_scale=2.0,
                          mlp=moe(9, 4, 4, (4, 4), 11)),
                     pair(heads=3, kv_heads=1, dim=12, vdim=12, softcap=None, q_temp=(0.2, 7), rec_heads=2, rec_dim=40, mlp=None),
                     latent(heads=5, dim=6, rot_dim=10, vdim=29, q_rank=40, kv_rank=33, mlp=moe(5, 6, 3, (6, 4), None))],
                    width=42, vocab=131, eps=3e-4, emb_scale=0.5),
    "tc": config([pair(heads=4, kv_heads=1, dim=32, vdim=48, softcap=9.0, q_temp=(0.3, 50), scale=0.1, rec_heads=3, rec_dim=64, mlp={"kind": "dense", "ff": 128}),
                  latent(heads=4, dim=32, rot_dim=32, vdim=48, q_rank=64, kv_rank=64, mlp=moe(32, 8, 3, (4, 2), 64)),
                  pair(heads=4, kv_heads=4, dim=16, vdim=16, rec_heads=4, rec_dim=16, mlp=moe(32, 8, 2, (2, 2), 32))],
                 width=256, vocab=211),
}


def draw_weights(cfg: dict, seed: int) -> Dict[str, torch.Tensor]:
    """bfloat16 tensors with spreads that make every stage matter (flat scores and logits hide faults): scores spread over
    several units so that single keys, near and far, carry a row; distances that cost a visible share; decays from a few tokens
    to hundreds; bonuses and mixtures of either sign and size; corrections that change choices and push choice scores below
    zero; router logits far enough apart that 16-bit rounding rarely flips a choice."""
    g = torch.Generator().manual_seed(seed)
    w = cfg["width"]

    def mat(rows, cols, gain=1.0):
        return (torch.randn(rows, cols, generator=g) * gain / math.sqrt(cols)).to(torch.bfloat16)

    def vec(n, mean, spread):
        return (mean + torch.randn(n, generator=g) * spread).to(torch.bfloat16)

    def positive(n, mean):
        return (mean * torch.exp(torch.randn(n, generator=g) * 0.6)).to(torch.bfloat16)

    # the table is the output head too: its scale sets the logits' spread
    t = {"embed": mat(cfg["vocab"], w, 3.0), "final.norm": vec(w, 0.0, 0.2)}
    for i, ly in enumerate(cfg["layers"]):
        m, p = ly["mixer"], f"l{i}."
        t[p + "norm1"], t[p + "norm1b"] = vec(w, 0.0, 0.2), vec(w, 0.0, 0.3)
        if ly["type"] == "latent_attention":
            H, d, r, dv, qr, kr = m["heads"], m["dim"], m.get("rot_dim", 0), m["vdim"], m["q_rank"], m["kv_rank"]
            t[p + "mix.dq"] = mat(qr, w, 1.5)
            t[p + "mix.dq.norm"] = vec(qr, 1.0, 0.2)
            t[p + "mix.uq"] = mat(H * (d + r), qr, 2.0)
            t[p + "mix.dkv"] = mat(kr + r, w, 1.5)
            t[p + "mix.dkv.norm"] = vec(kr, 1.0, 0.2)
            t[p + "mix.uk"] = mat(H * d, kr, 2.0)
            t[p + "mix.uv"] = mat(H * dv, kr, 1.5)
            t[p + "mix.g"] = mat(H * dv, w, 2.0)
            t[p + "mix.o"] = mat(w, H * dv, 1.0)
        else:
            a, s = m["left"], m["right"]
            H, G, d, dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            q = p + "mix.left."
            t[q + "q"], t[q + "k"], t[q + "v"] = mat(H * d, w, 2.0), mat(G * d, w, 2.0), mat(G * dv, w, 1.5)
            t[q + "r1"], t[q + "r2"] = positive(H, 0.5), positive(H, 0.2)
            t[q + "g"], t[q + "o"] = mat(H * dv, w, 2.0), mat(w, H * dv, 1.0)
            hd, R = s["heads"] * s["dim"], rank_of(s)
            q = p + "mix.right."
            for j in "rkvgw":
                t[q + "mu." + j] = vec(w, 0.5, 0.4)
            for j in "rkv":
                t[q + j] = mat(hd, w, 1.5)
            t[q + "g"] = mat(hd, w, 2.0)
            t[q + "w1"], t[q + "w2"], t[q + "w0"] = mat(R, w, 1.5), mat(hd, R, 1.5), vec(hd, -3.0, 1.5)
            t[q + "u"], t[q + "norm"] = vec(hd, 0.5, 0.7).view(s["heads"], s["dim"]), vec(hd, 1.0, 0.3)
            t[q + "o"] = mat(w, hd, 1.0)
        f = ly["mlp"]
        if f is None:
            continue
        t[p + "norm2"], t[p + "norm2b"] = vec(w, 0.0, 0.2), vec(w, 0.0, 0.3)
        if f["kind"] == "dense":
            t[p + "mlp.up"], t[p + "mlp.down"] = mat(f["ff"], w, 1.5), mat(w, f["ff"], 1.0)
        else:
            E = f["router"]["experts"]
            t[p + "mlp.router"], t[p + "mlp.correction"] = mat(E, w, 4.0), vec(E, -0.5, 0.4)
            forms = [(f"mlp.e{e}.", f["expert"]["ff"]) for e in range(E)]
            if f.get("shared") is not None:
                forms.append(("mlp.shared.", f["shared"]["ff"]))
            for name, ff in forms:
                t[p + name + "gate"], t[p + name + "up"], t[p + name + "down"] = mat(ff, w, 2.0), mat(ff, w, 2.0), mat(w, ff, 1.0)
    return {k: v.contiguous() for k, v in t.items()}


BF16_TOL = 0.04     # what rounding at every stage does to a typical row of logits of these narrow models (32-bit is the sharp test)
BF16_FAR = 0.2      # ... and to nine rows in ten: rounding flips close calls of the routers


def bf16_limits(cfg: dict, tensors: Dict[str, torch.Tensor], tokens: List[int]):
    """(typical row, nine rows in ten): three times what 16-bit rounding alone does to this model's logits, measured with
    the plain evaluation rounding what enters and leaves its matrix products, and no less than the fixed limits above."""
    import plain_puturax as P

    e = row_errors(P.forward(cfg, tensors, tokens, rounding=torch.bfloat16), P.forward(cfg, tensors, tokens)).double()
    return max(BF16_TOL, 3.0 * float(e.median())), max(BF16_FAR, 3.0 * float(e.quantile(0.9)))
