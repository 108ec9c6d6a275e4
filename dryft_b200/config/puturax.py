"""Typed configuration of the Puturax decoder, read from its own ``config.json`` keys.

The design: a 32-bit residual stream; every sublayer between two norms whose stored weights are deviations from one
(``x <- x + norm1b(mixer(norm1(x)))``, then ``x <- x + norm2b(ff(norm2(x)))``).  Two kinds of mixer -- attention over low-rank
latents with a gate per value, and two mixers side by side whose results are added with fixed factors: grouped-query attention
without rotation (queries, keys and values divided by their root mean square per head, queries multiplied by a temperature that
grows with the position, scores squashed by ``cap * tanh(. / cap)`` from which a logarithm of the distance is taken off, a one in
the softmax's denominator, a gate per value) and time mixing (a matrix state per head that decays per key channel, projections
that read mixtures of the token's and the previous token's input).  Two kinds of feed-forward -- an ungated dense one with the
square of relu, and routed experts (sigmoid scores, a correction that only the choice sees, groups ranked by their two best,
weights divided by their sum) beside an expert that always runs.  The output head is the embedding table.

    architecture        "Puturax"
    vocab, width
    embedding.scale     (absent: 1)
    norm.eps
    layers[i].type      "latent_attention" | "parallel"
    layers[i].mixer     latent_attention: heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot.{dims, base}
                        parallel: left.{heads, kv_heads, dim, vdim, scale, softcap, q_temp.{coef, every}}, left_scale,
                                  right.{heads, dim}, right_scale
    layers[i].mlp       null, or kind "dense" with ff, or kind "moe" with expert.ff, router.{experts, top, groups.{count, keep}},
                        shared.ff

Tensors: ``embed``, ``final.norm`` and per layer ``l<i>.norm1``, ``norm1b``, ``norm2``, ``norm2b``, ``l<i>.mix.*``, ``l<i>.mlp.*``.
Absent ``softcap``, ``q_temp``, ``groups``, ``shared``, ``left_scale`` and ``right_scale`` are served.  What the design fixes is a
constant below; everything ``config.json`` gives is read from there.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, List, Mapping, Optional, Tuple

from .kerirax import _check_latent
from .mogelix import _mapping
from .qwen3 import ConfigError
from .spec import ExtraPart, LayerSpec, ModelSpec, PartSpec, RunStep
from .vobusun import _number, _pos_int

RENORM_EPS = 1e-20                # joins the sum that the chosen experts' scores are divided by
DEFAULT_MAX_POSITIONS = 1 << 20   # the design has no longest sequence; the engine's own limits apply
MIXER_TYPES = ("latent_attention", "parallel")
MLP_KINDS = ("dense", "moe")


def _check_pair(m: Mapping[str, Any], where: str) -> None:
    left, right = _mapping(m, "left", where), _mapping(m, "right", where)
    lw, rw = where + ".left", where + ".right"
    heads, kv = _pos_int(left, "heads", lw), _pos_int(left, "kv_heads", lw)
    _pos_int(left, "dim", lw)
    _pos_int(left, "vdim", lw)
    if heads % kv:
        raise ConfigError(f"config.json: {lw}.heads ({heads}) must be a multiple of kv_heads ({kv})")
    _number(left, "scale", lw)
    if left.get("softcap") is not None and not _number(left, "softcap", lw) > 0.0:
        raise ConfigError(f"config.json: {lw}.softcap must be positive, got {left['softcap']!r}")
    qt = _mapping(left, "q_temp", lw, optional=True)
    if qt is not None:
        _number(qt, "coef", lw + ".q_temp")
        every = _number(qt, "every", lw + ".q_temp")
        if every < 1.0 or every != int(every):
            raise ConfigError(f"config.json: {lw}.q_temp.every must be a whole number of positions, got {qt['every']!r}")
    _pos_int(right, "heads", rw)
    _pos_int(right, "dim", rw)
    for key in ("left_scale", "right_scale"):
        if key in m:
            _number(m, key, where)


def _check_mlp(mlp: Mapping[str, Any], where: str) -> None:
    if mlp.get("kind") not in MLP_KINDS:
        raise ConfigError(f"config.json: {where}.kind {mlp.get('kind')!r} is not a feed-forward of this design (known: {', '.join(MLP_KINDS)})")
    if mlp["kind"] == "dense":
        _pos_int(mlp, "ff", where)
        return
    _pos_int(_mapping(mlp, "expert", where), "ff", where + ".expert")
    r, rw = _mapping(mlp, "router", where), where + ".router"
    experts, top = _pos_int(r, "experts", rw), _pos_int(r, "top", rw)
    groups = _mapping(r, "groups", rw, optional=True)
    allowed = experts
    if groups is not None:
        count, keep = _pos_int(groups, "count", rw + ".groups"), _pos_int(groups, "keep", rw + ".groups")
        if experts % count or keep > count:
            raise ConfigError(f"config.json: {rw}.groups: {experts} experts do not form {count} equal groups of which {keep} are kept")
        allowed = experts // count * keep
    if top > allowed:
        raise ConfigError(f"config.json: {rw}.top ({top}) exceeds the {allowed} experts that can be chosen")
    sh = _mapping(mlp, "shared", where, optional=True)
    if sh is not None:
        _pos_int(sh, "ff", where + ".shared")


@dataclass(frozen=True)
class PuturaxLayer:
    type: str
    mixer: Mapping[str, Any]                 # the validated mixer sizes, as config.json gives them
    mlp: Optional[Mapping[str, Any]]         # the validated feed-forward description, or None


@dataclass(frozen=True)
class PuturaxConfig:
    vocab: int
    width: int
    norm_eps: float
    embed_scale: float
    layers: Tuple[PuturaxLayer, ...]
    architecture: str = "Puturax"

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    # ------------------------------------------------------------------ construction
    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "PuturaxConfig":
        vocab, width = _pos_int(raw, "vocab", "config"), _pos_int(raw, "width", "config")
        eps = _number(_mapping(raw, "norm", "config"), "eps", "norm")
        if not eps > 0.0:
            raise ConfigError(f"config.json: norm.eps must be positive, got {eps!r}")
        emb = _mapping(raw, "embedding", "config", optional=True)
        scale = _number(emb, "scale", "embedding") if emb is not None and "scale" in emb else 1.0
        layers = raw.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json: layers must be a non-empty list")
        out: List[PuturaxLayer] = []
        for i, layer in enumerate(layers):
            where = f"layers[{i}]"
            if not isinstance(layer, Mapping):
                raise ConfigError(f"config.json: {where} must be a mapping")
            kind = layer.get("type")
            if kind not in MIXER_TYPES:
                raise ConfigError(f"config.json: {where}.type {kind!r} is not a mixer of this design (known: {', '.join(MIXER_TYPES)})")
            m = _mapping(layer, "mixer", where)
            (_check_latent if kind == "latent_attention" else _check_pair)(m, where + ".mixer")
            mlp = _mapping(layer, "mlp", where, optional=True)
            if mlp is not None:
                _check_mlp(mlp, where + ".mlp")
            out.append(PuturaxLayer(kind, dict(m), dict(mlp) if mlp is not None else None))
        arch = raw.get("architecture") or (raw.get("architectures") or ["Puturax"])[0]
        return cls(vocab, width, eps, scale, tuple(out), str(arch))

    def to_dict(self) -> dict:
        """The ``config.json`` this configuration is read back from."""
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                "embedding": {"scale": self.embed_scale},
                "layers": [{"type": l.type, "mixer": dict(l.mixer), "mlp": dict(l.mlp) if l.mlp is not None else None} for l in self.layers]}

    # ------------------------------------------------------------------ accounting (benchmarks)
    def _mixer_weights(self, l: PuturaxLayer) -> int:
        w, m = self.width, l.mixer
        if l.type == "latent_attention":
            r = m.get("rot_dim", 0)
            return ((m["q_rank"] + m["kv_rank"] + r) * w + m["heads"] * (m["dim"] + r) * m["q_rank"]
                    + m["heads"] * (m["dim"] + m["vdim"]) * m["kv_rank"] + 2 * w * m["heads"] * m["vdim"])
        a, s = m["left"], m["right"]
        hd, rank = s["heads"] * s["dim"], max(8, s["dim"] // 2)      # the rank that random weights use
        return ((a["heads"] * a["dim"] + a["kv_heads"] * (a["dim"] + a["vdim"]) + 2 * a["heads"] * a["vdim"]) * w
                + 5 * hd * w + rank * (w + hd))

    def _mlp_weights(self, l: PuturaxLayer, experts_read: Optional[int]) -> int:
        """Feed-forward weights a token passes through (``experts_read=None``: its ``top`` experts) or a step reads."""
        w, f = self.width, l.mlp
        if f is None:
            return 0
        if f["kind"] == "dense":
            return 2 * f["ff"] * w
        r = f["router"]
        n = r["experts"] * w + (r["top"] if experts_read is None else min(r["experts"], experts_read)) * 3 * f["expert"]["ff"] * w
        return n + (3 * f["shared"]["ff"] * w if f.get("shared") is not None else 0)

    def weight_bytes_per_decode_step(self, itemsize: int, batch: int = 1) -> int:
        """Bytes of weights one decode step of ``batch`` tokens reads at least: every layer's matrices, the experts the tokens
        choose and the output head."""
        total = self.vocab * self.width
        for l in self.layers:
            top = l.mlp["router"]["top"] if l.mlp is not None and l.mlp["kind"] == "moe" else 0
            total += self._mixer_weights(l) + self._mlp_weights(l, batch * top)
        return itemsize * total

    def matmul_flops_per_token(self) -> int:
        """Multiply-add flops of the weight matrices one token passes through, output head excluded."""
        return 2 * sum(self._mixer_weights(l) + self._mlp_weights(l, None) for l in self.layers)

    # ------------------------------------------------------------------ the parts of each layer
    def _mixer_spec(self, l: PuturaxLayer) -> PartSpec:
        m, w = l.mixer, self.width
        if l.type == "latent_attention":
            rot = m.get("rot") if m.get("rot_dim", 0) else None
            position = PartSpec("rope", {"theta": float(rot["base"]), "rotary_dim": int(rot["dims"]), "layout": "half",
                                         "freq": "rounded_once"}) if rot is not None else None
            return PartSpec("latent_attention", {
                "hidden_size": w, "num_heads": m["heads"], "qk_dim": m["dim"], "rot_dim": m.get("rot_dim", 0), "v_dim": m["vdim"],
                "q_rank": m["q_rank"], "kv_rank": m["kv_rank"], "scale": float(m["scale"]), "eps": self.norm_eps, "window": None,
                "gate": "value", "sink": False, "position": position,
                "names": {"dq": "dq", "dq_norm": "dq.norm", "uq": "uq", "dkv": "dkv", "dkv_norm": "dkv.norm", "uk": "uk", "uv": "uv",
                          "gate": "g", "o": "o"}})
        a, s = m["left"], m["right"]
        qt = a.get("q_temp")
        left = PartSpec("pooled_window_attention", {
            "hidden_size": w, "num_heads": a["heads"], "num_kv_heads": a["kv_heads"], "qk_dim": a["dim"], "v_dim": a["vdim"],
            "scale": float(a["scale"]), "window": None, "pool": None, "eps": self.norm_eps, "own_kv": True, "position": None,
            "unit_norm": True, "value_norm": True, "q_temp": {"coef": float(qt["coef"]), "every": int(qt["every"])} if qt else None,
            "softcap": float(a["softcap"]) if a.get("softcap") is not None else None, "distance_bias": True, "unit_sink": True,
            "value_gate": True, "names": {"q": "q", "k": "k", "v": "v", "o": "o", "gate": "g", "r1": "r1", "r2": "r2"}})
        right = PartSpec("time_mixing", {
            "hidden_size": w, "num_heads": s["heads"], "dim": s["dim"], "eps": self.norm_eps,
            "names": {**{"mu_" + j: "mu." + j for j in ("r", "k", "v", "g", "w")}, "r": "r", "k": "k", "v": "v", "g": "g", "w1": "w1", "w2": "w2",
                      "w0": "w0", "u": "u", "norm": "norm", "o": "o"}})
        return PartSpec("side_by_side", {"left": left, "right": right, "left_scale": float(m.get("left_scale", 1.0)),
                                         "right_scale": float(m.get("right_scale", 1.0))})

    def _ffn_spec(self, l: PuturaxLayer) -> Optional[PartSpec]:
        f = l.mlp
        if f is None:
            return None
        if f["kind"] == "dense":
            return PartSpec("relu2_mlp", {"hidden_size": self.width, "intermediate_size": f["ff"], "names": {"up": "up", "down": "down"}})
        r = f["router"]
        groups = r.get("groups") or {"count": 1, "keep": 1}
        shared = {"intermediate_size": f["shared"]["ff"], "gate": False} if f.get("shared") is not None else None
        return PartSpec("moe", {
            "hidden_size": self.width, "intermediate_size": f["expert"]["ff"], "experts": r["experts"], "top": r["top"],
            "groups": groups["count"], "keep": groups["keep"], "group_rank": "top2", "correction": True, "renormalize": True,
            "renorm_eps": RENORM_EPS, "score": "sigmoid", "activation": "swiglu", "shared": shared,
            "names": {"router": "router", "correction": "correction", "expert": "e{}.", "shared": "shared.", "gate": "gate", "up": "up",
                      "down": "down"}})

    def model_spec(self) -> ModelSpec:
        def norm(name: str) -> PartSpec:
            # the stored weight is the factor's distance from one
            return PartSpec("rmsnorm_offset", {"size": self.width, "eps": self.norm_eps, "offset": 1.0, "name": name})

        specs = []
        for i, l in enumerate(self.layers):
            p = f"l{i}."
            extra = [ExtraPart("mixer_out", "norm", norm("norm1b"), p)]
            if l.mlp is not None:
                extra.append(ExtraPart("ffn_out", "norm", norm("norm2b"), p))
            else:       # a checkpoint may hold the norms of a feed-forward that the layer leaves out
                extra.append(ExtraPart("unread", "connection", PartSpec("scaled_sum", {"unread": {"norm2": self.width, "norm2b": self.width}}), p))
            specs.append(LayerSpec(
                block="sandwich", mixer=self._mixer_spec(l), ffn=self._ffn_spec(l), norm_mixer=norm("norm1"),
                norm_ffn=norm("norm2") if l.mlp is not None else None,
                mixer_prefix=p + "mix.", ffn_prefix=p + "mlp.", norm_mixer_prefix=p, norm_ffn_prefix=p, extra=tuple(extra)))
        spec = ModelSpec(
            architecture=self.architecture,
            vocab_size=self.vocab,
            hidden_size=self.width,
            max_positions=DEFAULT_MAX_POSITIONS,
            embedding=PartSpec("pair_embedding", {"vocab_size": self.vocab, "hidden_size": self.width, "name": "embed",
                                                  "scale": self.embed_scale, "pair": None, "norm": None}),
            layers=tuple(specs),
            schedule=tuple(RunStep(layer=i) for i in range(len(specs))),
            final_norm=norm("final.norm"),
            head=PartSpec("lm_head", {"vocab_size": self.vocab, "hidden_size": self.width, "tied": True, "name": "head"}),
            embedding_prefix="",
            final_norm_prefix="",
            head_prefix="",
        )
        spec.validate()
        return spec
