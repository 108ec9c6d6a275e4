"""Typed configuration of the Dusupel decoder, read from its own ``config.json`` keys.

The design: a 32-bit residual stream; per layer TWO layer norms (with bias) of the same stream, one in front of the mixer and
one in front of the feed-forward, whose results join the stream together times a constant
(``x <- x + residual_mult * (mixer(norm1(x)) + ff(norm2(x)))``); a stretch of layers that runs several times in a row with the
same weights and a cache or state per pass; a gated delta rule with one decay per head and key channel whose decays and output
gate go through a low rank; two mixers side by side whose results are added with fixed factors -- attention over a sliding window that
also keeps a sequence's first tokens, behind short convolutions of queries, keys and values, with a gate per value, and a gated
delta rule with one decay per head; a gated dense feed-forward.

    architecture        "Dusupel"
    vocab, width, residual_mult
    norm.eps
    loop                absent, or start, stop, times: layers start .. stop-1 run ``times`` times in a row
    layers[i].type      "channel_delta" | "channel_delta_2" (the same mixer) | "parallel"
    layers[i].mixer     channel_delta: heads, kv_heads, dim, vdim, conv
                        parallel: left.{heads, kv_heads, dim, vdim, conv, scale, rot.{dims, base}, mask.{size, keep_first}}, left_scale,
                                  right.{heads, kv_heads, dim, vdim, conv}, right_scale
    layers[i].mlp       null, or kind "dense" with ff

Tensors: ``embed``, ``final.norm``, ``head`` and per layer ``l<i>.norm1``, ``l<i>.norm2`` (each with ``.b``), ``l<i>.mix.*``,
``l<i>.mlp.*``; the ranks of the low-rank maps are their tensors' own.  What the design fixes is a constant in the parts;
everything ``config.json`` gives is read from there.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, List, Mapping, Optional, Tuple

from .kerirax import DEFAULT_MAX_POSITIONS, _rot
from .mogelix import _mapping
from .qwen3 import ConfigError
from .spec import ExtraPart, LayerSpec, ModelSpec, PartSpec, RunStep
from .vobusun import _number, _pos_int

DELTA_TYPES = ("channel_delta", "channel_delta_2")
MIXER_TYPES = DELTA_TYPES + ("parallel",)


def _check_heads(m: Mapping[str, Any], where: str) -> None:
    for key in ("heads", "kv_heads", "dim", "vdim", "conv"):
        _pos_int(m, key, where)
    if m["heads"] % m["kv_heads"]:
        raise ConfigError(f"config.json: {where}.heads ({m['heads']}) must be a multiple of kv_heads ({m['kv_heads']})")


def _check_pair(m: Mapping[str, Any], where: str) -> None:
    left, right = _mapping(m, "left", where), _mapping(m, "right", where)
    lw = where + ".left"
    _check_heads(left, lw)
    _number(left, "scale", lw)
    _rot(left, lw, left["dim"], scaling=False)
    mask = _mapping(left, "mask", lw, optional=True)
    if mask is not None:
        _pos_int(mask, "size", lw + ".mask")
        keep = mask.get("keep_first", 0)
        if isinstance(keep, bool) or not isinstance(keep, int) or keep < 0:
            raise ConfigError(f"config.json: {lw}.mask.keep_first must be an integer >= 0, got {keep!r}")
    _check_heads(right, where + ".right")
    for key in ("left_scale", "right_scale"):
        if key in m:
            _number(m, key, where)


@dataclass(frozen=True)
class DusupelLayer:
    type: str
    mixer: Mapping[str, Any]                 # the validated mixer sizes, as config.json gives them
    mlp: Optional[Mapping[str, Any]]         # the validated feed-forward description, or None


@dataclass(frozen=True)
class DusupelConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    loop: Optional[Tuple[int, int, int]]     # (start, stop, times)
    layers: Tuple[DusupelLayer, ...]
    architecture: str = "Dusupel"

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    # ------------------------------------------------------------------ construction
    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "DusupelConfig":
        vocab, width = _pos_int(raw, "vocab", "config"), _pos_int(raw, "width", "config")
        eps = _number(_mapping(raw, "norm", "config"), "eps", "norm")
        if not eps > 0.0:
            raise ConfigError(f"config.json: norm.eps must be positive, got {eps!r}")
        mult = _number(raw, "residual_mult", "config") if "residual_mult" in raw else 1.0
        layers = raw.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json: layers must be a non-empty list")
        out: List[DusupelLayer] = []
        for i, layer in enumerate(layers):
            where = f"layers[{i}]"
            if not isinstance(layer, Mapping):
                raise ConfigError(f"config.json: {where} must be a mapping")
            kind = layer.get("type")
            if kind not in MIXER_TYPES:
                raise ConfigError(f"config.json: {where}.type {kind!r} is not a mixer of this design (known: {', '.join(MIXER_TYPES)})")
            m = _mapping(layer, "mixer", where)
            (_check_pair if kind == "parallel" else _check_heads)(m, where + ".mixer")
            mlp = _mapping(layer, "mlp", where, optional=True)
            if mlp is not None:
                if mlp.get("kind") != "dense":
                    raise ConfigError(f"config.json: {where}.mlp.kind {mlp.get('kind')!r} is not a feed-forward of this design (known: dense)")
                _pos_int(mlp, "ff", where + ".mlp")
            out.append(DusupelLayer(kind, dict(m), dict(mlp) if mlp is not None else None))
        loop = None
        lp = _mapping(raw, "loop", "config", optional=True)
        if lp is not None:
            times = _pos_int(lp, "times", "loop")
            start, stop = lp.get("start"), lp.get("stop")
            for key, v in (("start", start), ("stop", stop)):
                if isinstance(v, bool) or not isinstance(v, int):
                    raise ConfigError(f"config.json: loop.{key} must be an integer, got {v!r}")
            if not 0 <= start < stop <= len(out):
                raise ConfigError(f"config.json: loop.start .. loop.stop must name layers in order, got {start} .. {stop} of {len(out)}")
            loop = (start, stop, times)
        arch = raw.get("architecture") or (raw.get("architectures") or ["Dusupel"])[0]
        return cls(vocab, width, eps, mult, loop, tuple(out), str(arch))

    def to_dict(self) -> dict:
        """The ``config.json`` this configuration is read back from."""
        layers = [{"type": l.type, "mixer": dict(l.mixer), "mlp": dict(l.mlp) if l.mlp is not None else None} for l in self.layers]
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "residual_mult": self.residual_mult, "layers": layers}
        if self.loop is not None:
            d["loop"] = {"start": self.loop[0], "stop": self.loop[1], "times": self.loop[2]}
        return d

    # ------------------------------------------------------------------ the run order
    def run_order(self) -> List[int]:
        n = len(self.layers)
        if self.loop is None:
            return list(range(n))
        start, stop, times = self.loop
        return list(range(start)) + list(range(start, stop)) * times + list(range(stop, n))

    # ------------------------------------------------------------------ accounting (benchmarks)
    def _delta_weights(self, m: Mapping[str, Any], low_rank: bool) -> int:
        w, H, G, d, dv = self.width, m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        n = (2 * G * d + H * dv + H) * w + w * H * dv
        # random weights give the low-rank maps the key size as their rank
        return n + (2 * d * w + d * (H * d + H * dv) if low_rank else (H + H * dv) * w)

    def _layer_weights(self, l: DusupelLayer) -> int:
        w, m = self.width, l.mixer
        n = 3 * l.mlp["ff"] * w if l.mlp is not None else 0
        if l.type != "parallel":
            return n + self._delta_weights(m, True)
        a = m["left"]
        n += (a["heads"] * a["dim"] + a["kv_heads"] * (a["dim"] + a["vdim"])) * w + 2 * w * a["heads"] * a["vdim"]
        return n + self._delta_weights(m["right"], False)

    def weight_bytes_per_decode_step(self, itemsize: int, batch: int = 1) -> int:
        """Bytes of weights one decode step reads at least: every layer run's matrices (a layer that runs several times is read
        every time) and the output head."""
        return itemsize * (self.vocab * self.width + sum(self._layer_weights(self.layers[i]) for i in self.run_order()))

    def matmul_flops_per_token(self) -> int:
        """Multiply-add flops of the weight matrices one token passes through, output head excluded."""
        return 2 * sum(self._layer_weights(self.layers[i]) for i in self.run_order())

    # ------------------------------------------------------------------ the parts of each layer
    def _delta_spec(self, m: Mapping[str, Any], channel: bool) -> PartSpec:
        names = {r: r for r in ("q", "k", "v", "b", "norm", "o", "dt_bias")}
        names.update({r + "_conv": r + ".conv" for r in ("q", "k", "v")}, a_log="A_log")
        names.update({r: r for r in (("a1", "a2", "g1", "g2") if channel else ("a", "g"))})
        return PartSpec("gated_delta", {
            "hidden_size": self.width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "qk_dim": m["dim"], "v_dim": m["vdim"],
            "taps": m["conv"], "eps": self.norm_eps, "channel_decay": channel, "low_rank": channel,
            "gate_act": "sigmoid" if channel else "silu", "names": names})

    def _mixer_spec(self, l: DusupelLayer) -> PartSpec:
        m = l.mixer
        if l.type != "parallel":
            return self._delta_spec(m, True)
        a = m["left"]
        rot, mask = a.get("rot"), a.get("mask")
        rope = None if rot is None else PartSpec("rope", {"theta": float(rot["base"]), "rotary_dim": int(rot["dims"]), "freq": "rounded_once"})
        left = PartSpec("pooled_window_attention", {
            "hidden_size": self.width, "num_heads": a["heads"], "num_kv_heads": a["kv_heads"], "qk_dim": a["dim"], "v_dim": a["vdim"],
            "scale": float(a["scale"]), "window": mask["size"] if mask is not None else None,
            "keep_first": mask.get("keep_first", 0) if mask is not None else 0, "pool": None, "eps": self.norm_eps, "own_kv": True,
            "position": rope, "sink": False, "bias": False, "unit_norm": False, "conv_taps": a["conv"], "value_gate": True,
            "names": {"q": "q", "k": "k", "v": "v", "o": "o", "gate": "g", "q_conv": "q.conv", "k_conv": "k.conv", "v_conv": "v.conv"}})
        return PartSpec("side_by_side", {"left": left, "right": self._delta_spec(m["right"], False),
                                         "left_scale": float(m.get("left_scale", 1.0)), "right_scale": float(m.get("right_scale", 1.0))})

    def model_spec(self) -> ModelSpec:
        def norm(name: str) -> PartSpec:
            return PartSpec("layernorm", {"size": self.width, "eps": self.norm_eps, "name": name, "bias": name + ".b"})

        specs = []
        for i, l in enumerate(self.layers):
            ffn = None
            if l.mlp is not None:
                ffn = PartSpec("clamped_glu", {"hidden_size": self.width, "intermediate_size": l.mlp["ff"], "limit": None, "alpha": 1.0,
                                               "up_offset": 0.0, "names": {"gate": "gate", "up": "up", "down": "down"}})
            specs.append(LayerSpec(
                block="parallel_norms", mixer=self._mixer_spec(l), ffn=ffn, norm_mixer=norm("norm1"), norm_ffn=norm("norm2") if ffn else None,
                mixer_prefix=f"l{i}.mix.", ffn_prefix=f"l{i}.mlp.", norm_mixer_prefix=f"l{i}.", norm_ffn_prefix=f"l{i}.",
                extra=(ExtraPart("sum", "connection", PartSpec("scaled_sum", {
                    "mult": self.residual_mult, "unread": {} if ffn else {"norm2": self.width, "norm2.b": self.width}}), f"l{i}."),)))
        spec = ModelSpec(
            architecture=self.architecture,
            vocab_size=self.vocab,
            hidden_size=self.width,
            max_positions=DEFAULT_MAX_POSITIONS,
            embedding=PartSpec("pair_embedding", {"vocab_size": self.vocab, "hidden_size": self.width, "name": "embed", "scale": 1.0,
                                                  "pair": None, "norm": None}),
            layers=tuple(specs),
            schedule=tuple(RunStep(layer=i) for i in self.run_order()),
            final_norm=norm("final.norm"),
            head=PartSpec("lm_head", {"vocab_size": self.vocab, "hidden_size": self.width, "tied": False, "name": "head"}),
            embedding_prefix="",
            final_norm_prefix="",
            head_prefix="",
        )
        spec.validate()
        return spec
