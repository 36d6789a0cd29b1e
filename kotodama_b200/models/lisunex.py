"""Lisunex: a decoder-only language model of gated delta-rule layers and chunked attention layers, part of which runs
several times in a row.

* every layer entry names its mixer: ``delta`` (a matrix state per head, decayed and corrected token by token, behind short
  causal convolutions) or ``attention`` (grouped heads, YaRN rotary positions, unit-RMS queries and keys, soft-capped scores, keys
  visible inside the query's own chunk of the sequence only, one output gate per head);
* sub-layers are pre-norm; the feed-forward (SwiGLU) is optional per layer;
* layers ``start .. stop - 1`` of the loop run ``times`` times with the same weights; each pass has its own cache and state, and a
  learned vector is added to the residual stream before it.

This module is the description of the design: the configuration read from ``config.json`` and the named weights.
``kotodama_b200.serve.runners`` runs it.
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Any, Optional

import torch


@dataclass(frozen=True)
class Rotary:
    """Rotary positions on the first ``dims`` elements of a head, element ``i`` paired with ``i + dims / 2``; ``factor`` > 0:
    YaRN scaling between ``slow`` and ``fast`` turns over ``original`` positions."""

    dims: int
    base: float
    factor: float = 0.0
    original: float = 0.0
    fast: float = 0.0
    slow: float = 0.0

    @property
    def amplitude(self) -> float:
        """Multiplies cosine and sine."""
        return 0.1 * math.log(self.factor) + 1.0 if self.factor else 1.0

    def frequencies(self) -> torch.Tensor:
        """Angle per position of every pair, fp64 ``[dims / 2]``."""
        i = torch.arange(self.dims // 2, dtype=torch.float64)
        f = self.base ** (-2.0 * i / self.dims)
        if not self.factor:
            return f
        place = lambda turns: self.dims * math.log(self.original / (2.0 * math.pi * turns)) / (2.0 * math.log(self.base))
        lo, hi = max(math.floor(place(self.fast)), 0), min(math.ceil(place(self.slow)), self.dims - 1)
        ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
        return f / self.factor * ramp + f * (1.0 - ramp)

    def table(self, positions: int) -> tuple[torch.Tensor, torch.Tensor]:
        """Cosine and sine, fp32 ``[positions, dims / 2]`` (angles in fp64)."""
        a = torch.arange(positions, dtype=torch.float64)[:, None] * self.frequencies()
        return (a.cos() * self.amplitude).float(), (a.sin() * self.amplitude).float()


@dataclass(frozen=True)
class AttentionMixer:
    heads: int
    kv_heads: int
    dim: int                       # query / key size per head
    vdim: int                      # value size per head
    scale: float                   # multiplies the scores
    softcap: float                 # 0: none
    chunk: int                     # keys of the query's own chunk are visible; 0: all
    rot: Rotary


@dataclass(frozen=True)
class DeltaMixer:
    heads: int                     # value heads; each has a state of dim x vdim
    kv_heads: int                  # query / key heads
    dim: int
    vdim: int
    taps: int                      # of the short convolutions


@dataclass(frozen=True)
class GatedMLP:
    ff: int


@dataclass(frozen=True)
class LisunexLayer:
    mixer: Any                     # AttentionMixer | DeltaMixer
    mlp: Optional[GatedMLP]


@dataclass(frozen=True)
class Loop:
    start: int
    stop: int
    times: int


@dataclass
class LisunexConfig:
    vocab_size: int
    hidden_size: int
    layers: list[LisunexLayer]
    norm_eps: float = 1e-5
    embedding_scale: float = 1.0
    loop: Optional[Loop] = None
    max_position_embeddings: int = 4096    # default context limit of the serving engine; the design itself has none
    source: dict = field(default_factory=dict, repr=False)

    attn_res = False

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_dict(cls, d: dict[str, Any]) -> "LisunexConfig":
        layers = [LisunexLayer(_mixer_from_dict(e["type"], e["mixer"], i), _mlp_from_dict(e.get("mlp"), i))
                  for i, e in enumerate(d["layers"])]
        lp = d.get("loop")
        loop = Loop(int(lp["start"]), int(lp["stop"]), int(lp["times"])) if lp else None
        if loop and not (0 <= loop.start < loop.stop <= len(layers) and loop.times >= 1):
            raise ValueError(f"loop {loop} does not fit {len(layers)} layers")
        return cls(vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), layers=layers, norm_eps=float(d["norm"]["eps"]),
                   embedding_scale=float((d.get("embedding") or {}).get("scale", 1.0)), loop=loop, source=d)

    def to_dict(self) -> dict[str, Any]:
        return dict(self.source)

    def runs(self) -> list[tuple[int, Optional[int]]]:
        """The layers in the order of execution, each with the loop pass that begins right before it (or None)."""
        lp, n = self.loop, len(self.layers)
        if lp is None:
            return [(i, None) for i in range(n)]
        body = [(i, t if i == lp.start else None) for t in range(lp.times) for i in range(lp.start, lp.stop)]
        return [(i, None) for i in range(lp.start)] + body + [(i, None) for i in range(lp.stop, n)]

    def tensor_shapes(self) -> dict[str, tuple[int, ...]]:
        """Every weight's name and shape; linear weights are ``[out, in]``."""
        D = self.hidden_size
        out: dict[str, tuple[int, ...]] = {"embed": (self.vocab_size, D)}
        if self.loop:
            out["loop.step"] = (self.loop.times, D)
        for i, layer in enumerate(self.layers):
            p, m = f"l{i}.", layer.mixer
            nq = (m.heads if isinstance(m, AttentionMixer) else m.kv_heads) * m.dim
            nk, nv = m.kv_heads * m.dim, (m.kv_heads if isinstance(m, AttentionMixer) else m.heads) * m.vdim
            out[p + "norm1"] = (D,)
            out.update({p + "mix.q": (nq, D), p + "mix.k": (nk, D), p + "mix.v": (nv, D)})
            if isinstance(m, AttentionMixer):
                out.update({p + "mix.q.b": (nq,), p + "mix.k.b": (nk,), p + "mix.v.b": (nv,), p + "mix.g": (m.heads, D)})
            else:
                out.update({p + "mix.q.conv": (nq, m.taps), p + "mix.k.conv": (nk, m.taps), p + "mix.v.conv": (nv, m.taps),
                            p + "mix.a": (m.heads, D), p + "mix.b": (m.heads, D), p + "mix.A_log": (m.heads,),
                            p + "mix.dt_bias": (m.heads,), p + "mix.norm": (m.vdim,), p + "mix.g": (nv, D)})
            out[p + "mix.o"] = (D, m.heads * m.vdim)
            if layer.mlp is not None:
                ff = layer.mlp.ff
                out.update({p + "norm2": (D,), p + "mlp.gate": (ff, D), p + "mlp.up": (ff, D), p + "mlp.down": (D, ff)})
        out.update({"final.norm": (D,), "head": (self.vocab_size, D)})
        return out

    def param_count(self) -> int:
        return sum(math.prod(s) for s in self.tensor_shapes().values())


def _mixer_from_dict(kind: str, m: dict, i: int) -> Any:
    if kind not in ("attention", "delta"):
        raise ValueError(f"layer {i}: unknown mixer '{kind}'")
    heads, groups, dim, vdim = (int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
    if heads % groups:
        raise ValueError(f"layer {i}: {heads} heads in {groups} groups")
    if kind == "delta":
        return DeltaMixer(heads, groups, dim, vdim, int(m["conv"]))
    r = m["rot"]
    s = r.get("scaling")
    rot = Rotary(int(r["dims"]), float(r["base"]), *((float(s[k]) for k in ("factor", "original", "fast", "slow")) if s else ()))
    if rot.dims % 2 or rot.dims > dim:
        raise ValueError(f"layer {i}: rotary size {rot.dims} for heads of {dim}")
    return AttentionMixer(heads, groups, dim, vdim, float(m["scale"]), float(m.get("softcap") or 0.0),
                          int((m.get("mask") or {}).get("size") or 0), rot)


def _mlp_from_dict(d: Optional[dict], i: int) -> Optional[GatedMLP]:
    if d is None:
        return None
    if d["kind"] != "dense":
        raise ValueError(f"layer {i}: unknown feed-forward '{d['kind']}'")
    return GatedMLP(int(d["ff"]))


class LisunexModel:
    """The named weights of one model, as loaded (nothing padded, fused or converted)."""

    def __init__(self, config: LisunexConfig, weights: dict[str, torch.Tensor]) -> None:
        self.config = config
        self.weights = weights
        for name, shape in config.tensor_shapes().items():
            if name not in weights:
                raise KeyError(f"weight '{name}' is missing")
            if tuple(weights[name].shape) != shape:
                raise ValueError(f"weight '{name}' has shape {tuple(weights[name].shape)}, the configuration says {shape}")

    @classmethod
    def random_init(cls, config: LisunexConfig, seed: int = 0, device: torch.device | str = "cpu",
                    dtype: torch.dtype = torch.bfloat16) -> "LisunexModel":
        """Unit-variance activations: linear weights ~ N(0, 1 / in), gains near one, decays from fast to slow."""
        gen = torch.Generator(device=device).manual_seed(seed)
        w = {}
        for name, shape in config.tensor_shapes().items():
            t = torch.empty(shape, device=device, dtype=torch.float32).normal_(generator=gen)
            if name.endswith(".A_log"):
                t = 0.5 * t - 1.0
            elif name.endswith((".dt_bias", ".q.b", ".k.b", ".v.b")) or name == "loop.step":
                t = 0.5 * t
            elif name.endswith(".conv"):
                t *= shape[1] ** -0.5
            elif len(shape) == 1:
                t = 1.0 + 0.1 * t
            elif name != "embed":
                t *= shape[1] ** -0.5
            w[name] = t.to(dtype)
        return cls(config, w)

    def eval(self) -> "LisunexModel":
        return self
