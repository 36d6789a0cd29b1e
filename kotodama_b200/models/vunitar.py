"""Vunitar: a decoder-only language model with latent attention and a grouped mixture of experts.

* every token caches one normalised latent of ``kv_rank`` numbers per layer; keys and values are per-head linear
  maps of it (no positions enter the attention);
* a layer normalises the *output* of its sub-layers: ``x += norm1(mixer(x)) * ls1``, ``x += norm2(ff(x)) * ls2``;
* feed-forwards are dense (squared ReLU) or a mixture of small experts (exact GELU) chosen by a softmax router with
  group-limited top-k, with an optional shared expert behind a sigmoid gate, or absent;
* the embedding optionally adds a hashed bigram row of the (previous, current) token pair; logits are soft-capped.

This module is the description of the design: the configuration read from ``config.json`` and the named weights.
``kotodama_b200.serve.runners`` runs it.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Optional

import torch


@dataclass(frozen=True)
class LatentMixer:
    heads: int
    dim: int                       # query / key size per head
    vdim: int                      # value size per head
    kv_rank: int                   # size of the cached latent
    scale: float                   # multiplies the scores


@dataclass(frozen=True)
class DenseMLP:
    ff: int


@dataclass(frozen=True)
class MoEMLP:
    ff: int                        # hidden size of one expert
    experts: int
    top: int
    scale: float = 1.0             # multiplies the chosen experts' scores
    groups: int = 1                # equal groups of neighbouring experts ...
    keep: int = 1                  # ... of which only the best this many are eligible
    shared_ff: int = 0             # hidden size of the shared expert (0: none)


@dataclass(frozen=True)
class Bigram:
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class VunitarLayer:
    mixer: LatentMixer
    mlp: Any                       # DenseMLP | MoEMLP | None


@dataclass
class VunitarConfig:
    vocab_size: int
    hidden_size: int
    layers: list[VunitarLayer]
    norm_eps: float = 1e-5
    logit_softcap: float = 0.0     # 0: none
    bigram: Optional[Bigram] = None
    max_position_embeddings: int = 4096    # default context limit of the serving engine; the design itself has none
    source: dict = field(default_factory=dict, repr=False)

    attn_res = False

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_dict(cls, d: dict[str, Any]) -> "VunitarConfig":
        layers = []
        for i, entry in enumerate(d["layers"]):
            if entry["type"] != "latent_attention":
                raise ValueError(f"layer {i}: unknown mixer '{entry['type']}'")
            m = entry["mixer"]
            mixer = LatentMixer(int(m["heads"]), int(m["dim"]), int(m["vdim"]), int(m["kv_rank"]), float(m["scale"]))
            layers.append(VunitarLayer(mixer, _mlp_from_dict(entry.get("mlp"), i)))
        bg = (d.get("embedding") or {}).get("bigram")
        return cls(vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), layers=layers,
                   norm_eps=float(d["norm"]["eps"]), logit_softcap=float(d.get("logit_softcap") or 0.0),
                   bigram=Bigram(int(bg["buckets"]), int(bg["mul_prev"]), int(bg["mul_cur"])) if bg else None, source=d)

    def to_dict(self) -> dict[str, Any]:
        return dict(self.source)

    def tensor_shapes(self) -> dict[str, tuple[int, ...]]:
        """Every weight's name and shape; linear weights are ``[out, in]``."""
        D = self.hidden_size
        out: dict[str, tuple[int, ...]] = {"embed": (self.vocab_size, D)}
        if self.bigram:
            out["bigram"] = (self.bigram.buckets + 1, D)
        for i, layer in enumerate(self.layers):
            p, m, f = f"l{i}.", layer.mixer, layer.mlp
            out.update({p + "norm1": (D,), p + "mix.q": (m.heads * m.dim, D), p + "mix.dkv": (m.kv_rank, D),
                        p + "mix.dkv.norm": (m.kv_rank,), p + "mix.uk": (m.heads * m.dim, m.kv_rank),
                        p + "mix.uv": (m.heads * m.vdim, m.kv_rank), p + "mix.o": (D, m.heads * m.vdim), p + "ls1": (D,)})
            if f is None:
                continue
            out.update({p + "norm2": (D,), p + "ls2": (D,)})
            if isinstance(f, DenseMLP):
                out.update({p + "mlp.up": (f.ff, D), p + "mlp.down": (D, f.ff)})
                continue
            for e in range(f.experts):
                out.update({p + f"mlp.e{e}.up": (f.ff, D), p + f"mlp.e{e}.down": (D, f.ff)})
            out[p + "mlp.router"] = (f.experts, D)
            if f.shared_ff:
                out.update({p + "mlp.shared.up": (f.shared_ff, D), p + "mlp.shared.down": (D, f.shared_ff),
                            p + "mlp.shared.sg": (1, D)})
        out.update({"final.norm": (D,), "head": (self.vocab_size, D)})
        return out

    def param_count(self) -> int:
        n = 0
        for shape in self.tensor_shapes().values():
            k = 1
            for s in shape:
                k *= s
            n += k
        return n


def _mlp_from_dict(d: Optional[dict], i: int) -> Any:
    if d is None:
        return None
    if d["kind"] == "dense":
        return DenseMLP(int(d["ff"]))
    if d["kind"] != "moe":
        raise ValueError(f"layer {i}: unknown feed-forward '{d['kind']}'")
    r = d["router"]
    g = r.get("groups") or {"count": 1, "keep": 1}
    f = MoEMLP(ff=int(d["expert"]["ff"]), experts=int(r["experts"]), top=int(r["top"]), scale=float(r.get("scale", 1.0)),
               groups=int(g["count"]), keep=int(g["keep"]), shared_ff=int((d.get("shared") or {}).get("ff", 0)))
    if f.experts % f.groups or not 0 < f.keep <= f.groups or not 0 < f.top <= f.keep * (f.experts // f.groups):
        raise ValueError(f"layer {i}: {f.experts} experts in {f.groups} groups, {f.keep} kept, top {f.top}")
    return f


class VunitarModel:
    """The named weights of one model, as loaded (nothing padded, fused or converted)."""

    def __init__(self, config: VunitarConfig, weights: dict[str, torch.Tensor]) -> None:
        self.config = config
        self.weights = weights
        for name, shape in config.tensor_shapes().items():
            if name not in weights:
                raise KeyError(f"weight '{name}' is missing")
            if tuple(weights[name].shape) != shape:
                raise ValueError(f"weight '{name}' has shape {tuple(weights[name].shape)}, the configuration says {shape}")

    @classmethod
    def random_init(cls, config: VunitarConfig, seed: int = 0, device: torch.device | str = "cpu",
                    dtype: torch.dtype = torch.bfloat16) -> "VunitarModel":
        """Unit-variance activations: linear weights ~ N(0, 1 / in), gains near one."""
        gen = torch.Generator(device=device).manual_seed(seed)
        w = {}
        for name, shape in config.tensor_shapes().items():
            t = torch.empty(shape, device=device, dtype=torch.float32).normal_(generator=gen)
            if len(shape) == 1:
                t = 1.0 + 0.1 * t
            elif name not in ("embed", "bigram"):
                t *= shape[1] ** -0.5
            w[name] = t.to(dtype)
        return cls(config, w)

    def eval(self) -> "VunitarModel":
        return self
