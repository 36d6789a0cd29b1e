"""Model runners: the layer pipeline of each model family and the cache it keeps, behind one interface for the
serving engine.

A runner has ``make_cache(pages)``, ``forward(batch) -> logits[rows]`` and three traits: ``continues`` (a pass may
start from a cached context), ``needs_prev`` (the embedding looks at the token before) and ``context_buckets`` (the decode
attention is launched for a context size, so decode graphs are captured per size).  A runner that continues also has
``first_visible(n)``: the first position that tokens from position ``n`` on can still see.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Optional

import torch

from ..engine import ParamArena
from ..models.lisunex import AttentionMixer, DeltaMixer, LisunexModel
from ..models.registry import family_of
from ..models.vunitar import DenseMLP, MoEMLP, VunitarModel
from .cache import HybridCache, PagedKVCache, PagedLatentCache


@dataclass
class Batch:
    """One pass: the next tokens of several sequences, packed back to back."""

    ids: torch.Tensor                              # [N] int64
    positions: torch.Tensor                        # [N] int32
    slots: torch.Tensor                            # [N] int64 cache slot of every token
    rows: torch.Tensor                             # packed rows whose logits are asked for
    prev: Optional[torch.Tensor] = None            # [N] int32 the token before (-1: first of its sequence)
    decode: bool = False                           # one token per sequence
    cu_seqlens: Optional[torch.Tensor] = None      # [B + 1] first row of every sequence (not for decode)
    max_seqlen: int = 1
    page_table: Optional[torch.Tensor] = None      # [B, pages]
    ctx_lens: Optional[torch.Tensor] = None        # [B] tokens in the cache after this pass
    max_ctx: int = 0
    cu_context: Optional[torch.Tensor] = None      # [B + 1] prefix sums of ctx_lens
    total_context: int = 0
    states: Optional[torch.Tensor] = None          # [B] int32 state slot of every sequence (-1: its state is not kept)
    spans: Optional[list[tuple[int, int]]] = None  # per sequence (tokens in the cache before, new tokens); not for decode


def make_runner(engine: Any) -> Any:
    return globals()[family_of(engine.model).runner](engine)


class LlamaRunner:
    """Llama-family decoder with block attention residuals (``models/llama.py``): the executor's forward schedule
    on the same ops backend, keys and values in the paged cache."""

    continues = False
    needs_prev = False
    context_buckets = True

    def __init__(self, eng: Any) -> None:
        self.ops, self.cfg, self.tp, self.model = eng.ops, eng.model.config, eng.tp, eng.model
        self.device, self.dtype = eng.device, eng.dtype
        if self.tp is not None:
            self.tp.prepare_model(self.model)
        ar = self.arena = ParamArena(self.model, self.device, self.dtype, with_grads=False)
        cfg = self.cfg
        tpn = self.tp.size if self.tp is not None else 1
        self.H, self.KV = cfg.num_attention_heads // tpn, cfg.num_kv_heads // tpn
        self.hd = cfg.head_dim
        self.layers = []
        for i in range(cfg.num_layers):
            p = f"layers.{i}."
            g = lambda n: ar.view(p + n) if (p + n) in ar.by_name else None
            dw = self.ops.decode_weight          # on CUDA: adds the tile-major copy that decode-size products stream
            self.layers.append(dict(
                wqkv=dw(ar.fused(p + "attn.q_proj.weight", p + "attn.v_proj.weight")), wo=dw(ar.view(p + "attn.o_proj.weight")),
                wgu=dw(ar.fused(p + "ffn.gate_proj.weight", p + "ffn.up_proj.weight")), wd=dw(ar.view(p + "ffn.down_proj.weight")),
                attn_norm=g("attn_norm.weight"), ffn_norm=g("ffn_norm.weight"), qn=g("attn.q_norm.weight"),
                kn=g("attn.k_norm.weight"), aq=g("attn_res_query"), an=g("attn_res_norm.weight"),
                mq=g("mlp_res_query"), mn=g("mlp_res_norm.weight")))
        self.boundaries = frozenset(cfg.boundaries()) if cfg.attn_res else frozenset()
        self.cache: Any = None

    def make_cache(self, pages: int) -> PagedKVCache:
        self.cache = PagedKVCache(self.cfg, pages, self.device, self.dtype, n_kv_local=self.KV)
        return self.cache

    @torch.no_grad()
    def forward(self, b: Batch) -> torch.Tensor:
        """Runs all layers; keys/values go to ``b.slots`` (negative = padding, dropped).  A decode batch attends to
        the paged cache, any other to itself (causal within each of its sequences)."""
        ops, cfg, ar = self.ops, self.cfg, self.arena
        H, KV, hd = self.H, self.KV, self.hd
        eps = cfg.norm_eps
        cos, sin = self.model.rope_cos, self.model.rope_sin
        N = b.ids.numel()
        x = ops.embedding_fwd(b.ids, ar.view("embed_tokens.weight"))
        committed: list[torch.Tensor] = []
        partial: Optional[torch.Tensor] = x
        for i, lw in enumerate(self.layers):
            xn, _ = ops.route_norm_fwd(committed + [partial], lw["aq"], lw["an"], lw["attn_norm"], eps)
            if i in self.boundaries:
                committed = committed + [partial]
                partial = None
            qkv = ops.gemm_nt(xn, lw["wqkv"])
            # QK-norm + RoPE; the same launch puts the new keys and values into their cache slots
            qk, _ = ops.qknorm_rope_fwd(qkv, lw["qn"], lw["kn"], cos, sin, N, H, KV, hd, eps, positions=b.positions,
                                        append=(self.cache.k[i], self.cache.v[i], b.slots))
            k_rows = qk[:, H * hd:]
            v_rows = qkv[:, (H + KV) * hd:]
            if not b.decode:
                o, _ = ops.attention_fwd(qk[:, : H * hd].view(1, N, H, hd), k_rows.view(1, N, KV, hd),
                                         v_rows.view(1, N, KV, hd), need_grad=False, cu_seqlens=b.cu_seqlens,
                                         max_seqlen=b.max_seqlen)
                attn = o.reshape(N, H * hd)
            else:
                attn = ops.paged_decode_attention(qk[:, : H * hd], self.cache.k[i], self.cache.v[i],
                                                  b.page_table, b.ctx_lens, b.max_ctx, H, KV, hd)
            partial = self._row_linear(attn, lw["wo"], partial)
            xn2, _ = ops.route_norm_fwd(committed + [partial], lw["mq"], lw["mn"], lw["ffn_norm"], eps)
            act = ops.swiglu_fwd(ops.gemm_nt(xn2, lw["wgu"]))
            partial = self._row_linear(act, lw["wd"], partial)
        g = lambda n: ar.view(n) if n in ar.by_name else None
        xf, _ = ops.route_norm_fwd([s[b.rows] for s in committed + [partial]], g("final_res_query"),
                                   g("final_res_norm.weight"), ar.view("norm.weight"), eps)
        return ops.gemm_nt(xf, self.model.get_lm_head_weight())

    def _row_linear(self, x: torch.Tensor, w: torch.Tensor, residual: Optional[torch.Tensor]) -> torch.Tensor:
        if self.tp is None:
            return self.ops.gemm_nt(x, w, residual=residual)
        return self.tp.row_linear(self.ops, x, w, residual)


def _up(n: int, a: int) -> int:
    return (n + a - 1) // a * a


def _pad(t: torch.Tensor, *shape: int) -> torch.Tensor:
    """Zeros behind ``t`` in every dimension, up to ``shape``."""
    if tuple(t.shape) == shape:
        return t
    out = torch.zeros(shape, dtype=t.dtype, device=t.device)
    out[tuple(slice(0, n) for n in t.shape)] = t
    return out


class LatentRunner:
    """Latent-attention decoder with dense / mixture-of-experts feed-forwards and output norms
    (``models/vunitar.py``).

    The residual stream is fp32; the sub-layers read its rounding to the engine's dtype.  Per layer the cache keeps the
    normalised latent ``c`` of every token.  Two forms of the attention give the same numbers:

    * decoding and short portions work on the latents themselves: ``q . (W_uk c) = (W_uk^T q) . c`` and
      ``sum p W_uv c = W_uv sum p c``, so every cached row is read once for all heads;
    * long portions expand keys and values of the context (two products over ``c``) and run the flash kernel, whose
      cost per (query, key) pair is the head size instead of the latent size.

    Weights are padded once, at load, to what the kernels' tiles want (zero rows and columns, which change no sum).
    """

    continues = True
    context_buckets = False

    def __init__(self, eng: Any) -> None:
        if eng.tp is not None:
            raise ValueError("latent-attention models are served on one GPU")
        self.ops, self.device, self.dtype = eng.ops, eng.device, eng.dtype
        model: VunitarModel = eng.model
        cfg = self.cfg = model.config
        self.needs_prev = cfg.bigram is not None
        self.D = cfg.hidden_size
        self.Dp = _up(self.D, 8)
        self.short_portion = 16                 # most tokens per sequence for the latent form of the attention
        w = model.weights
        put = lambda t: t.to(self.device, self.dtype).contiguous()
        vec = lambda t, n: _pad(t.to(self.device, torch.float32), n)
        lin = lambda t, n, k: _pad(put(t), n, k)
        dw = self.ops.decode_weight
        Dp = self.Dp
        self.embed = lin(w["embed"], cfg.vocab_size, Dp)
        self.bigram = lin(w["bigram"], cfg.bigram.buckets + 1, Dp) if cfg.bigram else None
        self.layers = []
        for i, layer in enumerate(cfg.layers):
            p, m = f"l{i}.", layer.mixer
            # head sizes of the flash kernel where they fit (keys and values then share one size), else only the latent form
            fits = max(m.dim, m.vdim) <= 128 and self.ops.flash_latent(self.dtype)
            dp = dv = (64 if max(m.dim, m.vdim) <= 64 else 128) if fits else 0
            if not fits:
                dp, dv = _up(m.dim, 8), _up(m.vdim, 8)
            R = _up(m.kv_rank, self.ops.latent_multiple(self.dtype))
            H = m.heads
            uk = _pad(put(w[p + "mix.uk"]).view(H, m.dim, m.kv_rank), H, dp, R)
            uv = _pad(put(w[p + "mix.uv"]).view(H, m.vdim, m.kv_rank), H, dv, R)
            ukv = torch.cat([uk.reshape(H * dp, R), uv.reshape(H * dv, R)])
            q = _pad(put(w[p + "mix.q"]).view(H, m.dim, self.D), H, dp, Dp).reshape(H * dp, Dp)
            o = _pad(put(w[p + "mix.o"]).view(self.D, H, m.vdim), Dp, H, dv).reshape(Dp, H * dv)
            lw: dict[str, Any] = dict(
                H=H, dp=dp, dv=dv, R=R, rank=m.kv_rank, scale=m.scale, flash=fits,
                wqc=dw(torch.cat([q, lin(w[p + "mix.dkv"], R, Dp)])), cnorm=vec(w[p + "mix.dkv.norm"], R),
                wukv=ukv, uk=ukv[: H * dp].view(H, dp, R), uv=ukv[H * dp:].view(H, dv, R), wo=dw(o),
                # the norm's weight and the layer scale multiply the same element: one vector (exact in fp32)
                g1=vec(w[p + "norm1"].float() * w[p + "ls1"].float(), Dp), mlp=layer.mlp)
            f = layer.mlp
            if f is not None:
                lw["g2"] = vec(w[p + "norm2"].float() * w[p + "ls2"].float(), Dp)
            if isinstance(f, DenseMLP):
                fp = _up(f.ff, 8)
                lw.update(up=dw(lin(w[p + "mlp.up"], fp, Dp)), down=dw(lin(w[p + "mlp.down"], Dp, fp)))
            elif isinstance(f, MoEMLP):
                fp = _up(f.ff, 8)
                stack = lambda what, n, k: torch.stack([lin(w[p + f"mlp.e{e}.{what}"], n, k) for e in range(f.experts)])
                # the shared expert's gate is one more row of the router's product
                router = [w[p + "mlp.router"]] + ([w[p + "mlp.shared.sg"]] if f.shared_ff else [])
                lw.update(eup=stack("up", fp, Dp), edown=stack("down", Dp, fp),
                          router=lin(torch.cat([t.to(self.device) for t in router]), f.experts + len(router) - 1, Dp))
                if f.shared_ff:
                    sp = _up(f.shared_ff, 8)
                    lw.update(sup=dw(lin(w[p + "mlp.shared.up"], sp, Dp)), sdown=dw(lin(w[p + "mlp.shared.down"], Dp, sp)))
            self.layers.append(lw)
        self.final = vec(w["final.norm"], Dp)
        self.head = lin(w["head"], cfg.vocab_size, Dp)
        self.cache: Any = None
        self.layer_trace: Optional[list] = None      # when a list: the residual stream after every layer is appended

    def first_visible(self, n: int) -> int:
        return 0

    def make_cache(self, pages: int) -> PagedLatentCache:
        widths = [lw["R"] for lw in self.layers]
        self.cache = PagedLatentCache(widths, [self.ops.latent_block(self.dtype, w) for w in widths], pages, self.device, self.dtype)
        return self.cache

    def _attention(self, h: torch.Tensor, lw: dict, pages: torch.Tensor, b: Batch) -> torch.Tensor:
        """Returns the heads' outputs ``[N, H * dv]``; the new tokens' latents go to their cache slots."""
        ops = self.ops
        H, dp, dv, R = lw["H"], lw["dp"], lw["dv"], lw["R"]
        N = h.shape[0]
        qc = ops.gemm_nt(h, lw["wqc"])
        q = qc[:, : H * dp].view(N, H, dp)
        c = ops.latent_append(qc[:, H * dp:], lw["cnorm"], lw["rank"], self.cfg.norm_eps, pages, b.slots)
        if not b.decode and lw["flash"] and b.max_seqlen > self.short_portion:
            if b.total_context > N:
                c = ops.latent_gather(pages, b.page_table, b.cu_context, b.total_context)
            kv = ops.gemm_nt(c, lw["wukv"])
            k, v = kv[:, : H * dp].view(-1, H, dp), kv[:, H * dp:].view(-1, H, dv)
            return ops.attention_context(q, k, v, b.cu_seqlens, b.cu_context, b.max_seqlen, lw["scale"]).view(N, H * dv)
        qa = ops.head_gemm(q, lw["uk"], transposed=True)
        oc = ops.latent_attention(qa, pages, b.page_table, b.ctx_lens, b.cu_seqlens, b.max_seqlen, b.max_ctx, lw["scale"])
        return ops.head_gemm(oc, lw["uv"]).reshape(N, H * dv)

    def _experts(self, x: torch.Tensor, h: torch.Tensor, lw: dict) -> torch.Tensor:
        ops, f = self.ops, lw["mlp"]
        ids, wts, gate, plan = ops.moe_route(h, lw["router"], f.experts, f.top, f.scale, f.groups, f.keep)
        ye, at = ops.moe_experts(h, ids, lw["eup"], lw["edown"], "gelu", plan)
        ys = None
        if f.shared_ff:
            ys = ops.gemm_nt(ops.activate(ops.gemm_nt(h, lw["sup"]), "gelu"), lw["sdown"])
        return ops.moe_combine_norm_add(x, ye, at, wts, ys, gate, lw["g2"], self.D, self.cfg.norm_eps, h.dtype)

    @torch.no_grad()
    def forward(self, b: Batch) -> torch.Tensor:
        ops, cfg = self.ops, self.cfg
        eps, bg = cfg.norm_eps, cfg.bigram
        x, h = ops.embed_pairs(b.ids, b.prev, self.embed, self.bigram, (bg.buckets, bg.mul_prev, bg.mul_cur) if bg else (0, 0, 0))
        for i, lw in enumerate(self.layers):
            y = ops.gemm_nt(self._attention(h, lw, self.cache.c[i], b), lw["wo"])
            h = ops.norm_add(x, y, lw["g1"], self.D, eps)
            f = lw["mlp"]
            if isinstance(f, DenseMLP):
                y = ops.gemm_nt(ops.activate(ops.gemm_nt(h, lw["up"]), "relu2"), lw["down"])
                h = ops.norm_add(x, y, lw["g2"], self.D, eps)
            elif isinstance(f, MoEMLP):
                h = self._experts(x, h, lw)
            if self.layer_trace is not None:
                self.layer_trace.append(x[:, : self.D].clone().cpu())
        n = ops.norm_rows(x, b.rows, self.final, self.D, eps, h.dtype)
        logits = ops.gemm_nt(n, self.head, out=torch.empty(n.shape[0], cfg.vocab_size, device=n.device, dtype=torch.float32))
        return ops.softcap_(logits, cfg.logit_softcap) if cfg.logit_softcap else logits


class HybridRunner:
    """Pre-norm decoder whose layers mix tokens by grouped attention (optionally inside chunks of the sequence) or by a
    gated delta rule, some of them run several times (``models/lisunex.py``).

    The residual stream is fp32; a sub-layer's output is added by the norm in front of the next one.  Attention layers keep keys
    and values in pages, delta layers a matrix state and the last convolution inputs per sequence; every run of a looped layer has
    its own.  Attention takes one of two forms:

    * decoding and short portions read the paged cache where it lies;
    * in long portions every chunk of a sequence is a packed sequence of its own for the flash kernel, its queries the last of the
      chunk's positions so far; keys of the chunk that an earlier pass left are gathered in front of the new ones.
    """

    continues = True
    needs_prev = False

    def __init__(self, eng: Any) -> None:
        if eng.tp is not None:
            raise ValueError("hybrid models are served on one GPU")
        self.ops, self.device, self.dtype = eng.ops, eng.device, eng.dtype
        self.max_ctx, self.max_states = eng.max_ctx, eng.max_batch
        model: LisunexModel = eng.model
        cfg = self.cfg = model.config
        self.D, self.short_portion = cfg.hidden_size, 16
        Dp = self.Dp = _up(self.D, 8)
        w = model.weights
        f32 = lambda t: t.to(self.device, torch.float32).contiguous()
        put = lambda t: t.to(self.device, self.dtype)
        vec = lambda t: _pad(f32(t), Dp)
        dw = self.ops.decode_weight
        # one product for everything that reads the layer's input: the parts start at multiples of eight rows
        fuse = lambda parts: torch.cat([_pad(put(t), _up(t.shape[0], 8), Dp) for t in parts])
        self.embed = _pad(put(w["embed"]), cfg.vocab_size, Dp)
        self.steps = [vec(t) for t in w["loop.step"]] if cfg.loop else []
        tables: dict[Any, tuple[torch.Tensor, torch.Tensor]] = {}
        self.layers: list[dict[str, Any]] = []
        for i, layer in enumerate(cfg.layers):
            p, m = f"l{i}.", layer.mixer
            x = lambda n: w[p + "mix." + n]
            lw: dict[str, Any] = dict(m=m, norm1=vec(w[p + "norm1"]), delta=isinstance(m, DeltaMixer))
            if isinstance(m, AttentionMixer):
                lw["hd"] = hd = self.ops.flash_heads(self.dtype, m.dim, m.vdim)
                lw.update(kd=hd or _up(m.dim, 8), vd=hd or _up(m.vdim, 8), cols=_up(m.vdim, 8))
                if m.rot not in tables:
                    tables[m.rot] = tuple(t.to(self.device).contiguous() for t in m.rot.table(self.max_ctx))
                lw["win"] = dw(fuse([x("q"), x("k"), x("v"), x("g")]))
                lw["bias"] = torch.cat([_pad(put(b), _up(b.shape[0], 8)) for b in (x("q.b"), x("k.b"), x("v.b"), torch.zeros(m.heads))])
                lw["cs"] = tables[m.rot]
                lw["gate"] = _up(m.heads * m.dim, 8) + _up(m.kv_heads * m.dim, 8) + _up(m.kv_heads * m.vdim, 8)
                o = _pad(put(x("o")).view(self.D, m.heads, m.vdim), Dp, m.heads, lw["cols"])
                lw["wo"] = dw(o.reshape(Dp, m.heads * lw["cols"]))
            else:
                lw["win"] = dw(fuse([x("q"), x("k"), x("v"), x("g"), x("b"), x("a")]))
                lw["conv"] = torch.cat([f32(x(n + ".conv")) for n in "qkv"]).t().contiguous()
                lw.update(a_log=f32(x("A_log")), dt=f32(x("dt_bias")), norm=f32(x("norm")))
                lw["wo"] = dw(_pad(put(x("o")), Dp, _up(m.heads * m.vdim, 8)))
            if layer.mlp is not None:
                fp = _up(layer.mlp.ff, 8)
                lw.update(norm2=vec(w[p + "norm2"]), wgu=dw(fuse([w[p + "mlp.gate"], w[p + "mlp.up"]])),
                          wd=dw(_pad(put(w[p + "mlp.down"]), Dp, fp)))
            self.layers.append(lw)
        self.final = vec(w["final.norm"])
        self.head = _pad(put(w["head"]), cfg.vocab_size, Dp)
        self.runs = cfg.runs()
        self.chunks = {lw["m"].chunk for lw in self.layers if not lw["delta"]}
        self.context_buckets = 0 in self.chunks
        self.cache: Any = None
        self.layer_trace: Optional[list] = None      # when a list: the residual stream after every layer run is appended

    def first_visible(self, n: int) -> int:
        return min((n // c * c if c else 0 for c in self.chunks), default=n)

    def make_cache(self, pages: int) -> HybridCache:
        kv, rec = [], []
        for i, _ in self.runs:
            lw, m = self.layers[i], self.layers[i]["m"]
            kv.append(None if lw["delta"] else (m.kv_heads, lw["kd"], lw["vd"]))
            rec.append((m.heads, m.dim, m.vdim, m.taps) if lw["delta"] else None)
        self.cache = HybridCache(kv, rec, pages, self.max_states, self.device, self.dtype)
        return self.cache

    def _segments(self, b: Batch, chunk: int) -> dict[str, Any]:
        """The chunks (0: whole contexts) that the batch's queries lie in, as packed sequences."""
        cq, ck, seq, first = [0], [0], [], []
        cached = False
        for i, (start, n) in enumerate(b.spans):
            at = start
            while at < start + n:
                lo = at // chunk * chunk if chunk else 0
                end = min(start + n, lo + chunk) if chunk else start + n
                cached |= lo < start
                seq.append(i)
                first.append(lo)
                cq.append(cq[-1] + end - at)
                ck.append(ck[-1] + end - lo)
                at = end
        t = lambda v: torch.tensor(v, dtype=torch.int32).to(self.device)
        return dict(cq=t(cq), ck=t(ck), seq=t(seq), first=t(first), total=ck[-1], cached=cached, max_q=max(y - x for x, y in zip(cq, cq[1:])))

    def _attention(self, h: torch.Tensor, lw: dict, run: int, b: Batch, segments: dict) -> torch.Tensor:
        ops, m, N = self.ops, lw["m"], h.shape[0]
        rows = ops.gemm_nt(h, lw["win"], residual=lw["bias"].expand(N, -1))
        kp, vp = self.cache.k[run], self.cache.v[run]
        packed = lw["hd"] > 0 and not b.decode and b.max_seqlen > self.short_portion
        if packed and m.chunk not in segments:
            segments[m.chunk] = self._segments(b, m.chunk)
        s = segments.get(m.chunk)
        q, k, v = ops.head_rotary_norm(rows, m.heads, m.kv_heads, m.dim, m.vdim, *lw["cs"], b.positions, self.cfg.norm_eps, kp, vp, b.slots,
                                       packed and not s["cached"])
        gate = rows[:, lw["gate"]: lw["gate"] + m.heads]
        if not packed:
            return ops.paged_attention(q, kp, vp, b.page_table, b.ctx_lens, b.cu_seqlens, b.max_ctx, m.scale, m.softcap, m.chunk, gate,
                                       m.vdim, lw["cols"])
        if s["cached"]:
            k, v = ops.kv_gather(kp, vp, b.page_table, s["seq"], s["first"], s["ck"], s["total"])
        # unit-RMS queries and keys: |q . k| <= dim (rounding of the two included)
        bound = 1.02 * m.dim * abs(m.scale)
        return ops.attention_context(q, k, v, s["cq"], s["ck"], s["max_q"], m.scale, m.softcap, gate, lw["cols"], bound).view(N, -1)

    def _delta(self, h: torch.Tensor, lw: dict, run: int, b: Batch) -> torch.Tensor:
        m = lw["m"]
        return self.ops.delta_rule(self.ops.gemm_nt(h, lw["win"]), m.heads, m.kv_heads, m.dim, m.vdim, lw["conv"], lw["a_log"], lw["dt"],
                                   lw["norm"], self.cfg.norm_eps, self.cache.state[run], self.cache.ring[run], b.states, b.cu_seqlens,
                                   b.ctx_lens, b.max_seqlen)

    @torch.no_grad()
    def forward(self, b: Batch) -> torch.Tensor:
        ops, cfg = self.ops, self.cfg
        eps, D = cfg.norm_eps, self.D
        x, _ = ops.embed_pairs(b.ids, None, self.embed, None, (0, 0, 0), cfg.embedding_scale)
        y = None
        segments: dict[int, dict] = {}
        for run, (i, t) in enumerate(self.runs):
            lw = self.layers[i]
            h = ops.add_norm(x, y, None if t is None else self.steps[t], lw["norm1"], D, eps, self.dtype)
            o = self._delta(h, lw, run, b) if lw["delta"] else self._attention(h, lw, run, b, segments)
            y = ops.gemm_nt(o, lw["wo"])
            if "wd" in lw:
                h = ops.add_norm(x, y, None, lw["norm2"], D, eps, self.dtype)
                y = ops.gemm_nt(ops.swiglu_fwd(ops.gemm_nt(h, lw["wgu"])), lw["wd"])
            if self.layer_trace is not None:
                self.layer_trace.append((x + y.float())[:, :D].cpu())
        n = ops.add_norm(x, y, None, self.final, D, eps, self.dtype, rows=b.rows)
        return ops.gemm_nt(n, self.head, out=torch.empty(n.shape[0], cfg.vocab_size, device=n.device, dtype=torch.float32))
