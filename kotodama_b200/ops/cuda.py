"""sm_100a backend: the same op contract as :class:`TorchOps`, carried out by the kernels in
``csrc/`` through ``ctypes`` (raw pointers + the current CUDA stream).

Activations and parameters are bf16, statistics fp32, Newton-Schulz operands fp16.  A GEMM
whose operands break the TMA rules (16-byte aligned base, leading dimension a multiple of 8
elements) raises instead of taking another path.  Kernels that wait (mbarrier pipelines) bound
their waits and report through a device status word, read by :meth:`CudaOps.check_status`.
"""
from __future__ import annotations

import contextlib
import ctypes
import math
from typing import Optional, Sequence

import torch

from . import _build
from .reference import DecodeWeight, Fp8Weight, TorchOps

_VP = ctypes.c_void_p
_I = ctypes.c_int
_LL = ctypes.c_longlong
_F = ctypes.c_float

_FMT = {torch.float16: 0, torch.bfloat16: 1}
_TYPE = {torch.bfloat16: 0, torch.float32: 1}      # activation type of kernels that exist for both
_OUT = {torch.float16: 0, torch.bfloat16: 1, torch.float32: 2}


def _p(t: Optional[torch.Tensor]) -> _VP:
    return _VP(t.data_ptr()) if t is not None else _VP(None)


def _st() -> _VP:
    return _VP(torch.cuda.current_stream().cuda_stream)


class KernelError(RuntimeError):
    pass


class CudaOps(TorchOps):
    name = "sm100"

    def __init__(self, gemm_backend: str = "tcgen05", attention_backend: str = "auto") -> None:
        self.lib = _build.load()
        import os
        self.gemm_backend = os.environ.get("KOTODAMA_GEMM", gemm_backend)   # "cublas" = library baseline
        self.attention_backend = attention_backend
        self.mn_major = os.environ.get("KOTODAMA_MN_MAJOR", "1") == "1"   # MN-major GEMM operands (no transposes)
        self.launches = 0              # launches of kernels from this library
        self._status: dict[int, torch.Tensor] = {}
        self.gemm_max_ctas = 0
        self.split_k_small_m = True
        self._splitk_ws: dict = {}
        self.attention_library_calls = 0   # stays 0: attention runs on the native kernels in both directions
        self.gemm_2cta = os.environ.get("KOTODAMA_GEMM_2CTA", "1") == "1"   # CTA-pair kernel for large products
        # fp8 products: "mx" = hardware block-scaled MMA (power-of-two scales, accumulation stays in tensor
        # memory); "promote" = fp32 scales applied per K block in registers
        self.skinny_cluster = os.environ.get("KOTODAMA_SKINNY", "cluster") != "splitk"   # decode-size GEMMs: cluster split-K through DSMEM
        self._merge_counters: dict = {}
        # split merge of the decode attention: its own (dependent) launch, or inside the decode kernel by the last CTA
        # of a (request, kv head) pair.  Measured on the 3B decode step: 4.18 ms with the launch, 4.37 ms fused (the
        # device-wide fence and the election at the end of 2560 CTAs cost more than 28 short launches), so: launch
        self.decode_merge_fused = os.environ.get("KOTODAMA_DECODE_MERGE", "kernel") == "fused"
        self.pack_decode_weights = os.environ.get("KOTODAMA_PACK_DECODE", "0") == "1"   # serving: tile-major weight copies for decode (measured +3 %, costs a second copy of the weights: off)
        self.fp8_backend = os.environ.get("KOTODAMA_FP8", "mx")
        self.fp8_pow2 = self.fp8_backend == "mx"
        self.fp8_pair = int(os.environ.get("KOTODAMA_FP8_PAIR", "0"))       # mx kernel: 1 = SM-pair tiles, 0 = one CTA per tile (faster, default)
        for name in ("kb_route_bwd_grid", "kb_qknorm_grid_warps", "kb_route_pipe_grid", "kb_route_blocked_ok",
                     "kb_route_blocked_grid"):
            if hasattr(self.lib, name):          # a library of the serving kernels alone does not have the training ones
                getattr(self.lib, name).restype = _I
        for name in ("kb_delta_chunk_tt_bytes", "kb_delta_chunk_scalars"):
            if hasattr(self.lib, name):
                getattr(self.lib, name).restype = _LL

    # ------------------------------------------------------------------ utils
    def _rc(self, rc: int, what: str) -> None:
        self.launches += 1
        if rc != 0:
            raise KernelError(f"{what}: launcher returned {rc}")

    def _call(self, fn: str, *args) -> None:
        self._rc(getattr(self.lib, fn)(*args), fn)

    def status(self, device: torch.device) -> torch.Tensor:
        idx = device.index if device.index is not None else torch.cuda.current_device()
        if idx not in self._status:
            self._status[idx] = torch.zeros(1, dtype=torch.int32, device=device)
        return self._status[idx]

    def check_status(self, device: Optional[torch.device] = None) -> None:
        """Host-side check of the bounded-wait status word (synchronises)."""
        for idx, t in self._status.items():
            v = int(t.item())
            if v != 0:
                t.zero_()
                what = {5: "a kernel refused its arguments", 6: "an index read from data (token id, label or cache slot) "
                        "was out of range; the access was skipped"}.get(v, "a kernel wait timed out")
                raise KernelError(f"device {idx}: {what} (status {v})")
        if self._status:        # the decode kernels keep their own status word (no status argument)
            torch.cuda.synchronize()
            v = int(self.lib.kb_decode_status())
            if v != 0:
                raise KernelError(f"paged decode attention: a bulk copy did not arrive in time (status {v})")

    # ------------------------------------------------------------------ GEMM
    def _gemm(self, a: torch.Tensor, b: torch.Tensor, M: int, N: int, K: int, a_mn: bool, b_mn: bool,
              out: Optional[torch.Tensor] = None, cin: Optional[torch.Tensor] = None, alpha: float = 1.0,
              beta: float = 0.0, out_dtype: Optional[torch.dtype] = None, batch: int = 1,
              sym_upper: bool = False, diag: float = 0.0, b_const: bool = False) -> torch.Tensor:
        """``b_const``: ``b`` is a weight that nothing writes while kernels are in flight (serving), so a
        decode-size product launched as a dependent may fetch it before the kernels ahead have finished.
        ``diag`` is added to the diagonal of the result (fused into the CTA-pair kernel's epilogue when
        there is an addend, a separate in-place add otherwise)."""
        if a.dtype == torch.float32:
            return self._gemm_f32(a, b, M, N, K, a_mn, b_mn, out, cin, alpha, beta, batch)
        out_dtype = out_dtype or (out.dtype if out is not None else a.dtype)
        lead = (batch,) if batch > 1 else ()
        if out is None:
            out = torch.empty(*lead, M, N, device=a.device, dtype=out_dtype)
        if self.gemm_backend == "cublas":
            # library arm for A/B runs: one cuBLAS call with alpha/beta where the dtypes allow it (no
            # fp32 round trip, no extra passes over the result), so that the comparison is fair
            am = a.transpose(-1, -2) if a_mn else a
            bm = b if b_mn else b.transpose(-1, -2)
            same = out.dtype == a.dtype == b.dtype and (cin is None or cin.dtype == out.dtype)
            if same and cin is None and alpha == 1.0:
                torch.matmul(am, bm, out=out)
            elif same and batch == 1:
                torch.addmm(cin if cin is not None else out, am, bm, beta=beta if cin is not None else 0.0, alpha=alpha, out=out)
            elif same:
                torch.baddbmm(cin if cin is not None else out, am, bm, beta=beta if cin is not None else 0.0, alpha=alpha, out=out)
            else:                                  # mixed dtypes (fp32 accumulation targets): library product, then one fused pass
                r = torch.matmul(am, bm)
                if cin is not None:
                    torch.add(cin.to(out.dtype) * beta, r.to(out.dtype), alpha=alpha, out=out)
                else:
                    out.copy_(r if alpha == 1.0 else r * alpha)
            if diag:
                out.diagonal(dim1=-2, dim2=-1).add_(diag)
            return out
        for t in (a, b):
            if t.stride(-1) != 1 or t.stride(-2) % 8 or t.data_ptr() % 16 or t.dtype not in _FMT:
                raise KernelError(f"GEMM operand not TMA-compatible: shape {tuple(t.shape)} stride {t.stride()} {t.dtype}")
        if out.stride(-1) != 1 or (cin is not None and (cin.stride(-1) != 1 or cin.dtype != out.dtype)):
            raise KernelError("GEMM output/addend must be row-major and of one dtype")
        bs = lambda t: t.stride(0) if batch > 1 else 0
        tiles = ((M + 127) // 128) * ((N + 255) // 256)
        kblocks = (K + 63) // 64
        if (batch == 1 and M <= 128 and tiles <= 74 and kblocks >= 8 and out.dtype == torch.bfloat16
                and out.is_contiguous() and (cin is None or cin.stride(-1) == 1) and self.split_k_small_m):
            # skinny (decode-size) products: too few output tiles to fill the GPU.  bf16 K-major operands: the K
            # range is split over the CTAs of a thread-block cluster and the partial tiles are summed through
            # distributed shared memory (one launch); otherwise split-K with fp32 atomics and a finishing kernel
            if (self.skinny_cluster and not a_mn and not b_mn and a.dtype == torch.bfloat16 and b.dtype == torch.bfloat16
                    and not diag):
                rc = self.lib.kb_gemm_skinny(_p(a), _p(b), _p(out), _p(cin), _I(M), _I(N), _I(K), _LL(a.stride(-2)),
                                             _LL(b.stride(-2)), _LL(out.stride(-2)),
                                             _LL(cin.stride(-2) if cin is not None else 0), _F(alpha), _F(beta), _I(0),
                                             _I(0), _I(2 if b_const else 0), _p(self.status(a.device)), _st())
                if rc == 0:
                    self.launches += 1
                    return out
                if rc != 9:                          # 9: the runtime could not place the cluster - use the atomics path
                    self._rc(rc, "kb_gemm_skinny")
                self.skinny_cluster = False
            cin = cin.contiguous() if cin is not None else None
            split = max(2, min(148 // tiles, kblocks // 2, 16))
            # one fp32 workspace per output size, zeroed once: the finishing kernel clears it again
            key = (M * N, a.device.index)
            ws = self._splitk_ws.get(key)
            if ws is None:
                ws = self._splitk_ws[key] = torch.zeros(M * N, device=a.device, dtype=torch.float32)
            rc = self.lib.kb_gemm(_p(a), _p(b), _p(ws), _p(None), _I(M), _I(N), _I(K), _I(1),
                                  _LL(a.stride(-2)), _LL(b.stride(-2)), _LL(N), _LL(0), _LL(0), _LL(0), _LL(0), _LL(0),
                                  _I(int(a_mn)), _I(int(b_mn)), _I(_FMT[a.dtype]), _I(_FMT[b.dtype]), _I(2),
                                  _F(alpha), _F(0.0), _p(self.status(a.device)), _I(self.gemm_max_ctas), _I(split),
                                  _st())
            self._rc(rc, "kb_gemm(split-k)")
            self._rc(self.lib.kb_f32_to_bf16_add(_p(ws), _p(cin), _F(beta), _p(out), _LL(M * N), _I(1), _st()),
                     "kb_f32_to_bf16_add")
            if diag:
                out.diagonal(dim1=-2, dim2=-1).add_(diag)
            return out
        if self.gemm_2cta and M >= 256 and N >= 256:
            # large products: CTA pairs (256x256 tiles, tcgen05 cta_group::2)
            rc = self.lib.kb_gemm_2cta(_p(a), _p(b), _p(out), _p(cin), _I(M), _I(N), _I(K), _I(batch),
                                       _LL(a.stride(-2)), _LL(b.stride(-2)), _LL(out.stride(-2)),
                                       _LL(cin.stride(-2) if cin is not None else 0),
                                       _LL(bs(a)), _LL(bs(b)), _LL(bs(out)), _LL(bs(cin) if cin is not None else 0),
                                       _I(int(a_mn)), _I(int(b_mn)), _I(_FMT[a.dtype]), _I(_FMT[b.dtype]),
                                       _I(_OUT[out.dtype]), _F(alpha), _F(beta), _p(self.status(a.device)),
                                       _I(self.gemm_max_ctas), _I(int(sym_upper)), _F(diag if cin is not None else 0.0), _st())
            self._rc(rc, "kb_gemm_2cta")
            if diag and cin is None:
                out.diagonal(dim1=-2, dim2=-1).add_(diag)
            # sym_upper: only tiles on/above the diagonal are computed; the epilogue writes each of them
            # to its mirrored position as well (16-bit outputs)
            if sym_upper and out.dtype == torch.float32:
                self._rc(self.lib.kb_mirror_upper16(_p(out), _I(M), _LL(out.stride(-2)), _I(batch), _LL(bs(out)),
                                                    _st()), "kb_mirror_upper16")
            return out
        rc = self.lib.kb_gemm(_p(a), _p(b), _p(out), _p(cin), _I(M), _I(N), _I(K), _I(batch),
                              _LL(a.stride(-2)), _LL(b.stride(-2)), _LL(out.stride(-2)),
                              _LL(cin.stride(-2) if cin is not None else 0),
                              _LL(bs(a)), _LL(bs(b)), _LL(bs(out)), _LL(bs(cin) if cin is not None else 0),
                              _I(int(a_mn)), _I(int(b_mn)), _I(_FMT[a.dtype]), _I(_FMT[b.dtype]), _I(_OUT[out.dtype]),
                              _F(alpha), _F(beta), _p(self.status(a.device)), _I(self.gemm_max_ctas), _I(1), _st())
        self._rc(rc, "kb_gemm")
        if diag:
            out.diagonal(dim1=-2, dim2=-1).add_(diag)
        return out

    def _gemm_f32(self, a, b, M, N, K, a_mn, b_mn, out, cin, alpha, beta, batch):
        """The 32-bit mode: plain fp32 products (no reduced-precision matrix mode)."""
        if a_mn or alpha != 1.0 or (cin is not None and beta != 1.0) or b.dtype != torch.float32:
            raise KernelError(f"fp32 products take K-major fp32 operands and alpha = beta = 1, got {a.dtype}, {b.dtype}")
        if out is None:
            out = torch.empty(*((batch,) if batch > 1 else ()), M, N, device=a.device, dtype=torch.float32)
        if a.stride(-1) != 1 or b.stride(-1) != 1 or out.stride(-1) != 1 or out.dtype != torch.float32 or (
                cin is not None and (cin.stride(-1) != 1 or (batch > 1 and cin.stride() != out.stride()))):
            raise KernelError("fp32 products take row-major operands; the addend of a batch is laid out like the output")
        bs = lambda t: t.stride(0) if batch > 1 else 0
        self._call("kb_gemm_f32", _p(a), _p(b), _p(out), _p(cin), _I(M), _I(N), _I(K), _I(batch), _LL(a.stride(-2)),
                   _LL(b.stride(-2)), _LL(out.stride(-2)), _LL(cin.stride(-2) if cin is not None else 0), _LL(bs(a)), _LL(bs(b)), _LL(bs(out)),
                   _I(int(b_mn)), _p(None), _st())
        return out

    # ------------------------------------------------------------------ block-scaled fp8
    def quant_rows(self, x):
        M, K = x.shape
        x = x.contiguous()
        q = torch.empty(M, K, device=x.device, dtype=torch.float8_e4m3fn)
        s = torch.empty(K // 128, M, device=x.device, dtype=torch.float32)
        self._call("kb_quant_rows", _p(x), _LL(K), _p(q), _LL(K), _p(s), _I(M), _I(K), _I(int(self.fp8_pow2)), _st())
        return q, s

    def quant_blocks(self, w, transposed=False):
        N, K = w.shape
        w = w.contiguous()
        dev = w.device
        q = torch.empty(N, K, device=dev, dtype=torch.float8_e4m3fn)
        s = torch.empty(K // 128, N // 128, device=dev, dtype=torch.float32)
        qt = torch.empty(K, N, device=dev, dtype=torch.float8_e4m3fn) if transposed else None
        st = torch.empty(N // 128, K // 128, device=dev, dtype=torch.float32) if transposed else None
        self._call("kb_quant_blocks", _p(w), _LL(K), _p(q), _p(s), _p(qt), _p(st), _I(N), _I(K), _I(int(self.fp8_pow2)), _st())
        return (q, s, qt, st) if transposed else (q, s)

    def quant_cols_t(self, x):
        M, N = x.shape
        x = x.contiguous()
        qt = torch.empty(N, M, device=x.device, dtype=torch.float8_e4m3fn)
        s = torch.empty(M // 128, N, device=x.device, dtype=torch.float32)
        self._call("kb_quant_cols_t", _p(x), _LL(N), _p(qt), _p(s), _I(M), _I(N), _I(int(self.fp8_pow2)), _st())
        return qt, s

    def gemm_fp8(self, qa, sa, qb, sb, b_gran, out=None, accumulate=False, out_dtype=torch.bfloat16, residual=None):
        M, K = qa.shape
        N = qb.shape[0]
        if out is None:
            out = torch.empty(M, N, device=qa.device, dtype=out_dtype)
        cin = residual if residual is not None else (out if accumulate else None)
        otype = {torch.bfloat16: 1, torch.float32: 2}[out.dtype]
        self._call("kb_gemm_mxfp8" if self.fp8_backend == "mx" else "kb_gemm_fp8", _p(qa), _p(qb), _p(sa), _p(sb), _p(out), _p(cin), _I(M), _I(N), _I(K), _LL(K), _LL(K),
                   _LL(out.stride(0)), _I(b_gran), _I(sb.shape[1]), _I(otype), _F(1.0), _F(1.0 if cin is not None else 0.0),
                   _p(self.status(qa.device)), _I(self.fp8_pair if self.fp8_backend == "mx" else 0), _st())
        return out

    @contextlib.contextmanager
    def dependent_launch(self, on: bool = True):
        """Inside the block the decode-path kernels (routing + norm forward, QK-norm + RoPE, cache append, decode
        attention and its merge, SwiGLU, the decode-size product) are launched as programmatic dependents of
        the kernel before them: their launch and prologue - for the product also the first ring-full of weight
        tiles - overlap that kernel's tail.  A CUDA graph captured inside the block keeps the edges."""
        was = self.lib.kb_set_dependent_launch(_I(1 if on else 0))
        try:
            yield
        finally:
            self.lib.kb_set_dependent_launch(_I(was))

    def decode_weight(self, w: torch.Tensor) -> DecodeWeight:
        N, K = w.shape
        if not (self.skinny_cluster and self.pack_decode_weights and w.is_cuda and w.dtype == torch.bfloat16
                and w.is_contiguous() and K % 64 == 0):
            return DecodeWeight(w)
        packed = torch.empty(((N + 127) // 128) * (K // 64) * 8192, device=w.device, dtype=torch.bfloat16)
        self._call("kb_pack_weight_tiles", _p(w), _LL(K), _p(packed), _I(N), _I(K), _st())
        return DecodeWeight(w, packed)

    def gemm_nt(self, a, b, out=None, residual=None, accumulate=False):
        b_const = isinstance(b, DecodeWeight)
        if b_const:
            M, K = a.shape
            N = b.w.shape[0]
            if (b.packed is not None and self.skinny_cluster and M <= 128 and a.dtype == torch.bfloat16
                    and a.stride(-1) == 1 and a.stride(-2) % 8 == 0 and a.data_ptr() % 16 == 0
                    and (N + 255) // 256 <= 74 and K >= 512):
                if out is None:
                    out = torch.empty(M, N, device=a.device, dtype=torch.bfloat16)
                cin = residual if residual is not None else (out if accumulate else None)
                if out.stride(-1) == 1 and (cin is None or (cin.stride(-1) == 1 and cin.dtype == out.dtype)):
                    rc = self.lib.kb_gemm_skinny(_p(a), _p(b.packed), _p(out), _p(cin), _I(M), _I(N), _I(K), _LL(a.stride(-2)),
                                                 _LL(K), _LL(out.stride(-2)), _LL(cin.stride(-2) if cin is not None else 0),
                                                 _F(1.0), _F(1.0), _I(0), _I(0), _I(3), _p(self.status(a.device)), _st())
                    if rc == 0:
                        self.launches += 1
                        return out
                    if rc != 9:
                        self._rc(rc, "kb_gemm_skinny(packed)")
                    self.skinny_cluster = False
            b = b.w
        if isinstance(b, Fp8Weight):
            if self.fp8_ok(a.shape[0], a.shape[1], b.shape[0]) and a.dtype == torch.bfloat16 and not (
                    accumulate and residual is not None):
                qa, sa = self.quant_rows(a)
                return self.gemm_fp8(qa, sa, b.q, b.s, 128, out=out, accumulate=accumulate, residual=residual)
            b = b.w
        cin = residual if residual is not None else (out if accumulate else None)
        return self._gemm(a, b, a.shape[0], b.shape[0], a.shape[1], False, False, out, cin, 1.0, 1.0, b_const=b_const)

    def gemm_nn(self, a, b, out=None):
        if isinstance(b, Fp8Weight):
            if self.fp8_ok(a.shape[0], a.shape[1], b.shape[1]) and a.dtype == torch.bfloat16:
                qa, sa = self.quant_rows(a)
                return self.gemm_fp8(qa, sa, b.qt, b.st, 128, out=out)
            b = b.w
        if self.mn_major:
            return self._gemm(a, b, a.shape[0], b.shape[1], a.shape[1], False, True, out)
        return self._gemm(a, self.transpose(b), a.shape[0], b.shape[1], a.shape[1], False, False, out)

    def gemm_tn(self, a, b, out=None, accumulate=False, fp8=False):
        if fp8 and self.fp8_ok(a.shape[0], a.shape[1], b.shape[1]) and a.dtype == torch.bfloat16:
            qa, sa = self.quant_cols_t(a)
            qb, sb = self.quant_cols_t(b)
            return self.gemm_fp8(qa, sa, qb, sb, 1, out=out, accumulate=accumulate)
        cin = out if accumulate else None
        if self.mn_major:
            return self._gemm(a, b, a.shape[1], b.shape[1], a.shape[0], True, True, out, cin, 1.0, 1.0)
        return self._gemm(self.transpose(a), self.transpose(b), a.shape[1], b.shape[1], a.shape[0], False, False,
                          out, cin, 1.0, 1.0)

    # ------------------------------------------------------------------ routing
    def route_norm_fwd(self, srcs: Sequence[torch.Tensor], q, rn_w, n_w, eps: float):
        S = len(srcs)
        N, D = srcs[0].shape
        dev = srcs[0].device
        xn = torch.empty(N, D, device=dev, dtype=torch.bfloat16)
        routing = q is not None
        alpha = torch.empty(N, S, device=dev, dtype=torch.float32) if routing else None
        r = torch.empty(N, S, device=dev, dtype=torch.float32) if routing else None
        logit = torch.empty(N, S, device=dev, dtype=torch.float32) if routing else None
        rstd = torch.empty(N, device=dev, dtype=torch.float32)
        arr = (_VP * S)(*[s.data_ptr() for s in srcs])
        if self.lib.kb_route_pipe_grid(_I(N), _I(S), _I(D), _I(0)) > 0:
            rc = self.lib.kb_route_pipe_fwd(arr, _I(S), _p(q), _p(rn_w), _p(n_w), _p(xn), _p(alpha), _p(r), _p(logit),
                                            _p(rstd), _I(N), _I(D), _F(eps), _p(self.status(dev)), _st())
            self._rc(rc, "kb_route_pipe_fwd")
        else:       # rows too large for the shared-memory ring: register-resident kernel
            rc = self.lib.kb_route_norm_fwd(arr, _I(S), _p(q), _p(rn_w), _p(n_w), _p(xn), _p(alpha), _p(r), _p(logit),
                                            _p(rstd), _I(N), _I(D), _F(eps), _st())
            self._rc(rc, "kb_route_norm_fwd")
        return xn, (alpha, r, logit, rstd)

    def route_norm_bwd(self, dxn, srcs, q, rn_w, n_w, eps, stats, dsrcs, acc):
        alpha, r, logit, rstd = stats
        S = len(srcs)
        N, D = srcs[0].shape
        dev = dxn.device
        pipe_grid = self.lib.kb_route_pipe_grid(_I(N), _I(S), _I(D), _I(1))
        grid = pipe_grid if pipe_grid > 0 else self.lib.kb_route_bwd_grid(_I(N))
        routing = q is not None
        dnw_part = torch.empty(grid, D, device=dev, dtype=torch.float32)
        dw_part = torch.empty(grid, D, device=dev, dtype=torch.float32) if routing else None
        sa = (_VP * S)(*[s.data_ptr() for s in srcs])
        da = (_VP * S)(*[d.data_ptr() for d in dsrcs])
        mask = sum(1 << i for i, a in enumerate(acc) if a)
        if pipe_grid > 0:
            rc = self.lib.kb_route_pipe_bwd(sa, da, ctypes.c_uint(mask), _I(S), _p(dxn), _p(q), _p(rn_w), _p(n_w),
                                            _p(alpha), _p(r), _p(logit), _p(rstd), _p(dw_part), _p(dnw_part), _I(N),
                                            _I(D), _p(self.status(dev)), _st())
            self._rc(rc, "kb_route_pipe_bwd")
        else:
            rc = self.lib.kb_route_norm_bwd(sa, da, ctypes.c_uint(mask), _I(S), _p(dxn), _p(q), _p(rn_w), _p(n_w),
                                            _p(alpha), _p(r), _p(logit), _p(rstd), _p(dw_part), _p(dnw_part), _I(N),
                                            _I(D), _st())
            self._rc(rc, "kb_route_norm_bwd")
        dn_w = self._colsum(dnw_part)
        if not routing:
            return None, None, dn_w
        dw = self._colsum(dw_part)
        return dw * rn_w.float(), dw * q.float(), dn_w

    # ------------------------------------------------------------------ sampling
    def sample(self, logits, temperature, top_k, top_p, rep_penalty, seeds, counters, seen, slots):
        """Batched device sampler (``csrc/sampler.cu``); per-row parameter sequences go to the device in
        one small copy each."""
        B, V = logits.shape
        dev = logits.device
        f = lambda x: torch.as_tensor(list(x), dtype=torch.float32).to(dev, non_blocking=True)
        i32 = lambda x: torch.as_tensor(list(x), dtype=torch.int32).to(dev, non_blocking=True)
        m = (1 << 63) - 1
        sd = torch.as_tensor([int(x) & m for x in seeds], dtype=torch.int64).to(dev, non_blocking=True)
        out = torch.empty(B, device=dev, dtype=torch.long)
        t, k, p, r, c, sl = f(temperature), i32(top_k), f(top_p), f(rep_penalty), i32(counters), i32(slots)
        if logits.dtype not in (torch.bfloat16, torch.float32) or logits.stride(1) != 1:
            raise KernelError(f"sampler takes bf16/fp32 row-major logits, got {logits.dtype} {logits.stride()}")
        self._call("kb_sample", _p(logits), _I(0 if logits.dtype == torch.bfloat16 else 1), _LL(logits.stride(0)), _I(B),
                   _I(V), _p(t), _p(k), _p(p), _p(r), _p(sd), _p(c), _p(seen), _I(seen.shape[1] if seen is not None else 0),
                   _p(sl), _p(out), _st())
        return out

    # ------------------------------------------------------------------ AttnRes route, blocked form
    def route_blocked_ok(self, S: int, D: int) -> bool:
        return bool(self.lib.kb_route_blocked_ok(_I(S), _I(D)))

    def _fold_w(self, q: torch.Tensor, rn_w: torch.Tensor) -> torch.Tensor:
        w = torch.empty(q.shape, device=q.device, dtype=torch.float32)
        self._call("kb_route_fold_w", _p(q.contiguous()), _p(rn_w.contiguous()), _p(w), _I(q.numel()), _st())
        return w

    @staticmethod
    def _p1_chunk(S: int, D: int) -> int:
        """Queries per phase-1 launch: 8, or 4 where two backward ring stages of 8 would not fit."""
        return 8 if 2 * (S + 8) * (2 * D + 16) <= 200 * 1024 else 4

    def route_p1_fwd(self, srcs, qs, rn_ws, eps):
        S, Q = len(srcs), qs.shape[0]
        N, D = srcs[0].shape
        dev = srcs[0].device
        wf = self._fold_w(qs, rn_ws)
        o = torch.empty(Q, N, D, device=dev, dtype=torch.bfloat16)
        lse = torch.empty(Q, N, device=dev, dtype=torch.float32)
        r = torch.empty(N, S, device=dev, dtype=torch.float32)
        logit = torch.empty(Q, N, S, device=dev, dtype=torch.float32)
        arr = (_VP * S)(*[t.data_ptr() for t in srcs])
        qc = self._p1_chunk(S, D)
        for q0 in range(0, Q, qc):
            n = min(qc, Q - q0)
            self._call("kb_route_p1_fwd", arr, _I(S), _I(n), _p(wf[q0:]), _p(o[q0:]), _p(lse[q0:]), _p(r),
                       _p(logit[q0:]), _I(N), _I(D), _F(eps), _p(self.status(dev)), _st())
        return o, lse, (r, logit, wf)

    def route_p2_fwd(self, o, lse, partial, q, rn_w, n_w, eps):
        N, D = o.shape
        xn = torch.empty(N, D, device=o.device, dtype=torch.bfloat16)
        stats2 = torch.empty(N, 4, device=o.device, dtype=torch.float32)
        w = self._fold_w(q, rn_w) if partial is not None else None
        self._call("kb_route_p2_fwd", _p(o), _p(lse), _p(partial), _p(w), _p(n_w), _p(xn), _p(stats2), _I(N), _I(D),
                   _F(eps), _st())
        return xn, (stats2, w)

    def route_p2_bwd(self, dxn, o, lse, partial, q, rn_w, n_w, eps, stats2, do_out, dlse_out, dpart, dpart_acc):
        stats2, w = stats2
        N, D = o.shape
        dev = o.device
        grid = self.lib.kb_route_blocked_grid(_I(N), _I(2))
        dnw_part = torch.empty(grid, D, device=dev, dtype=torch.float32)
        dw_part = torch.empty(grid, D, device=dev, dtype=torch.float32) if partial is not None else None
        self._call("kb_route_p2_bwd", _p(dxn), _p(o), _p(partial), _p(w), _p(n_w), _p(stats2), _p(do_out), _p(dlse_out),
                   _p(dpart), _I(1 if dpart_acc else 0), _p(dw_part), _p(dnw_part), _I(N), _I(D), _p(self.status(dev)),
                   _st())
        dn_w = self._colsum(dnw_part)
        return (self._colsum(dw_part) if partial is not None else None), dn_w

    def route_p1_bwd(self, srcs, qs, rn_ws, do, dlse, lse, stats, dsrcs, acc):
        r, logit, wf = stats
        S, Q = len(srcs), qs.shape[0]
        N, D = srcs[0].shape
        dev = srcs[0].device
        grid = self.lib.kb_route_blocked_grid(_I(N), _I(1))
        sa = (_VP * S)(*[t.data_ptr() for t in srcs])
        da = (_VP * S)(*[t.data_ptr() for t in dsrcs])
        mask = sum(1 << i for i, a in enumerate(acc) if a)
        dws = torch.empty(Q, D, device=dev, dtype=torch.float32)
        qc = self._p1_chunk(S, D)
        cw = torch.empty(S, N, 8, device=dev, dtype=torch.float32)
        for q0 in range(0, Q, qc):
            n = min(qc, Q - q0)
            self._call("kb_route_p1_bwd", sa, da, ctypes.c_uint(mask), _I(S), _I(n), _p(wf[q0:]), _p(do[q0:]),
                       _p(dlse[q0:]), _p(lse[q0:]), _p(r), _p(logit[q0:]), _p(cw), _I(N), _I(D), _p(self.status(dev)),
                       _st())
            # query gradients: dw_q = sum over tokens and sources of cw * source (streaming pass + column sum)
            part = torch.empty(grid, n * D, device=dev, dtype=torch.float32)
            self._call("kb_route_dw", sa, _I(S), _I(n), _p(cw), _p(part), _I(N), _I(D), _st())
            dws[q0:q0 + n] = self._colsum(part).view(n, D)
            mask = (1 << S) - 1                     # later query chunks add to what the first one wrote
        return dws

    def _colsum(self, part: torch.Tensor) -> torch.Tensor:
        out = torch.empty(part.shape[1], device=part.device, dtype=torch.float32)
        self._rc(self.lib.kb_colsum(_p(part), _p(out), _I(part.shape[0]), _I(part.shape[1]), _st()), "kb_colsum")
        return out

    # ------------------------------------------------------------------ QK-norm + RoPE
    def qknorm_rope_fwd(self, qkv, qw, kw, cos, sin, seq_len, n_q, n_kv, hd, eps, pos_offset=0, positions=None,
                        append=None):
        """``append=(k_pages, v_pages, slots)``: the same launch also writes the rotated keys and the values of
        every token into its cache slot (what ``kv_append`` does as a launch of its own)."""
        N = qkv.shape[0]
        out = torch.empty(N, (n_q + n_kv) * hd, device=qkv.device, dtype=qkv.dtype)
        rstd = torch.empty(N, n_q + n_kv, device=qkv.device, dtype=torch.float32)
        if append is not None:
            k_pages, v_pages, slots = append
            rc = self.lib.kb_qknorm_rope_append(_p(qkv), _p(qw), _p(kw), _p(cos), _p(sin), _p(out), _p(rstd), _I(N),
                                                _I(seq_len), _I(n_q), _I(n_kv), _I(hd), _I(pos_offset), _F(eps),
                                                _p(positions), _p(k_pages), _p(v_pages), _p(slots),
                                                _LL(k_pages.shape[0] * k_pages.shape[-2]), _p(self.status(qkv.device)),
                                                _st())
            self._rc(rc, "kb_qknorm_rope_append")
            return out, rstd
        rc = self.lib.kb_qknorm_rope_fwd(_p(qkv), _p(qw), _p(kw), _p(cos), _p(sin), _p(out), _p(rstd), _I(N),
                                         _I(seq_len), _I(n_q), _I(n_kv), _I(hd), _I(pos_offset), _F(eps), _p(positions),
                                         _st())
        self._rc(rc, "kb_qknorm_rope_fwd")
        return out, rstd

    def qknorm_rope_bwd(self, dqk, qkv, qw, kw, cos, sin, rstd, seq_len, n_q, n_kv, hd, dqkv_out, pos_offset=0):
        N = qkv.shape[0]
        norm = qw is not None
        warps = self.lib.kb_qknorm_grid_warps()
        part = torch.empty(warps, 2 * hd, device=qkv.device, dtype=torch.float32) if norm else None
        rc = self.lib.kb_qknorm_rope_bwd(_p(dqk), _p(qkv), _p(qw), _p(kw), _p(cos), _p(sin), _p(rstd), _p(dqkv_out),
                                         _p(part), _I(N), _I(seq_len), _I(n_q), _I(n_kv), _I(hd), _I(pos_offset), _st())
        self._rc(rc, "kb_qknorm_rope_bwd")
        if not norm:
            return None, None
        dw = self._colsum(part)
        return dw[:hd], dw[hd:]

    # ------------------------------------------------------------------ attention
    def attention_fwd(self, q, k, v, need_grad=True, cu_seqlens=None, max_seqlen=0):
        from .attention import attention_fwd
        return attention_fwd(self, q, k, v, need_grad, cu_seqlens=cu_seqlens, max_seqlen=max_seqlen)

    def attention_bwd(self, do, q, k, v, o, lse, dq_out, dk_out, dv_out):
        from .attention import attention_bwd
        return attention_bwd(self, do, q, k, v, o, lse, dq_out, dk_out, dv_out)

    # ------------------------------------------------------------------ SwiGLU
    def swiglu_fwd(self, gu):
        N, F2 = gu.shape
        act = torch.empty(N, F2 // 2, device=gu.device, dtype=gu.dtype)
        if gu.dtype == torch.float32:
            self._call("kb_swiglu_f32", _p(gu), _p(act), _LL(N), _I(F2 // 2), _st())
            return act
        self._rc(self.lib.kb_swiglu_fwd(_p(gu), _p(act), _LL(N), _I(F2 // 2), _st()), "kb_swiglu_fwd")
        return act

    def swiglu_bwd(self, gu, dact, out=None):
        N, F2 = gu.shape
        out = out if out is not None else torch.empty_like(gu)
        self._rc(self.lib.kb_swiglu_bwd(_p(gu), _p(dact), _p(out), _LL(N), _I(F2 // 2), _st()), "kb_swiglu_bwd")
        return out

    # ------------------------------------------------------------------ loss head
    def linear_ce(self, h, w, labels, z_weight, grad_scale, dw, dw_accumulate, chunk=4096, need_grad=True,
                  count=None):
        N, D = h.shape
        V = w.shape[0]
        dev = h.device
        row_ce = torch.empty(N, device=dev, dtype=torch.float32)
        row_z = torch.empty(N, device=dev, dtype=torch.float32)
        nv = (labels >= 0).sum().clamp(min=1).float() if count is None else count.reshape(()).float()
        inv = (1.0 / nv).reshape(1)
        dh = torch.empty_like(h) if need_grad else None
        first = not dw_accumulate
        logits = torch.empty(min(chunk, N), V, device=dev, dtype=h.dtype)
        for s in range(0, N, chunk):
            e = min(N, s + chunk)
            lg = logits[: e - s]
            self.gemm_nt(h[s:e], w, out=lg)
            rc = self.lib.kb_ce_zloss(_p(lg), _p(labels[s:e]), _p(row_ce[s:e]), _p(row_z[s:e]), _p(inv),
                                      _F(z_weight), _F(grad_scale), _I(e - s), _I(V), _I(int(need_grad)),
                                      _p(self.status(dev)), _st())
            self._rc(rc, "kb_ce_zloss")
            if need_grad:
                self.gemm_nn(lg, w, out=dh[s:e])
                if dw is not None:
                    self.gemm_tn(lg, h[s:e], out=dw, accumulate=not first)
                    first = False
        sums = torch.empty(2, device=dev, dtype=torch.float32)
        self._rc(self.lib.kb_sum_f32(_p(row_ce), _I(N), _p(sums[0:1]), _st()), "kb_sum_f32")
        self._rc(self.lib.kb_sum_f32(_p(row_z), _I(N), _p(sums[1:2]), _st()), "kb_sum_f32")
        return sums[0] * inv[0], sums[1] * (z_weight * inv[0]), dh

    # ------------------------------------------------------------------ embedding
    def embedding_fwd(self, ids, w):
        N, D = ids.numel(), w.shape[1]
        out = torch.empty(N, D, device=w.device, dtype=w.dtype)
        self._rc(self.lib.kb_embedding_fwd(_p(ids), _p(w), _p(out), _I(N), _I(D), _I(w.shape[0]),
                                           _p(self.status(w.device)), _st()), "kb_embedding_fwd")
        return out

    def embedding_bwd(self, dout, ids, dw):
        self._rc(self.lib.kb_embedding_bwd(_p(ids), _p(dout), _p(dw), _I(ids.numel()), _I(dw.shape[1]), _I(dw.shape[0]),
                                           _p(self.status(dw.device)), _st()), "kb_embedding_bwd")

    # ------------------------------------------------------------------ optimizer math
    def sumsq(self, x, out: Optional[torch.Tensor] = None, accumulate: bool = False):
        dt = {torch.bfloat16: 0, torch.float16: 1, torch.float32: 2}[x.dtype]
        partial = torch.empty(1024, device=x.device, dtype=torch.float32)
        res = out if out is not None else torch.empty(1, device=x.device, dtype=torch.float32)
        self._rc(self.lib.kb_sumsq(_p(x), _LL(x.numel()), _I(dt), _p(partial), _p(res), _I(int(accumulate)), _st()),
                 "kb_sumsq")
        self.launches += 1
        return res[0] if out is None else res

    def adamw_step(self, p, g, m, v, step, lr, b1, b2, eps, wd, gscale):
        gs = gscale.reshape(1).float() if isinstance(gscale, torch.Tensor) else None
        if gs is None and gscale != 1.0:
            gs = torch.full((1,), float(gscale), device=p.device)
        self._rc(self.lib.kb_adamw(_p(p), _p(g), _p(m), _p(v), _LL(p.numel()), _p(gs), _F(lr), _F(b1), _F(b2),
                                   _F(eps), _F(wd), _I(step), _st()), "kb_adamw")

    def muon_momentum(self, g, buf, momentum, nesterov, gscale):
        gs = gscale.reshape(1).float() if isinstance(gscale, torch.Tensor) else None
        x = torch.empty(g.shape, device=g.device, dtype=torch.float16)
        partial = torch.empty(1024, device=g.device, dtype=torch.float32)
        sq = torch.empty(1, device=g.device, dtype=torch.float32)
        self._rc(self.lib.kb_muon_momentum(_p(g), _p(buf), _p(x), _LL(g.numel()), _p(gs), _F(momentum),
                                           _I(int(nesterov)), _p(partial), _p(sq), _st()), "kb_muon_momentum")
        self.launches += 1
        return x, sq

    def ns_normalize(self, x, sumsq):
        self._rc(self.lib.kb_ns_normalize(_p(x), _LL(x.numel()), _p(sumsq.reshape(1)), _st()), "kb_ns_normalize")
        return x

    def ns_iteration(self, x, a, b, c):
        """``A = X X^T``, ``B = bA + cA^2``, ``X' = aX + BX``: three tcgen05 GEMMs with the polynomial
        terms fused into their epilogues.  ``A`` and ``A^2`` are symmetric, so only the tiles on and
        above the diagonal are computed and then mirrored."""
        R, C = x.shape[-2], x.shape[-1]
        batch = x.shape[0] if x.ndim == 3 else 1
        sym = self.gemm_2cta and R >= 512 and x.element_size() == 2
        A = self._gemm(x, x, R, R, C, False, False, batch=batch, sym_upper=sym)
        # aX + BX = (B + aI) X: the identity term goes onto B's diagonal in the epilogue that produces B,
        # so the last (largest) product needs no addend
        B = self._gemm(A, A, R, R, R, False, False, cin=A, alpha=c, beta=b, batch=batch, sym_upper=sym, diag=a)
        if self.mn_major:
            return self._gemm(B, x, R, C, R, False, True, batch=batch)
        xt = self.transpose(x) if x.ndim == 2 else x.transpose(-1, -2).contiguous()
        return self._gemm(B, xt, R, C, R, False, False, batch=batch)

    def muon_apply(self, p, orth, lr, wd, scale, transposed):
        R, C = p.shape
        self._rc(self.lib.kb_muon_apply(_p(p), _p(orth), _I(R), _I(C), _F(lr), _F(wd), _F(scale),
                                        _I(int(transposed)), _st()), "kb_muon_apply")

    def transpose(self, x):
        assert x.ndim == 2 and x.is_contiguous() and x.element_size() == 2
        out = torch.empty(x.shape[1], x.shape[0], device=x.device, dtype=x.dtype)
        self._rc(self.lib.kb_transpose16(_p(x), _p(out), _I(x.shape[0]), _I(x.shape[1]), _st()), "kb_transpose16")
        return out

    # ------------------------------------------------------------------ serving
    def kv_append(self, k, v, k_pages, v_pages, slots):
        """Copy rows ``k[n], v[n]`` (``[N, n_kv*hd]`` views) into cache slot ``slots[n]`` (page*16 + offset)."""
        N, row = k.shape
        self._rc(self.lib.kb_kv_append(_p(k), _p(v), _LL(k.stride(0)), _LL(v.stride(0)), _p(k_pages), _p(v_pages),
                                       _p(slots), _I(N), _I(row), _I(k_pages.shape[-1]),
                                       _LL(k_pages.shape[0] * k_pages.shape[-2]), _p(self.status(k.device)), _st()),
                 "kb_kv_append")

    def paged_decode_attention(self, q, k_pages, v_pages, page_table, ctx_lens, max_ctx, n_q, n_kv, hd, split=512):
        """``q[B, n_q*hd]`` (one new token per request) against the paged cache; returns ``[B, n_q*hd]``."""
        B = q.shape[0]
        nsplit = (max_ctx + split - 1) // split
        G = n_q // n_kv
        part_o = torch.empty(B * n_kv * nsplit * G * hd, device=q.device, dtype=torch.float32)
        part_ml = torch.empty(B * n_kv * nsplit * G * 2, device=q.device, dtype=torch.float32)
        out = torch.empty(B, n_q * hd, device=q.device, dtype=q.dtype)
        # election counters of the in-kernel merge: zero once, left at zero by every call
        key = (q.device.index, B * n_kv)
        counters = self._merge_counters.get(key)
        if counters is None:
            counters = self._merge_counters[key] = torch.zeros(B * n_kv, device=q.device, dtype=torch.int32)
        rc = self.lib.kb_paged_decode_merged(_p(q), _LL(q.stride(0)), _p(k_pages), _p(v_pages), _p(page_table),
                                             _I(page_table.shape[1]), _p(ctx_lens), _I(B), _I(n_q), _I(n_kv), _I(hd),
                                             _I(max_ctx), _I(split), _F(1.0 / math.sqrt(hd)), _p(part_o), _p(part_ml),
                                             _p(out), _LL(out.stride(0)), _I(k_pages.shape[0]),
                                             _p(counters if self.decode_merge_fused else None), _st())
        self._rc(rc, "kb_paged_decode")
        self.launches += 1
        return out

    # ------------------------------------------------------------------ latent attention, output norms, experts
    def flash_latent(self, dtype):
        return dtype == torch.bfloat16

    def latent_multiple(self, dtype):
        return 128 if dtype == torch.bfloat16 else 8       # 128-row blocks of the tensor-core kernel

    def latent_block(self, dtype, R):
        return 64 if dtype == torch.bfloat16 else R        # a block of a page is one TMA copy

    def embed_pairs(self, ids, prev, table, bigram, consts, scale=1.0):
        N, D = ids.numel(), table.shape[1]
        x = torch.empty(N, D, device=table.device, dtype=torch.float32)
        h = x if table.dtype == torch.float32 else torch.empty(N, D, device=table.device, dtype=table.dtype)
        self._call("kb_embed_pairs", _p(ids), _p(prev), _p(table), _p(bigram), _LL(consts[0]), _LL(consts[1]), _LL(consts[2]),
                   _F(scale), _p(x), _p(h), _I(N), _I(D), _I(table.shape[0]), _I(_TYPE[table.dtype]), _p(self.status(table.device)), _st())
        return x, h

    def latent_append(self, rows, w, width, eps, pages, slots):
        N, R = rows.shape
        out = torch.empty(N, R, device=rows.device, dtype=rows.dtype)
        self._call("kb_latent_append", _p(rows), _LL(rows.stride(0)), _p(w), _I(width), _F(eps), _p(pages), _I(pages.shape[3]), _p(slots), _p(out),
                   _I(N), _I(R), _LL(pages.shape[0] * pages.shape[2]), _I(_TYPE[rows.dtype]), _p(self.status(rows.device)), _st())
        return out

    def latent_gather(self, pages, page_table, cu_context, total):
        R = pages.shape[1] * pages.shape[3]
        out = torch.empty(total, R, device=pages.device, dtype=pages.dtype)
        self._call("kb_latent_gather", _p(pages), _I(pages.shape[3]), _p(page_table), _I(page_table.shape[1]), _p(cu_context), _I(page_table.shape[0]),
                   _p(out), _I(total), _I(R), _I(pages.shape[0]), _I(_TYPE[pages.dtype]), _p(self.status(pages.device)), _st())
        return out

    def latent_attention(self, q, pages, page_table, ctx_lens, cu_seqlens, max_q, max_ctx, scale):
        """bf16: the tensor-core kernel (``csrc/latent_attn_sm100.cu``); the 32-bit mode, and latents too large for its
        ring, take the plain kernel (``csrc/latent_attn.cu``)."""
        N, H, R = q.shape
        B = page_table.shape[0]
        dev = q.device
        out = torch.empty(N, H, R, device=dev, dtype=q.dtype)
        if not q.is_contiguous():
            raise KernelError("latent queries must be dense")
        if q.dtype == torch.bfloat16 and pages.shape[3] == 64 and self.lib.kb_latent_ok(_I(B), _I(max_q), _I(H), _I(R)):
            cols = self.lib.kb_latent_cols(_I(max_q), _I(H))
            slots = self.lib.kb_latent_partials(_I(B), _I(max_q), _I(H))
            part_o = torch.empty(slots * cols * R, device=dev, dtype=torch.float32)
            part_ml = torch.empty(slots * cols * 2, device=dev, dtype=torch.float32)
            unit_off = torch.empty(2 * 2048 + 3, device=dev, dtype=torch.int32)
            self._call("kb_latent_attn", _p(q), _p(pages), _p(page_table), _I(page_table.shape[1]), _I(pages.shape[0]), _p(ctx_lens),
                       _p(cu_seqlens), _I(B), _I(max_q), _I(N), _I(H), _I(R), _F(scale), _p(part_o), _p(part_ml), _p(unit_off),
                       _p(out), _p(self.status(dev)), _st())
            self.launches += 1
            return out
        self._call("kb_latent_attn_plain", _p(q), _p(pages), _I(pages.shape[3]), _p(page_table), _I(page_table.shape[1]), _I(pages.shape[0]), _p(ctx_lens),
                   _p(cu_seqlens), _I(B), _p(out), _I(N), _I(H), _I(R), _F(scale), _I(_TYPE[q.dtype]), _p(self.status(dev)), _st())
        return out

    def attention_context(self, q, k, v, cu_seqlens, cu_context, max_q, scale, softcap=0.0, gate=None, cols=0, bound=0.0):
        Nq, H, hd = q.shape
        Nk, KV = k.shape[0], k.shape[1]
        if q.dtype != torch.bfloat16 or hd not in (64, 128) or v.shape[2] != hd:
            raise KernelError(f"flash attention takes bf16 heads of 64 or 128, got {q.dtype} {tuple(q.shape)} {tuple(v.shape)}")
        for t in (q, k, v):
            if t.stride(2) != 1 or t.stride(1) != hd:
                raise KernelError("attention operands are token-major rows with the heads side by side")
        if gate is not None and gate.stride(1) != 1:
            raise KernelError("attention gates are rows of one number per head")
        cols = cols or hd
        out = torch.empty(Nq, H, cols, device=q.device, dtype=q.dtype)
        self._call("kb_flash_fwd_context", _p(q), _LL(q.stride(0)), _I(H * hd), _p(k), _LL(k.stride(0)), _I(KV * hd), _p(v),
                   _LL(v.stride(0)), _I(KV * hd), _p(out), _LL(H * cols), _p(cu_seqlens), _LL(Nq), _p(cu_context), _LL(Nk),
                   _I(cu_seqlens.numel() - 1), _I(max_q), _I(H), _I(KV), _I(hd), _F(scale), _F(softcap), _F(bound), _p(gate),
                   _LL(gate.stride(0) if gate is not None else 0), _I(cols), _p(self.status(q.device)), _st())
        return out

    def head_gemm(self, a, w, transposed=False):
        N, H, K = a.shape
        M = w.shape[2] if transposed else w.shape[1]
        out = torch.empty(N, H, M, device=a.device, dtype=a.dtype)
        if H == 1:
            self._gemm(a[:, 0], w[0], N, M, K, False, transposed, out=out[:, 0])
        else:
            self._gemm(a.transpose(0, 1), w, N, M, K, False, transposed, out=out.transpose(0, 1), batch=H)
        return out

    def activate(self, u, kind):
        out = torch.empty_like(u)
        self._call("kb_activate", _p(u), _p(out), _LL(u.numel()), _I({"gelu": 1, "relu2": 2}[kind]), _I(_TYPE[u.dtype]), _st())
        return out

    def _norm_add(self, x, y, ys, g, width, eps, at, wts, gate, dtype):
        N, D = x.shape
        h = x if dtype == torch.float32 else torch.empty(N, D, device=x.device, dtype=dtype)
        self._call("kb_norm_add", _p(x), _p(y), _p(ys), _p(g), _p(h), _I(N), _I(D), _I(width), _F(eps), _p(at), _p(wts), _p(gate),
                   _I(at.shape[1] if at is not None else 0), _LL(y.shape[0]), _I(_TYPE[y.dtype]), _p(self.status(x.device)), _st())
        return h

    def norm_add(self, x, y, g, width, eps):
        return self._norm_add(x, y, None, g, width, eps, None, None, None, y.dtype)

    def moe_combine_norm_add(self, x, ye, at, wts, ys, gate, g, width, eps, dtype):
        return self._norm_add(x, ye, ys, g, width, eps, at, wts, gate, dtype)

    def norm_rows(self, x, rows, w, width, eps, dtype):
        out = torch.empty(rows.numel(), x.shape[1], device=x.device, dtype=dtype)
        self._call("kb_norm_rows", _p(x), _p(rows), _p(w), _p(out), _I(rows.numel()), _I(x.shape[0]), _I(x.shape[1]), _I(width),
                   _F(eps), _I(_TYPE[dtype]), _p(self.status(x.device)), _st())
        return out

    moe_few = 256           # tokens up to which the router is dot products and the grouping is found from the choices alone

    def moe_route(self, h, router, experts, top, scale, groups, keep):
        """Returns ``(ids, weights, gate, plan)``; ``plan`` (counts per expert, ranks) is for :meth:`moe_experts`."""
        N, D = h.shape
        E = router.shape[0]
        dev = h.device
        gated = E > experts
        ids = torch.empty(N, top, device=dev, dtype=torch.int32)
        wts = torch.empty(N, top, device=dev, dtype=torch.float32)
        gate = torch.empty(N, device=dev, dtype=torch.float32) if gated else None
        counts = rank = None
        if N <= self.moe_few and 8 * D * h.element_size() <= 200 * 1024:
            ld = E
            logits = torch.empty(N, E, device=dev, dtype=torch.float32)
            self._call("kb_router_dot", _p(h), _p(router), _p(logits), _I(N), _I(E), _I(D), _I(_TYPE[h.dtype]), _st())
        else:
            ld = (E + 3) // 4 * 4            # rows the epilogue can store four numbers at a time
            # one zeroed buffer: the logits (the product adds the parts of its K range up in it) and the experts' counters
            buf = torch.zeros(N * ld + experts * 32, device=dev, dtype=torch.float32)
            logits, counts = buf[: N * ld].view(N, ld), buf[N * ld:].view(torch.int32)
            if h.dtype == torch.float32:
                self._gemm(h, router, N, E, D, False, False, out=logits[:, :E])
            else:
                # a product this narrow has one tile per 128 tokens: K is cut so that all SMs stream rows
                split = max(1, min(4, 148 // ((N + 127) // 128), (D + 63) // 64 // 4))
                self._call("kb_gemm", _p(h), _p(router), _p(logits), _p(None), _I(N), _I(E), _I(D), _I(1), _LL(h.stride(0)),
                           _LL(router.stride(0)), _LL(ld), _LL(0), _LL(0), _LL(0), _LL(0), _LL(0), _I(0), _I(0), _I(1), _I(1), _I(2),
                           _F(1.0), _F(0.0), _p(self.status(dev)), _I(0), _I(split), _st())
            rank = torch.empty(N, top, device=dev, dtype=torch.int32)
        self._call("kb_moe_select", _p(logits), _I(ld), _I(N), _I(experts), _I(top), _F(scale), _I(groups), _I(keep), _I(int(gated)),
                   _p(ids), _p(wts), _p(gate), _p(counts), _p(rank), _st())
        return ids, wts, gate, None if counts is None else (counts, rank)

    def moe_experts(self, h, ids, up, down, kind, plan=None):
        rows, offsets, at = self._moe_group(h, ids, up.shape[0], plan)
        return self._grouped(self._grouped(rows, up, offsets, kind), down, offsets, None), at

    def _moe_group(self, h, ids, E, plan):
        N, top = ids.shape
        D = h.shape[1]
        dev = h.device
        counts, at = plan if plan is not None else (None, torch.empty(N, top, device=dev, dtype=torch.int32))
        offsets = torch.empty(E + 1, device=dev, dtype=torch.int32)
        rows = torch.empty(N * top, D, device=dev, dtype=h.dtype)
        self._call("kb_moe_group", _p(h), _p(ids), _p(counts), _I(N), _I(top), _I(E), _I(D * h.element_size()), _p(at), _p(offsets),
                   _p(rows), _p(self.status(dev)), _st())
        return rows, offsets, at

    def _grouped(self, rows, w, offsets, kind):
        A, K = rows.shape
        E, M, _ = w.shape
        out = torch.empty(A, M, device=rows.device, dtype=rows.dtype)
        if rows.dtype == torch.float32:
            self._call("kb_gemm_f32", _p(rows), _p(w), _p(out), _p(None), _I(A), _I(M), _I(K), _I(E), _LL(K), _LL(K), _LL(M), _LL(0),
                       _LL(0), _LL(M * K), _LL(0), _I(0), _p(offsets), _st())
            return self.activate(out, kind) if kind else out
        self._call("kb_gemm_grouped", _p(rows), _p(w), _p(out), _p(offsets), _I(A), _I(E), _I(M), _I(K), _LL(M),
                   _I({None: 0, "gelu": 1, "relu2": 2}[kind]), _I(int(A <= 24 * E)), _p(self.status(rows.device)), _st())
        return out

    # ------------------------------------------------------------------ pre-norm decoders with grouped attention and delta rule
    def add_norm(self, x, y, step, w, width, eps, dtype, rows=None):
        n = x.shape[0] if rows is None else rows.numel()
        h = torch.empty(n, x.shape[1], device=x.device, dtype=dtype)
        self._call("kb_add_norm", _p(x), _p(y), _p(step), _p(rows), _p(w), _p(h), _I(n), _I(x.shape[0]), _I(x.shape[1]), _I(width), _F(eps),
                   _I(_TYPE[dtype]), _p(self.status(x.device)), _st())
        return h

    def flash_heads(self, dtype, dim, vdim):
        return super().flash_heads(dtype, dim, vdim) if dtype == torch.bfloat16 else 0

    def head_rotary_norm(self, rows, H, G, dim, vdim, cos, sin, positions, eps, k_pages, v_pages, slots, keep):
        N = rows.shape[0]
        kd, vd = k_pages.shape[3], v_pages.shape[3]
        up8 = lambda n: (n + 7) // 8 * 8
        col_k = up8(H * dim)
        q = torch.empty(N, H, kd, device=rows.device, dtype=rows.dtype)
        k = torch.empty(N, G, kd, device=rows.device, dtype=rows.dtype) if keep else None
        v = torch.empty(N, G, vd, device=rows.device, dtype=rows.dtype) if keep else None
        self._call("kb_head_rotary", _p(rows), _LL(rows.stride(0)), _I(H), _I(G), _I(dim), _I(vdim), _I(kd), _I(vd), _I(cos.shape[1]), _I(col_k),
                   _I(col_k + up8(G * dim)), _p(cos), _p(sin), _I(cos.shape[0]), _p(positions), _F(eps), _p(q), _p(k), _p(v), _p(k_pages),
                   _p(v_pages), _p(slots), _LL(k_pages.shape[0] * k_pages.shape[2]), _I(N), _I(_TYPE[rows.dtype]), _p(self.status(rows.device)),
                   _st())
        return q, k, v

    def kv_gather(self, k_pages, v_pages, page_table, seg_seq, seg_first, cu, total):
        G, kd, vd = k_pages.shape[1], k_pages.shape[3], v_pages.shape[3]
        k = torch.empty(total, G, kd, device=k_pages.device, dtype=k_pages.dtype)
        v = torch.empty(total, G, vd, device=k_pages.device, dtype=k_pages.dtype)
        self._call("kb_kv_gather", _p(k_pages), _p(v_pages), _I(G), _I(kd), _I(vd), _p(page_table), _I(page_table.shape[0]), _I(page_table.shape[1]),
                   _I(k_pages.shape[0]), _p(seg_seq), _p(seg_first), _p(cu), _I(seg_seq.numel()), _p(k), _p(v), _I(total),
                   _I(_TYPE[k_pages.dtype]), _p(self.status(k_pages.device)), _st())
        return k, v

    def paged_attention(self, q, k_pages, v_pages, page_table, ctx_lens, cu_seqlens, max_ctx, scale, softcap, chunk, gate, vdim, cols):
        N, H, kd = q.shape
        B = page_table.shape[0]
        if ctx_lens.numel() != B or (cu_seqlens.numel() - 1 if cu_seqlens is not None else N) != B:
            raise KernelError(f"paged attention: {B} page lists, {ctx_lens.numel()} lengths, {N} rows, boundaries "
                              f"{None if cu_seqlens is None else tuple(cu_seqlens.shape)}")
        out = torch.empty(N, H * cols, device=q.device, dtype=q.dtype)
        G, size = k_pages.shape[1], k_pages.shape[3]
        if q.dtype == torch.bfloat16 and cu_seqlens is None and size in (64, 128) and v_pages.shape[3] == size:
            # decoding: the tensor-core kernel over splits of the visible keys, short enough to fill the GPU
            visible = min(max_ctx, chunk + 15) if chunk else max_ctx
            split = 512
            while split > 64 and B * G * ((visible + split - 1) // split) < 296:
                split //= 2
            nsplit = (visible + split - 1) // split
            part_o = torch.empty(B * H * nsplit * size, device=q.device, dtype=torch.float32)
            part_ml = torch.empty(B * H * nsplit * 2, device=q.device, dtype=torch.float32)
            self._call("kb_paged_decode_ext", _p(q), _p(k_pages), _p(v_pages), _p(page_table), _I(page_table.shape[1]), _p(ctx_lens), _I(B), _I(H),
                       _I(G), _I(size), _I(visible), _I(split), _F(scale), _F(softcap), _I(chunk), _p(gate),
                       _LL(gate.stride(0) if gate is not None else 0), _p(part_o), _p(part_ml), _p(out), _I(cols), _I(k_pages.shape[0]), _st())
            self.launches += 1
            return out
        self._call("kb_paged_attn_plain", _p(q), _p(k_pages), _p(v_pages), _I(k_pages.shape[1]), _I(kd), _I(v_pages.shape[3]), _p(page_table),
                   _I(page_table.shape[1]), _I(k_pages.shape[0]), _p(ctx_lens), _p(cu_seqlens), _I(page_table.shape[0]), _p(gate),
                   _LL(gate.stride(0) if gate is not None else 0), _p(out), _I(N), _I(H), _I(vdim), _I(cols), _F(scale), _F(softcap), _I(chunk),
                   _I(_TYPE[q.dtype]), _p(self.status(q.device)), _st())
        return out

    delta_short = 16        # most tokens of a sequence in one pass for which the recurrence is walked token by token

    def delta_rule(self, rows, H, G, d, dv, conv, a_log, dt_bias, norm, eps, state, ring, slots, cu_seqlens, ctx_lens, max_q):
        N = rows.shape[0]
        up8 = lambda n: (n + 7) // 8 * 8
        cols = [0]
        for n in (G * d, G * d, H * dv, H * dv, H):
            cols.append(cols[-1] + up8(n))
        width, taps, B, dev = up8(H * dv), conv.shape[0], slots.numel(), rows.device
        if ctx_lens.numel() != B or (cu_seqlens.numel() - 1 if cu_seqlens is not None else N) != B:
            raise KernelError(f"delta rule: {B} state slots, {ctx_lens.numel()} lengths, {N} rows, boundaries "
                              f"{None if cu_seqlens is None else tuple(cu_seqlens.shape)}")
        out = (torch.empty if width == H * dv else torch.zeros)(N, width, device=dev, dtype=rows.dtype)
        if (rows.dtype == torch.bfloat16 and cu_seqlens is not None and max_q > self.delta_short
                and self.lib.kb_delta_chunk_ok(_I(H), _I(G), _I(d), _I(dv), _I(taps))):
            D, dvt = 64 if d <= 64 else 128, (dv + 63) // 64 * 64
            buf = lambda n, exact: (torch.empty if exact else torch.zeros)(N, n, device=dev, dtype=rows.dtype)
            q, k, v, o = buf(G * D, d == D), buf(G * D, d == D), buf(H * dvt, dv == dvt), buf(H * dvt, True)
            tt = torch.empty(self.lib.kb_delta_chunk_tt_bytes(_I(N), _I(B), _I(H)), device=dev, dtype=torch.uint8)
            scal = torch.empty(self.lib.kb_delta_chunk_scalars(_I(N), _I(B), _I(H)), device=dev, dtype=torch.float32)
            self._call("kb_delta_chunks", _p(rows), _LL(rows.stride(0)), *map(_I, cols), _p(conv), _p(a_log), _p(dt_bias), _p(norm), _I(taps),
                       _I(N), _I(B), _I(H), _I(G), _I(d), _I(dv), _I(D), _I(dvt), _I(state.shape[3]), _F(eps), _p(state), _p(ring),
                       _I(ring.shape[2]), _I(state.shape[0]), _p(slots), _p(cu_seqlens), _p(ctx_lens), _p(q), _p(k), _p(v), _p(o), _p(tt),
                       _p(scal), _p(out), _LL(width), _p(self.status(dev)), _st())
            self.launches += 4 - (taps == 1)
            return out
        self._call("kb_delta_step", _p(rows), _LL(rows.stride(0)), *map(_I, cols), _p(conv), _p(a_log), _p(dt_bias), _p(norm),
                   _I(taps), _I(H), _I(G), _I(d), _I(dv), _I(state.shape[3]), _F(eps), _p(state), _p(ring), _I(ring.shape[2]),
                   _I(state.shape[0]), _p(slots), _p(cu_seqlens), _p(ctx_lens), _I(slots.numel()), _p(out), _LL(width), _I(_TYPE[rows.dtype]),
                   _p(self.status(rows.device)), _st())
        return out

    def softcap_(self, logits, cap):
        self._call("kb_softcap", _p(logits), _LL(logits.numel()), _F(cap), _st())
        return logits

    def argmax(self, logits):
        out = torch.empty(logits.shape[0], device=logits.device, dtype=torch.long)
        self._rc(self.lib.kb_argmax(_p(logits), _LL(logits.stride(0)), _I(logits.shape[0]), _I(logits.shape[1]),
                                    _p(out), _I(_TYPE[logits.dtype]), _st()), "kb_argmax")
        return out
