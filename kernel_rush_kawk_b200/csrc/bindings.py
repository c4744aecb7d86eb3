"""Python bindings of the CUDA kernels (ctypes over the compiled libraries).

``Kernels`` is the one object through which the engine computes. Every method
launches this package's own kernels on torch's current CUDA stream; the only
library routine on the path is the dense matrix product of many rows in
bfloat16 (cuBLASLt, called by csrc/lt_gemm.cu with the algorithm picked by
measurement; ``torch.matmul`` for layouts that it does not take), which is
where the reference calls the library too (engine/model.py:295,299,301,303 of
willzeng274/kernel-rush-kawk).
There is no fallback: without a CUDA device and the compiled libraries,
construction raises.
"""

from __future__ import annotations

import ctypes
import os
from ctypes import c_float, c_int, c_longlong, c_uint, c_void_p

import torch

from .build import build_library

F32, BF16 = 0, 1
_P = c_void_p


def _code(dtype: torch.dtype) -> int:
    if dtype == torch.float32:
        return F32
    if dtype == torch.bfloat16:
        return BF16
    raise TypeError(f"kernels take float32 or bfloat16 tensors, got {dtype}")


class KernelError(RuntimeError):
    pass


_SIGNATURES = {
    "krk_rmsnorm": [_P, _P, _P, _P, _P, c_int, c_int, c_int, c_float, c_int, _P],
    "krk_gather_rows": [_P, _P, _P, c_int, c_int, c_int, _P, c_int, _P],
    "krk_swiglu": [_P, _P, c_int, c_int, c_int, _P],
    "krk_qk_norm_rope_write": [_P, _P, _P, c_int, _P, _P, _P, _P, _P, _P, c_int, _P, _P, c_int, c_int, c_int, c_int,
                               c_int, c_float, c_int, _P, c_int, _P],
    "krk_gemm_nt": [_P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, _P],
    "krk_select_tokens": [_P, _P, c_int, c_int, c_float, c_uint, _P, c_uint, _P, _P, _P, _P, _P],
    "krk_gemm_tcgen05": [_P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, _P, _P],
    "krk_selftest_wait_runs_out": [_P, c_int, _P],
    "krk_skinny_linear": [_P, _P, _P, _P, _P, _P, c_int, _P, c_int, c_int, c_int, c_float, c_int, c_int, _P],
    "krk_lt_gemm_bf16": [_P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, c_int, _P, _P],
    "krk_lt_gemm_report": [_P, _P],
}
_MIX_SIGNATURES = {
    "krk_embed_scaled": [_P, _P, _P, c_int, c_int, c_int, c_float, _P, c_int, _P, c_int, _P],
    "krk_post_norm": [_P, _P, _P, _P, _P, c_float, c_int, c_int, c_float, c_int, _P],
    "krk_tanh_cap": [_P, c_longlong, c_float, _P],
    "krk_rmsnorm_wide": [_P, _P, _P, _P, _P, c_float, c_int, c_int, c_float, _P, c_float, _P, _P, c_int, _P],
    "krk_tanh_norm": [_P, _P, _P, _P, _P, c_float, _P, _P, c_int, c_int, c_int, _P],
    "krk_gated_act": [_P, _P, c_int, c_int, c_int, c_int, c_int, c_int, _P, c_float, c_float],
    "krk_hyper_rmsnorm": [_P, _P, _P, _P, _P, _P, _P, c_float, c_int, c_int, c_int, c_float, c_int, _P],
    "krk_bias_row_norm": [_P, c_int, c_int, c_int, c_int, c_int, _P, _P, c_float, c_int, c_int, _P],
    "krk_rotate_norm_write": [_P, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, _P, c_int, c_int, c_float, _P, _P,
                              _P, _P, c_int, _P, _P, c_int, c_int, _P, c_int, c_float, c_int, _P],
    "krk_sink_attention": [_P, c_int, c_int, c_float, _P, c_int, c_int, c_int, c_int, c_int, c_int, _P, _P, _P, _P, _P,
                           c_int, _P, _P, c_int, c_int, c_float, c_int, c_int, c_int, _P, c_int, c_int, c_int, _P, c_float,
                           c_int, _P],
    "krk_sink_attention_single": [_P, c_int, c_int, c_float, _P, c_int, c_int, c_int, c_int, c_int, c_int, _P, _P, _P, _P,
                                  c_int, _P, _P, c_int, c_int, c_float, c_int, c_int, _P, c_int, c_int, c_int, _P, c_int, c_int, c_float,
                                  c_int, c_int, _P, c_int, c_int, c_int, _P, c_float, c_int, _P],
    "krk_latent_norm_write": [_P, c_int, c_int, c_int, _P, c_float, _P, _P, _P, _P, c_int, c_int, _P, c_int, _P, c_int, _P],
    "krk_head_linear": [_P, c_int, c_int, c_int, c_float, _P, c_int, c_int, _P, c_int, c_int, c_int, c_int, c_int, _P, c_float,
                        _P, _P, c_int, c_int, _P],
    "krk_latent_rows": [_P, _P, c_int, c_int, c_int, _P, c_int, c_int, _P, c_int, _P, c_float, c_float, _P, _P, _P, _P, c_int,
                        _P, c_int, c_int, _P],
    "krk_latent_decode": [_P, _P, _P, c_int, c_int, c_int, c_int, _P, _P, _P, c_int, _P, c_float, c_int, c_int, _P],
    "krk_latent_gather": [_P, _P, c_int, c_int, c_int, _P, _P, _P, _P, _P, c_int, c_int, _P],
    "krk_embed_bigram": [_P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_longlong, c_longlong, _P, _P, _P, _P, _P, c_int, _P],
    "krk_bias_norm_rotate_write": [_P, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, _P, _P, c_float, c_int, c_float,
                                   c_int, _P, c_int, c_int, _P, _P, _P, _P, c_int, _P, _P, c_int, c_int, c_int, _P],
    "krk_mixed_attention": [_P, c_int, c_int, c_float, _P, c_int, c_int, c_int, c_int, c_int, c_int, _P, _P, _P, _P, _P, _P,
                            c_int, _P, _P, c_int, c_float, c_int, _P, c_int, c_int, c_int, c_int, _P],
    "krk_mixed_attention_single": [_P, c_int, c_int, c_float, _P, c_int, c_int, c_int, c_int, c_int, c_int, _P, _P, _P, _P,
                                   _P, c_int, _P, _P, c_int, c_float, c_int, c_int, _P, _P, c_int, c_int, c_int, c_int, _P],
    "krk_mixed_attention_merge": [_P, c_int, c_int, c_float, _P, c_int, c_int, c_int, c_int, _P, c_int, c_int, c_int, c_int, _P],
    "krk_norm_sum": [_P, _P, _P, _P, _P, c_int, _P, c_int, c_int, c_float, c_float, c_int, _P],
    "krk_act_rows": [_P, _P, c_int, c_int, c_int, c_int, c_float, c_float, c_int, _P],
}
_MOE_SIGNATURES = {
    "krk_moe_route": [_P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, _P, c_int],
    "krk_moe_route_groups": [_P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, c_float, _P],
    "krk_moe_route_softmax_groups": [_P, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, c_int, _P],
    "krk_moe_gate_up_pairs": [_P, _P, c_int, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, _P, c_float, c_float, c_int, _P],
    "krk_moe_down_pairs": [_P, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, _P, c_int, _P, c_int, _P],
    "krk_moe_sort": [_P, _P, _P, c_int, c_int, c_int, _P],
    "krk_moe_gather": [_P, _P, c_int, _P, _P, _P, c_int, c_int, c_int, c_int, _P, _P, c_int, _P],
    "krk_grouped_gemm": [_P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, c_int, _P, c_float, c_float, _P, _P],
    "krk_moe_combine": [_P, _P, _P, _P, _P, _P, _P, c_int, _P, c_int, c_int, c_int, _P, c_int, _P, c_int, _P],
}
_MEMORY_SIGNATURES = {
    "krk_memory_gates": [_P, _P, c_int, _P, c_float, _P, c_int, c_int, c_int, c_int, _P, _P, _P, c_int, _P],
    "krk_memory_decays": [_P, _P, c_int, _P, _P, c_float, c_int, c_int, c_int, c_int, _P],
    "krk_memory_scan": [_P, _P, _P, c_int, _P, c_int, _P, c_int, c_float, _P, _P, _P, _P, c_int, c_int, c_int, c_int, _P, _P, _P,
                        c_int, _P],
    "krk_memory_step": [_P, c_int, c_int, c_float, _P, c_int, _P, c_int, _P, c_int, _P, c_int, c_float, _P, c_int, _P, _P, c_float,
                        c_int, _P, _P, _P, c_float, c_int, c_int, c_int, c_int, c_int, _P, c_int, _P],
    "krk_memory_chunk_tokens": [c_int, c_int, c_int],
    "krk_memory_chunk_decays": [_P, _P, c_int, _P, _P, c_float, c_int, c_int, c_int, c_int, _P, _P, _P],
    "krk_memory_chunks": [_P, _P, _P, c_int, _P, c_int, _P, c_int, c_float, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int,
                          _P, _P, _P, _P],
    "krk_memory_finish": [_P, c_int, c_int, c_float, _P, _P, _P, _P, c_int, _P, c_int, c_int, c_float, c_int, c_int, _P],
}
_LATENT_SIGNATURES = {
    "krk_latent_prefill": [_P, c_int, c_float, _P, c_int, c_int, c_int, _P, _P, c_int, c_int, _P, c_float, c_float, c_int, c_int,
                           _P, _P, _P, _P, _P, c_int, _P],
}
_SCAN_SIGNATURES = {
    "krk_token_shift": [_P, _P, c_int, _P, _P, c_int, c_int, c_int, _P, _P, _P, c_int, _P, c_int],
    "krk_linear_recurrence": [c_int, _P, c_int, _P, c_int, _P, c_int, _P, c_int, _P, c_int, _P, c_int, _P, _P, _P, _P, _P,
                              _P, _P, c_int, c_int, _P, _P, c_int, c_int, c_float, c_float, c_float, c_int, c_int, c_int,
                              c_int, _P, _P, _P, c_int, _P, _P, c_int, _P],
    "krk_causal_conv_silu": [_P, _P, c_int, _P, _P, _P, c_int, c_int, c_int, c_int, _P, _P, _P, _P, c_int, _P],
    "krk_ssd_scan": [_P, _P, c_int, _P, c_int, _P, c_int, _P, c_int, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int,
                     c_int, _P, _P, _P, c_int, _P, _P, c_int, _P],
    "krk_gated_group_norm": [_P, c_int, c_int, c_float, _P, _P, c_int, _P, c_int, c_int, c_int, c_float, c_int, _P],
}
_ACTIVATIONS = {"silu": 0, "gelu_tanh": 1, "sigmoid": 2, "swish_clamped": 3, "xielu": 4, "relu2": 5}
_ATTN_SIGNATURES = {
    "krk_attention_simple": [_P, _P, c_int, c_int, c_int, _P, _P, _P, _P, c_int, _P, _P, c_int, c_float, c_int, c_int, _P],
    "krk_attention_head_dim": [],
    "krk_attention_prefill": [_P, _P, c_int, c_int, c_int, _P, _P, _P, _P, _P, c_int, _P, _P, c_int, c_int, c_float,
                              c_int, _P],
    "krk_sink_window_prefill": [_P, c_int, c_float, _P, c_int, c_int, c_int, _P, _P, _P, _P, _P, _P, c_int, _P, _P, c_int,
                                c_int, c_float, c_int, c_int, c_int, _P, c_int, c_int, _P, c_float, _P],
    "krk_sink_window_decode": [_P, c_int, c_float, _P, c_int, c_int, c_int, _P, _P, _P, _P, c_int, _P, _P, c_int, c_float, c_int,
                               c_int, c_int, _P, c_int, c_int, _P, c_float, c_int, _P],
    "krk_mixed_prefill": [_P, c_int, c_float, _P, c_int, c_int, c_int, _P, _P, _P, _P, _P, _P, _P, c_int, _P, _P, c_int,
                          c_int, c_float, c_int, _P, c_int, c_int, _P, c_int, _P],
    "krk_attention_decode": [_P, _P, c_int, c_int, c_int, _P, _P, _P, c_int, _P, _P, c_int, c_float, c_int, c_int, _P,
                             _P],
    "krk_attention_prefill_tcgen05": [_P, _P, c_int, c_int, c_int, _P, _P, _P, _P, _P, c_int, _P, _P, c_int, c_int, c_int,
                                      c_int, c_float, c_int, _P, _P],
    "krk_attention_decode_fused": [_P, _P, c_int, c_int, c_int, _P, _P, c_int, _P, _P, c_float, _P, _P, _P, c_int, _P,
                                   _P, c_int, c_float, c_int, c_int, c_int, _P, _P],
    "krk_attention_decode_fused_tma": [_P, _P, c_int, c_int, c_int, _P, _P, c_int, _P, _P, c_float, _P, _P, _P, c_int, _P,
                                       _P, c_int, c_int, c_float, c_int, c_int, c_int, _P, _P],
}


def _load(path, signatures) -> ctypes.CDLL:
    lib = ctypes.CDLL(str(path))
    for name, args in signatures.items():
        try:
            fn = getattr(lib, name)
        except AttributeError:
            continue
        fn.argtypes = args
        fn.restype = c_int
    return lib


def _ptr(t) -> int | None:
    return None if t is None else t.data_ptr()


class Kernels:
    """All kernels, for one device. ``head_dims``: the head sizes whose attention
    libraries are needed (compiled at first use)."""

    SKINNY_MAX_ROWS = 16  # rows up to which the fused skinny kernels serve a bfloat16 product
    # Every block of a skinny product redoes the norm of all rows in its prologue. That is
    # cheaper than a separate norm kernel for one or two rows and dearer beyond.
    FUSED_NORM_MAX_ROWS = 2

    def __init__(self, head_dims=(), device="cuda:0"):
        if not torch.cuda.is_available():
            raise KernelError("no CUDA device: this library computes with its CUDA kernels only")
        self.device = torch.device(device)
        self.core = _load(build_library("core"), _SIGNATURES)
        self._mix = self._scan = self._moe = self._memory = None
        self.attn: dict[int, ctypes.CDLL] = {}
        self.latent: dict[tuple, ctypes.CDLL] = {}
        for d in head_dims:
            self._attn_lib(int(d))
        self.error = torch.zeros(1, dtype=torch.int32, device=self.device)
        self.has_skinny = hasattr(self.core, "krk_skinny_linear")
        self._partials: dict = {}
        self._select_scratch = None
        self.use_tcgen05_attention = True
        self.use_tma_decode_attention = True
        # Key-split counts that take the TMA-fed single-token attention. It splits keys over a cluster like the
        # cp.async kernel, bit for bit; measured on the 4B shape it wins with one block or two per item (16 sequences
        # at 8,000 tokens of context: 4.95 against 5.53 ms a step) and loses with more (one sequence at 32,000
        # tokens: 4.08 against 3.14 ms), where a block's own pace, not the bytes in flight, is the bound.
        self.tma_decode_splits = {1, 2}
        self.use_tuned_library_gemm = hasattr(self.core, "krk_lt_gemm_bf16")
        # steps of many tokens: prepare / scan / finish kernels instead of the fused one. Bit-equal to it and, on one
        # prompt, no faster (the scan itself bounds both), so it is off; it needs rows * channels * 28 bytes of scratch
        self.split_recurrence = False
        # single-token steps: rotation, value norm and cache write inside the attention kernel (one launch fewer a
        # layer). Right, and slower (8 sequences of the 1.5k-wide preset: 0.608 against 0.563 ms a step; one sequence
        # 0.510 against 0.497): every block of an item repeats the prologue on its critical path, where the kernel of
        # its own runs under the product before it. Off.
        self.fuse_single_token_attention = os.environ.get("KRK_FUSE_SINGLE_ATTENTION") is not None
        self.launches = 0

    def _attn_lib(self, head_dim: int) -> ctypes.CDLL:
        lib = self.attn.get(head_dim)
        if lib is None:
            if head_dim % 2 or head_dim > 256:
                raise KernelError(f"attention kernels take an even head size up to 256, got {head_dim}")
            lib = self.attn[head_dim] = _load(build_library("attn", head_dim), _ATTN_SIGNATURES)
            assert lib.krk_attention_head_dim() == head_dim
        return lib

    def _latent_lib(self, key_dim: int, value_dim: int) -> ctypes.CDLL:
        """The prompt attention of a pair of head sizes over keys and values made from latent rows, compiled and loaded
        at its first call."""
        lib = self.latent.get((key_dim, value_dim))
        if lib is None:
            lib = self.latent[(key_dim, value_dim)] = _load(build_library("latent", (key_dim, value_dim)), _LATENT_SIGNATURES)
        return lib

    # -- plumbing -------------------------------------------------------------
    def _stream(self):
        return torch.cuda.current_stream(self.device).cuda_stream

    def _ok(self, code: int, what: str) -> None:
        self.launches += 1
        if code != 0:
            detail = {-2: "a size is outside what the kernel takes", -3: "the grid would be too large",
                      -4: "unsupported dtype combination"}.get(code, f"CUDA error {code}")
            raise KernelError(f"{what}: {detail}")

    def check(self) -> None:
        """Read the kernels' error word; if a kernel flagged bad input (a token id or position out of
        range: the row was zeroed or skipped) or gave up on a bounded wait since the last look, clear
        the word and raise. The results of the step that raised it are not to be used. The generation
        loop reads the word with every step's tokens, the step function at the end of every
        multi-token step."""
        flag = int(self.error.item())
        if flag:
            self.error.zero_()
            raise KernelError(self.describe(flag))

    @staticmethod
    def describe(flag: int) -> str:
        known = {1: "a token id outside the embedding table reached the device",
                 2: "a position outside the rotary table reached the device",
                 3: "a tensor-core GEMM gave up waiting for a free shared-memory stage",
                 4: "a tensor-core GEMM gave up waiting for a TMA load",
                 5: "a tensor-core GEMM gave up waiting for its accumulator",
                 21: "the wait of the self-test kernel ran out (as it is meant to)"}
        if flag in known:
            return known[flag]
        if 6 <= flag <= 14:
            return f"the tensor-core attention kernel gave up on a barrier wait (code {flag})"
        return f"error flag {flag}"

    def selftest_wait_runs_out(self, limit_us: int = 1000) -> None:
        """Launch a kernel whose only wait, on a barrier nobody arrives at, runs out after ``limit_us``
        and sets the error word; ``check`` then raises. For the tests of the error path."""
        self._ok(self.core.krk_selftest_wait_runs_out(self.error.data_ptr(), int(limit_us), self._stream()), "self-test wait")

    def empty_like(self, x):
        return torch.empty_like(x)

    @staticmethod
    def _resolve(x):
        return x if isinstance(x, torch.Tensor) else x.tensor()

    # -- rows -------------------------------------------------------------------
    def embed(self, table, tokens, n_rows):
        out = torch.empty((n_rows, table.shape[1]), dtype=table.dtype, device=table.device)
        self._ok(self.core.krk_gather_rows(out.data_ptr(), table.data_ptr(), tokens.data_ptr(), n_rows, table.shape[1],
                                           table.shape[0], self.error.data_ptr(), _code(table.dtype), self._stream()),
                 "embedding gather")
        return out

    def gather_rows(self, x, idx):
        n = idx.shape[0]
        out = torch.empty((n, x.shape[1]), dtype=x.dtype, device=x.device)
        self._ok(self.core.krk_gather_rows(out.data_ptr(), x.data_ptr(), idx.data_ptr(), n, x.shape[1], x.shape[0],
                                           self.error.data_ptr(), _code(x.dtype), self._stream()), "row gather")
        return out

    def rmsnorm(self, x, gain, eps):
        out = torch.empty_like(x)
        self._ok(self.core.krk_rmsnorm(out.data_ptr(), None, x.data_ptr(), None, gain.data_ptr(),
                                       int(gain.dtype == torch.float32), x.shape[0], x.shape[1], eps, _code(x.dtype),
                                       self._stream()), "rmsnorm")
        return out

    def add_rmsnorm(self, x, branch, gain, eps, x_new):
        out = torch.empty_like(x)
        self._ok(self.core.krk_rmsnorm(out.data_ptr(), x_new.data_ptr(), x.data_ptr(), branch.data_ptr(),
                                       gain.data_ptr(), int(gain.dtype == torch.float32), x.shape[0], x.shape[1], eps,
                                       _code(x.dtype), self._stream()), "add + rmsnorm")
        return out

    def swiglu(self, gu, intermediate):
        out = torch.empty((gu.shape[0], intermediate), dtype=gu.dtype, device=gu.device)
        self._ok(self.core.krk_swiglu(out.data_ptr(), gu.data_ptr(), gu.shape[0], intermediate, _code(gu.dtype),
                                      self._stream()), "swiglu")
        return out

    # -- matrix products ----------------------------------------------------------
    def _gemm_nt(self, x, w, out_dtype):
        M, K = x.shape
        N = w.shape[0]
        out = torch.empty((M, N), dtype=out_dtype, device=x.device)
        self._ok(self.core.krk_gemm_nt(out.data_ptr(), x.data_ptr(), w.data_ptr(), M, N, K, x.stride(0), w.stride(0), N,
                                       _code(x.dtype), _code(out_dtype), self._stream()), "gemm")
        return out

    def gemm_tcgen05(self, x, w, swiglu_rows=0, variant=0, out_float32=False):
        """y = x W^T (bfloat16 inputs) on the tcgen05 tensor cores; with ``swiglu_rows`` = I,
        W is [2I, K] and y is the activated [M, I] product; ``out_float32`` keeps the
        accumulator's precision (output-head logits)."""
        M, K = x.shape
        N = swiglu_rows if swiglu_rows else w.shape[0]
        out = torch.empty((M, N), dtype=torch.float32 if out_float32 else torch.bfloat16, device=x.device)
        self._ok(self.core.krk_gemm_tcgen05(out.data_ptr(), x.data_ptr(), w.data_ptr(), M, N, K, x.stride(0), w.stride(0),
                                            N, int(swiglu_rows > 0), variant, int(out_float32), self.error.data_ptr(),
                                            self._stream()),
                 "tcgen05 gemm")
        return out

    def _skinny(self, x, w, out_dtype, swiglu_rows=0, gate_act=1, act_limit=0.0):
        """x: a tensor or a Normed not yet computed (then the add and the norm run in
        the kernel's prologue)."""
        lazy = not isinstance(x, torch.Tensor)
        src = x.x if lazy else x
        M, K = src.shape
        N = swiglu_rows if swiglu_rows else w.shape[0]
        out = torch.empty((M, N), dtype=out_dtype, device=src.device)
        branch = x.branch if lazy else None
        gain = x.gain if lazy else None
        x_new = x.x_new if lazy and x.branch is not None else None
        self._ok(self.core.krk_skinny_linear(
            out.data_ptr(), src.data_ptr(), w.data_ptr(), _ptr(branch), _ptr(gain), _ptr(x_new),
            int(gain is not None and gain.dtype == torch.float32), None, M, N, K, float(x.eps) if lazy else float(act_limit),
            int(gate_act if swiglu_rows > 0 or gate_act == 4 else 0), _code(out_dtype), self._stream()), "skinny product")
        if lazy:
            x.mark_fused()
        return out

    def _use_skinny(self, x, w) -> bool:
        rows = x.shape[0]
        return (self.has_skinny and w.dtype == torch.bfloat16 and 0 < rows <= self.SKINNY_MAX_ROWS
                and w.shape[1] % 32 == 0 and w.is_contiguous())

    @staticmethod
    def _fits_prologue(x) -> bool:
        """Whether the normalised rows fit the fused kernel's shared memory."""
        rows, k = x.shape
        if rows > Kernels.FUSED_NORM_MAX_ROWS:
            return False
        tiles = 1 if rows <= 8 else 2
        return 65536 + rows * (k + 64) * 2 + 8 * 2 * tiles * 512 <= 216 * 1024

    def _skinny_input(self, x):
        """A Normed goes to the kernel as it is if its norm is still to be done and fits
        the prologue; otherwise its rows are computed first."""
        if isinstance(x, torch.Tensor):
            return x
        if x.done or not self._fits_prologue(x):
            return x.tensor()
        return x

    def linear(self, x, w, out_float32=False):
        """y = x W^T; W is [out, in]. x may be a Normed (see parts/norm.py)."""
        out_dtype = torch.float32 if out_float32 else w.dtype
        if self._use_skinny(x, w):
            return self._skinny(self._skinny_input(x), w, out_dtype)
        x = self._resolve(x)
        if x.shape[0] == 0:
            return torch.empty((0, w.shape[0]), dtype=out_dtype, device=x.device)
        if w.dtype == torch.float32:
            return self._gemm_nt(x, w, out_dtype)
        if out_float32:  # many rows of float32 logits: the tcgen05 GEMM keeps the accumulator's precision
            if (x.shape[1] % 8 == 0 and x.stride(0) % 8 == 0 and w.stride(0) % 8 == 0 and x.data_ptr() % 16 == 0
                    and w.data_ptr() % 16 == 0 and hasattr(self.core, "krk_gemm_tcgen05")):
                return self.gemm_tcgen05(x, w, out_float32=True)
            return self._gemm_nt(x, w, out_dtype)
        if (self.use_tuned_library_gemm and x.stride(1) == 1 and w.stride(1) == 1 and x.stride(0) % 8 == 0
                and w.stride(0) % 8 == 0 and w.shape[0] % 8 == 0 and x.data_ptr() % 16 == 0 and w.data_ptr() % 16 == 0):
            return self._library_gemm(x, w)
        return torch.matmul(x, w.t())

    def _library_gemm(self, x, w):
        """The library's product with the algorithm picked by measurement (csrc/lt_gemm.cu)."""
        M, K = x.shape
        N = w.shape[0]
        out = torch.empty((M, N), dtype=torch.bfloat16, device=x.device)
        rc = self.core.krk_lt_gemm_bf16(x.data_ptr(), w.data_ptr(), out.data_ptr(), M, N, K, x.stride(0), w.stride(0), N, 1,
                                        None, self._stream())
        if rc:
            raise KernelError(f"the library product of {M} x {N} x {K} failed with code {rc}")
        return out

    def library_gemm_report(self):
        """(shape classes with a measured choice, how many of them kept the heuristic's first proposal)."""
        a, b = c_int(0), c_int(0)
        self.core.krk_lt_gemm_report(ctypes.byref(a), ctypes.byref(b))
        return a.value, b.value

    def gate_up_swiglu(self, h, w_gate_up, intermediate):
        if self._use_skinny(h, w_gate_up):
            return self._skinny(self._skinny_input(h), w_gate_up, w_gate_up.dtype, swiglu_rows=intermediate)
        return self.swiglu(self.linear(h, w_gate_up), intermediate)

    # -- attention ------------------------------------------------------------------
    def qk_norm_rope_write(self, qkv, heads, kv_in_row, head_dim, q_gain, k_gain, eps, cos, sin, batch, cache):
        gain = q_gain if q_gain is not None else k_gain
        n_pos = cos.shape[0] if cos is not None else 0x7fffffff
        rot = self._rotated_width(cos, head_dim)
        self._ok(self.core.krk_qk_norm_rope_write(
            qkv.data_ptr(), _ptr(q_gain), _ptr(k_gain), int(gain is not None and gain.dtype == torch.float32),
            _ptr(cos), _ptr(sin), batch.row_seq.data_ptr(), batch.row_pos.data_ptr(), batch.seq_slot.data_ptr(),
            cache.table.data_ptr(), cache.width, cache.k.data_ptr() if kv_in_row else None,
            cache.v.data_ptr() if kv_in_row else None, qkv.shape[0], heads, kv_in_row, head_dim, rot, eps, n_pos,
            self.error.data_ptr(), _code(qkv.dtype), self._stream()), "q/k norm + rope + cache write")

    @staticmethod
    def _rotated_width(cos, head_dim: int) -> int:
        """The width of the head that the tables rotate: all of it, or its first 2 * columns elements."""
        if cos is None:
            return head_dim
        rot = 2 * cos.shape[1]
        if rot > head_dim or not cos.is_contiguous():
            raise KernelError(f"rotary tables of {cos.shape[1]} columns do not fit a head of {head_dim} (at most half of it, contiguous)")
        return rot

    def rope_attention(self, qkv, heads, kv_in_row, head_dim, q_gain, k_gain, eps, cos, sin, batch, cache, scale,
                       window):
        """Per-head q/k norm, rotation, cache write and attention. A single-token step in
        bfloat16 runs them as one kernel; everything else as two."""
        lib = self._attn_lib(head_dim)
        if (batch.is_decode and qkv.dtype == torch.bfloat16 and head_dim % 16 == 0 and kv_in_row > 0
                and hasattr(lib, "krk_attention_decode_fused") and qkv.shape[0] > 0
                and self._rotated_width(cos, head_dim) == head_dim):  # the fused kernel rotates the whole head
            n = batch.n_seqs
            out = torch.empty((n, heads * head_dim), dtype=qkv.dtype, device=qkv.device)
            row_tiles = -(-(heads // cache.kv_heads) // 16)
            # key splits (blocks per cluster) by the number of (sequence, kv head, row tile) items alone,
            # never by lengths, so a captured step stays valid; measured best on B200 at 1, 2 to 4, 8, 16 and 32 or
            # 64 sequences of the 4B shape: 16, 8, 4, 2 and 1 (one block per item runs a deeper page pipeline). One
            # sequence has eight items: sixteen splits are 128 blocks where eight are 64, and what bounds the
            # kernel is the bytes its blocks have in flight (one step of the 4B shape at 32,000 tokens of context:
            # 4.41 -> 3.14 ms, at 8,000: 2.51 -> 2.17, at 1,000: 1.93 -> 1.91; at two sequences sixteen gain nothing)
            items = n * cache.kv_heads * row_tiles
            splits = 16 if items <= 9 else 8 if items <= 37 else 4 if items <= 74 else 2 if items <= 192 else 1
            gain = q_gain if q_gain is not None else k_gain
            n_pos = cos.shape[0] if cos is not None else 0x7fffffff
            if (splits in self.tma_decode_splits and self.use_tma_decode_attention and head_dim % 64 == 0
                    and cache.width <= 1024 and hasattr(lib, "krk_attention_decode_fused_tma")):
                # many sequences: one block or two per (sequence, kv head), pages by TMA into a ring of half page-pairs
                rc = lib.krk_attention_decode_fused_tma(
                    out.data_ptr(), qkv.data_ptr(), qkv.stride(0), heads, cache.kv_heads, _ptr(q_gain), _ptr(k_gain),
                    int(gain is not None and gain.dtype == torch.float32), _ptr(cos), _ptr(sin), eps,
                    batch.seq_slot.data_ptr(), batch.seq_start.data_ptr(), cache.table.data_ptr(), cache.width,
                    cache.k.data_ptr(), cache.v.data_ptr(), cache.k.shape[0], n, scale, int(window or 0), splits, n_pos,
                    self.error.data_ptr(), self._stream())
                if rc != -2:  # -2: the shapes do not fit this kernel's shared memory; the kernel below takes them
                    self._ok(rc, "fused decode attention (TMA)")
                    return out
            self._ok(lib.krk_attention_decode_fused(
                out.data_ptr(), qkv.data_ptr(), qkv.stride(0), heads, cache.kv_heads, _ptr(q_gain), _ptr(k_gain),
                int(gain is not None and gain.dtype == torch.float32), _ptr(cos), _ptr(sin), eps,
                batch.seq_slot.data_ptr(), batch.seq_start.data_ptr(), cache.table.data_ptr(), cache.width,
                cache.k.data_ptr(), cache.v.data_ptr(), n, scale, int(window or 0), splits, n_pos,
                self.error.data_ptr(), self._stream()), "fused decode attention")
            return out
        self.qk_norm_rope_write(qkv, heads, kv_in_row, head_dim, q_gain, k_gain, eps, cos, sin, batch, cache)
        return self.attention(qkv, heads, kv_in_row, head_dim, batch, cache, scale, window)

    def attention(self, qkv, heads, kv_in_row, head_dim, batch, cache, scale, window):
        lib = self._attn_lib(head_dim)
        rows = qkv.shape[0]
        out = torch.empty((rows, heads * head_dim), dtype=qkv.dtype, device=qkv.device)
        if rows == 0:
            return out
        stride = qkv.stride(0)
        win = int(window or 0)
        fast = qkv.dtype == torch.bfloat16 and head_dim % 16 == 0
        if fast and batch.is_decode and hasattr(lib, "krk_attention_decode"):
            splits, parts = self._decode_partials(batch.n_seqs, heads, cache.kv_heads, head_dim)
            self._ok(lib.krk_attention_decode(
                out.data_ptr(), qkv.data_ptr(), stride, heads, cache.kv_heads, batch.seq_slot.data_ptr(),
                batch.seq_start.data_ptr(), cache.table.data_ptr(), cache.width, cache.k.data_ptr(),
                cache.v.data_ptr(), batch.n_seqs, scale, win, splits, parts.data_ptr(), self._stream()),
                "decode attention")
        elif (fast and self.use_tcgen05_attention and head_dim in (64, 128) and hasattr(lib, "krk_attention_prefill_tcgen05")
              and batch.max_q_len * (heads // cache.kv_heads) >= 128 and stride % 8 == 0):
            # long steps: the tcgen05 kernel (128-row tiles of (token, group member) pairs)
            self._ok(lib.krk_attention_prefill_tcgen05(
                out.data_ptr(), qkv.data_ptr(), stride, heads, cache.kv_heads, batch.seq_slot.data_ptr(),
                batch.seq_start.data_ptr(), batch.seq_qlen.data_ptr(), batch.cu_q.data_ptr(), cache.table.data_ptr(),
                cache.width, cache.k.data_ptr(), cache.v.data_ptr(), cache.k.shape[0], batch.n_seqs, batch.max_q_len,
                rows, scale, win, self.error.data_ptr(), self._stream()), "tcgen05 prefill attention")
        elif fast and hasattr(lib, "krk_attention_prefill"):
            self._ok(lib.krk_attention_prefill(
                out.data_ptr(), qkv.data_ptr(), stride, heads, cache.kv_heads, batch.seq_slot.data_ptr(),
                batch.seq_start.data_ptr(), batch.seq_qlen.data_ptr(), batch.cu_q.data_ptr(), cache.table.data_ptr(),
                cache.width, cache.k.data_ptr(), cache.v.data_ptr(), batch.n_seqs, batch.max_q_len, scale, win,
                self._stream()), "prefill attention")
        else:
            self._ok(lib.krk_attention_simple(
                out.data_ptr(), qkv.data_ptr(), stride, heads, cache.kv_heads, batch.row_seq.data_ptr(),
                batch.row_pos.data_ptr(), batch.seq_slot.data_ptr(), cache.table.data_ptr(), cache.width,
                cache.k.data_ptr(), cache.v.data_ptr(), rows, scale, win, _code(qkv.dtype), self._stream()),
                "attention")
        return out

    def _decode_partials(self, n_seqs: int, heads: int, kv_heads: int, head_dim: int):
        """Number of key splits for a decode step and the float32 scratch its partial
        results go through. The split count depends on the batch size only, never on
        lengths, so a captured step stays valid as sequences grow."""
        row_tiles = -(-(heads // kv_heads) // 16)
        splits = max(1, min(32, -(-296 // (n_seqs * kv_heads * row_tiles))))
        key = (n_seqs, heads, head_dim, splits)
        buf = self._partials.get(key)
        if buf is None:
            buf = self._partials[key] = torch.empty(n_seqs * heads * splits * (head_dim + 2), dtype=torch.float32,
                                                    device=self.device)
        return splits, buf

    # -- 32-bit residual stream, windowed attention with a sink, recurrent state -------------------
    @property
    def mix(self) -> ctypes.CDLL:
        """The library of these kernels, compiled and loaded when a model first asks for one of them."""
        if self._mix is None:
            self._mix = _load(build_library("mix"), _MIX_SIGNATURES)
        return self._mix

    @property
    def scan(self) -> ctypes.CDLL:
        """The library of the recurrent-state kernels, compiled and loaded at their first call."""
        if self._scan is None:
            self._scan = _load(build_library("scan"), _SCAN_SIGNATURES)
        return self._scan

    @property
    def memory(self) -> ctypes.CDLL:
        """The library of the matrix-state mixers without a removal term, compiled and loaded at their first call."""
        if self._memory is None:
            self._memory = _load(build_library("memory"), _MEMORY_SIGNATURES)
        return self._memory

    @property
    def moe(self) -> ctypes.CDLL:
        """The library of the routed-experts kernels, compiled and loaded at their first call."""
        if self._moe is None:
            self._moe = _load(build_library("moe"), _MOE_SIGNATURES)
        return self._moe

    @staticmethod
    def _rows_view(t):
        """(pointer, row stride) of a 2-D view whose rows are contiguous."""
        if t.dim() != 2 or t.stride(1) != 1:
            raise KernelError("a kernel input must be a 2-D tensor (or column slice) with contiguous rows")
        return t.data_ptr(), t.stride(0)

    def embed_scaled(self, table, tokens, n_rows, scale, copies=1, rounded=False):
        """float32 rows table[token] * scale, each written ``copies`` times side by side. With ``rounded`` (one copy) a
        pair: the rows, and the same rows in the table's dtype."""
        if rounded and copies != 1:
            raise KernelError("rounded rows come with one copy of the row")
        out = torch.empty((n_rows, copies * table.shape[1]), dtype=torch.float32, device=table.device)
        again = torch.empty(out.shape, dtype=table.dtype, device=table.device) if rounded and table.dtype != torch.float32 else None
        self._ok(self.mix.krk_embed_scaled(out.data_ptr(), table.data_ptr(), tokens.data_ptr(), n_rows, table.shape[1],
                                           table.shape[0], float(scale), self.error.data_ptr(), _code(table.dtype),
                                           self._stream(), int(copies), _ptr(again)), "scaled embedding gather")
        if rounded:
            return out, (again if again is not None else out)
        return out

    def post_norm(self, x, branch, gain, offset, eps, out_dtype):
        """(x + norm(branch) * (offset + gain), the same rows in ``out_dtype``): a float32 stream takes a sublayer's output,
        RMS-normed on its way in. Without a branch the stream is only rounded."""
        if x.dtype != torch.float32 or not x.is_contiguous() or (branch is not None and gain.dtype != torch.float32):
            raise KernelError("the norm of an output reads a contiguous float32 stream and a float32 gain")
        if branch is not None and (branch.dtype != out_dtype or not branch.is_contiguous() or branch.shape != x.shape):
            raise KernelError("a sublayer's output must have the path's dtype and the stream's shape")
        x_new = torch.empty_like(x) if branch is not None else x
        rows = x_new if out_dtype == torch.float32 else torch.empty(x.shape, dtype=out_dtype, device=x.device)
        if branch is None and rows is x:
            return x, x
        self._ok(self.mix.krk_post_norm(x_new.data_ptr(), rows.data_ptr() if rows is not x_new else None, x.data_ptr(),
                                        _ptr(branch), _ptr(gain), float(offset), x.shape[0], x.shape[1], float(eps),
                                        _code(out_dtype), self._stream()), "norm of an output into the stream")
        return x_new, rows

    def tanh_cap_(self, logits, cap):
        """logits <- cap * tanh(logits / cap), in place (float32, contiguous)."""
        if logits.dtype != torch.float32 or not logits.is_contiguous():
            raise KernelError("logits are capped as contiguous float32 rows")
        self._ok(self.mix.krk_tanh_cap(logits.data_ptr(), logits.numel(), float(cap), self._stream()), "logit cap")
        return logits

    def hyper_rmsnorm(self, x, branch, fold, read, gain, offset, eps, x_new, out_dtype):
        """Rows of S float32 streams side by side. With a pending ``branch``, the streams are rewritten into ``x_new``
        through ``fold`` (M [S, S] indexed [from, to], then b [S]): x_t = sum_s M[s, t] x_s + b_t * branch. Returns
        norm(sum_s read[s] x_s) * (offset + gain) in ``out_dtype``."""
        S = read.shape[0]
        rows, C = x.shape[0], x.shape[1] // S
        if x.dtype != torch.float32 or not x.is_contiguous() or gain.dtype != torch.float32 or gain.shape[0] != C:
            raise KernelError("the hyper-connection norm reads contiguous float32 streams and a float32 gain")
        if branch is not None and (branch.dtype != out_dtype or not branch.is_contiguous() or branch.shape != (rows, C)
                                   or fold is None or fold.numel() != S * S + S):
            raise KernelError("the pending output must have the path's dtype and one stream's shape, with its M and b")
        out = torch.empty((rows, C), dtype=out_dtype, device=x.device)
        self._ok(self.mix.krk_hyper_rmsnorm(out.data_ptr(), x_new.data_ptr() if branch is not None else None, x.data_ptr(),
                                            _ptr(branch), _ptr(fold) if branch is not None else None, read.data_ptr(),
                                            gain.data_ptr(), float(offset), rows, S, C, float(eps), _code(out_dtype),
                                            self._stream()), "hyper-connection rmsnorm")
        return out

    def bias_row_norm(self, proj, cols, bias, gain, eps):
        """In place on a stacked q | k | v product: ``cols`` = (q0, k0, v0, end) column bounds; float32 ``bias`` over
        q0..end is added (None: none), and with ``gain`` (float32 over q0..v0) the q columns and the k columns are each
        divided by their root mean square and multiplied by it."""
        ptr, stride = self._rows_view(proj)
        q0, k0, v0, end = (int(c) for c in cols)
        if (bias is not None and bias.numel() != end - q0) or (gain is not None and gain.numel() != v0 - q0):
            raise KernelError("bias and gain must cover the columns they are applied to")
        self._ok(self.mix.krk_bias_row_norm(ptr, stride, q0, k0, v0, end, _ptr(bias), _ptr(gain), float(eps), proj.shape[0],
                                            _code(proj.dtype), self._stream()), "projection biases + row norms")

    def rmsnorm_wide(self, x, branch, gain, offset, eps, x_new, out_dtype, branch2=None, scale=1.0, gain2=None):
        """Rows of a float32 stream, normalised into ``out_dtype``; with a branch, ``x_new`` = x + scale * (branch +
        branch2) (float32). With a second gain, two results of the one pass: (rows, rows2)."""
        if x.dtype != torch.float32 or gain.dtype != torch.float32 or not x.is_contiguous():
            raise KernelError("the wide norm reads a contiguous float32 stream and a float32 gain")
        for b in (branch, branch2):
            if b is not None and (b.dtype != out_dtype or not b.is_contiguous() or b.shape != x.shape):
                raise KernelError("the wide norm's branch must have the path's dtype and the stream's shape")
        if gain2 is not None and (gain2.dtype != torch.float32 or gain2.shape != gain.shape):
            raise KernelError("the wide norm's second gain must be float32 and of the first one's size")
        out = torch.empty(x.shape, dtype=out_dtype, device=x.device)
        out2 = torch.empty(x.shape, dtype=out_dtype, device=x.device) if gain2 is not None else None
        self._ok(self.mix.krk_rmsnorm_wide(out.data_ptr(), x_new.data_ptr() if branch is not None else None, x.data_ptr(),
                                           _ptr(branch), gain.data_ptr(), float(offset), x.shape[0], x.shape[1], float(eps),
                                           _ptr(branch2), float(scale), _ptr(gain2), _ptr(out2), _code(out_dtype),
                                           self._stream()), "wide rmsnorm")
        return out if gain2 is None else (out, out2)

    def tanh_norm(self, x, branch, fold, alpha, gain, shift, x_new, out_dtype):
        """tanh(alpha * s) * gain + shift in ``out_dtype`` with s = x (float32), or x + fold * branch, written to ``x_new``
        (``fold``: a float32 vector, None: 1)."""
        C = x.shape[1]
        if x.dtype != torch.float32 or not x.is_contiguous() or any(
                t is not None and (t.dtype != torch.float32 or t.numel() != C) for t in (gain, shift, fold)):
            raise KernelError("this norm reads a contiguous float32 stream and float32 vectors of its width")
        if branch is not None and (branch.dtype != out_dtype or not branch.is_contiguous() or branch.shape != x.shape):
            raise KernelError("the pending output must have the path's dtype and the stream's shape")
        out = torch.empty(x.shape, dtype=out_dtype, device=x.device)
        self._ok(self.mix.krk_tanh_norm(out.data_ptr(), x_new.data_ptr() if branch is not None else None, x.data_ptr(),
                                        _ptr(branch), _ptr(fold) if branch is not None else None, float(alpha),
                                        gain.data_ptr(), shift.data_ptr(), x.shape[0], C, _code(out_dtype), self._stream()),
                 "tanh norm")
        return out

    def gated_act(self, gu, intermediate, activation, row_gate_col=None, act_params=None):
        """act(gu[:, :I]) * gu[:, I:2I], times sigmoid(gu[:, row_gate_col]) per row if that column is given.
        "swish_clamped" takes ``act_params`` = (limit, slope)."""
        ptr, stride = self._rows_view(gu)
        out = torch.empty((gu.shape[0], intermediate), dtype=gu.dtype, device=gu.device)
        limit, slope = act_params if act_params is not None else (0.0, 1.0)
        if activation == "swish_clamped" and act_params is None:
            raise KernelError("the clamped activation needs its limit and slope")
        self._ok(self.mix.krk_gated_act(out.data_ptr(), ptr, stride, gu.shape[0], intermediate, _ACTIVATIONS[activation],
                                        -1 if row_gate_col is None else int(row_gate_col), _code(gu.dtype),
                                        self._stream(), float(limit), float(slope)), "gated activation")
        return out

    def latent_norm_write(self, proj, c_col, rank, gain, eps, batch, cache, keep_rows=False):
        """The rows' ``rank`` columns from ``c_col`` on, RMS-normed with a float32 gain, into the cache (one head);
        with ``keep_rows`` the normalised rows are returned as well, [rows, rank]."""
        ptr, stride = self._rows_view(proj)
        if cache.k.dtype != proj.dtype or cache.head_dim != rank or cache.kv_heads != 1 or gain.dtype != torch.float32:
            raise KernelError("the cache does not fit the latent rows it is to receive")
        kept = torch.empty((proj.shape[0], rank), dtype=proj.dtype, device=proj.device) if keep_rows else None
        self._ok(self.mix.krk_latent_norm_write(ptr, stride, int(c_col), int(rank), gain.data_ptr(), float(eps),
                                                batch.row_seq.data_ptr(), batch.row_pos.data_ptr(),
                                                batch.seq_slot.data_ptr(), cache.table.data_ptr(), cache.width,
                                                int(getattr(cache, "keep_pages", 0)), cache.k.data_ptr(), proj.shape[0],
                                                _ptr(kept), _code(proj.dtype), self._stream()), "latent norm + cache write")
        return kept

    def head_linear(self, x, w, out=None, out_col=0, out_scale=1.0):
        """out[r, h, :] = out_scale * W_h x[r, h, :]; W [heads, N, K] contiguous, x [rows, heads * K] (rows may be strided)."""
        heads, N, K = w.shape
        ptr, stride = self._rows_view(x)
        if x.shape[1] != heads * K or w.dtype != x.dtype or not w.is_contiguous():
            raise KernelError("the per-head product reads [rows, heads * K] rows and a contiguous [heads, N, K] weight of one dtype")
        if out is None:
            out = torch.empty((x.shape[0], heads * N), dtype=x.dtype, device=x.device)
        optr, ostride = self._rows_view(out)
        rows = x.shape[0]
        if rows > self.SKINNY_MAX_ROWS and x.dtype == torch.bfloat16:
            # many rows in bfloat16: the library's batched product, one batch entry per head
            y = torch.bmm(x.view(rows, heads, K).transpose(0, 1), w.transpose(1, 2))  # [heads, rows, N]
            dst = out[:, out_col:out_col + heads * N].view(rows, heads, N)
            if out_scale == 1.0:
                dst.copy_(y.transpose(0, 1))
            else:
                torch.mul(y.transpose(0, 1), out_scale, out=dst)
            return out
        self._ok(self.mix.krk_head_linear(optr, ostride, int(out_col), N, float(out_scale), ptr, stride, K, w.data_ptr(), heads,
                                          N, K, x.shape[0], 0, None, 1.0, None, None, 0, _code(x.dtype), self._stream()),
                 "per-head product")
        return out

    # -- latent attention with a rotated part ------------------------------------------------
    def latent_rows(self, proj, query, rows, rot_dim, inv_freq, rot_factor, eps, batch, cache):
        """``query`` (column, size, gain): those columns of ``proj``, RMS-normed with a float32 gain, are returned. ``rows``
        (column, rank, gain) or None: that many columns likewise, and behind them ``rot_dim`` columns rotated, go to the
        positions' places in the cache."""
        ptr, stride = self._rows_view(proj)
        q_col, q_size, q_gain = query
        c_col, rank, c_gain = rows if rows is not None else (0, 0, None)
        if rows is not None and (cache.k.dtype != proj.dtype or cache.head_dim != rank + rot_dim or cache.kv_heads != 1
                                 or c_gain.dtype != torch.float32):
            raise KernelError("the cache does not fit the latent rows it is to receive")
        out = torch.empty((proj.shape[0], q_size), dtype=proj.dtype, device=proj.device)
        self._ok(self.mix.krk_latent_rows(out.data_ptr(), ptr, stride, int(q_col), int(q_size), q_gain.data_ptr(), int(c_col),
                                          int(rank), _ptr(c_gain), int(rot_dim), inv_freq.data_ptr(), float(rot_factor),
                                          float(eps), batch.row_seq.data_ptr(), batch.row_pos.data_ptr(),
                                          batch.seq_slot.data_ptr(), cache.table.data_ptr(), cache.width,
                                          cache.k.data_ptr() if rows is not None else None, proj.shape[0], _code(proj.dtype),
                                          self._stream()), "low-rank rows")
        return out

    def rotated_latent_attention(self, q, m, batch, cache, gate, out, out_col, out_scale, shared):
        """Attention of queries [rows, heads * (dim + rot)] (not rotated yet) over the cached rows [latent | rotated key],
        times sigmoid of ``gate`` = (rows, first column), into ``out``'s columns. ``m`` gives the sizes and weights
        (parts/latent_attention.py)."""
        H, D, E, R, P = m.heads, m.dim, m.rot, m.rank, m.vdim
        rows = q.shape[0]
        W = R + E
        g_ptr, g_stride = self._rows_view(gate[0])
        g_ptr += int(gate[1]) * gate[0].element_size()
        optr, ostride = self._rows_view(out)
        if self._latent_prefill(q, m, batch, cache, g_ptr, g_stride, optr, ostride, out_col, out_scale, shared):
            return
        # a head's query is carried into the latent space, attention runs over the cached rows themselves
        qx = torch.empty((rows, H * W), dtype=q.dtype, device=q.device)
        self._ok(self.mix.krk_head_linear(qx.data_ptr(), H * W, 0, W, 1.0, q.data_ptr(), q.stride(0), D + E, m.uk_t.data_ptr(), H,
                                          R, D, rows, E, m.inv_freq.data_ptr(), float(m.rot_factor), batch.row_pos.data_ptr(),
                                          None, 0, _code(q.dtype), self._stream()), "queries into the latent space")
        mixed = torch.empty((rows, H * R), dtype=q.dtype, device=q.device)
        if not self._latent_decode(qx, H, R, W, m.scale, batch, cache, mixed):
            self.sink_attention(qx, 0, H, W, R, None, m.scale, None, batch, cache, mixed, 0, 1.0)
        self._ok(self.mix.krk_head_linear(optr, ostride, int(out_col), P, float(out_scale), mixed.data_ptr(), H * R, R,
                                          m.uv.data_ptr(), H, P, R, rows, 0, None, 1.0, None, g_ptr, g_stride, _code(q.dtype),
                                          self._stream()), "values out of the latent space")

    def _latent_decode(self, qx, H, R, W, scale, batch, cache, mixed) -> bool:
        """A single-token step in bfloat16 on the tensor cores; False where the step or the sizes are not of that kind."""
        if not batch.is_decode or qx.dtype != torch.bfloat16 or R % 16 or W % 16 or R > 512:
            return False
        # blocks that share a sequence's pages by the step's shape alone, so that a captured step stays valid
        splits = max(1, min(32, 148 // (batch.n_seqs * -(-H // 16))))
        key = ("latent", batch.n_seqs, H, R, splits)
        scratch = self._partials.get(key)
        if scratch is None:
            scratch = self._partials[key] = torch.empty(batch.n_seqs * H * splits * (R + 2), dtype=torch.float32, device=self.device)
        rc = self.mix.krk_latent_decode(mixed.data_ptr(), scratch.data_ptr(), qx.data_ptr(), qx.stride(0), H, R, W,
                                        batch.seq_slot.data_ptr(), batch.seq_start.data_ptr(), cache.table.data_ptr(), cache.width,
                                        cache.k.data_ptr(), float(scale), splits, batch.n_seqs, self._stream())
        if rc == -2:
            return False
        self._ok(rc, "single-token attention over latent rows")
        self.launches += 1
        return True

    LATENT_DENSE_BYTES = 4 << 30  # keys and values of a step's whole context beyond this size are not written out

    def _latent_prefill(self, q, m, batch, cache, g_ptr, g_stride, optr, ostride, out_col, out_scale, shared) -> bool:
        """A step of many tokens in bfloat16: the sequences' cached rows as one dense matrix, keys and values from it by one
        product, tensor-core attention over those. False where the step or the sizes are not of that kind."""
        H, D, E, R, P = m.heads, m.dim, m.rot, m.rank, m.vdim
        if (batch.is_decode or q.dtype != torch.bfloat16 or D % 8 or E % 8 or R % 8 or (D + E) % 16 or P % 16 or D + E > 256
                or P > 256 or q.stride(0) % 8):
            return False
        lengths = [s + n for s, n in zip(batch.starts, batch.q_lens)]
        if 2 * sum(lengths) * H * (D + P) > self.LATENT_DENSE_BYTES:
            return False
        offsets = shared.get("latent_offsets")
        if offsets is None:
            at, first = [], 0
            for n in lengths:
                at.append(first)
                first += n
            offsets = shared["latent_offsets"] = torch.tensor(at, dtype=torch.int32).to(q.device)
        key = ("latent_rows", cache.k.data_ptr())  # layers that read one cache share the matrix
        rows = shared.get(key)
        if rows is None:
            rows = shared[key] = torch.empty((sum(lengths), R + E), dtype=q.dtype, device=q.device)
            self._ok(self.mix.krk_latent_gather(rows.data_ptr(), cache.k.data_ptr(), R + E, batch.n_seqs, max(lengths),
                                                batch.seq_slot.data_ptr(), batch.seq_start.data_ptr(), batch.seq_qlen.data_ptr(),
                                                offsets.data_ptr(), cache.table.data_ptr(), cache.width, _code(q.dtype),
                                                self._stream()), "cached rows as a matrix")
        latent = rows[:, :R]
        kv = self.linear(latent if rows.shape[0] > self.SKINNY_MAX_ROWS else latent.contiguous(), m.w_expand)
        rc = self._latent_lib(D + E, P).krk_latent_prefill(
            optr + int(out_col) * 2, ostride, float(out_scale), q.data_ptr(), q.stride(0), H, D, kv.data_ptr(), rows.data_ptr(),
            R + E, R, m.inv_freq.data_ptr(), float(m.rot_factor), float(m.scale), batch.n_seqs, batch.max_q_len,
            batch.seq_start.data_ptr(), batch.seq_qlen.data_ptr(), batch.cu_q.data_ptr(), offsets.data_ptr(), g_ptr, g_stride,
            self._stream())
        if rc == -2:  # odd strides or offsets; the general kernels take them
            return False
        self._ok(rc, "prompt attention over latent rows")
        return True

    # -- routed experts ------------------------------------------------------------------------
    MOE_PAIR_ROWS = 16  # rows up to which every (row, expert) pair reads its expert's weights by itself

    def moe_route(self, x, w, b, top, gate_row=False, over_all=False, sigmoid_groups=None, sigmoid=False):
        """(experts int32 [rows, top], weights float32 [rows, top], row gate float32 [rows] or None): the ``top`` largest
        of x W^T + b in 32-bit (ties: the lower index) and the softmax over them, or with ``over_all`` their shares of
        the softmax over all experts, or with ``sigmoid`` the sigmoid of each chosen logit. With ``gate_row`` the last row of W is no expert but a gate's weights: sigmoid
        of its product is the row gate. ``sigmoid_groups`` = (correction, groups, keep, scale): sigmoid scores, the choice
        by score + correction among the experts of the ``keep`` best of ``groups`` groups of neighbours, the weights
        the chosen scores over their sum, times ``scale``."""
        E = w.shape[0] - int(gate_row)
        rows, K = x.shape
        experts = torch.empty((rows, top), dtype=torch.int32, device=x.device)
        weights = torch.empty((rows, top), dtype=torch.float32, device=x.device)
        row_gate = torch.empty(rows, dtype=torch.float32, device=x.device) if gate_row else None
        logits = self.linear(x, w, out_float32=True)
        if sigmoid_groups is not None:
            correction, groups, keep, scale = sigmoid_groups
            if correction.dtype != torch.float32 or correction.numel() != E:
                raise KernelError("the routing correction is one float32 number per expert")
            self._ok(self.moe.krk_moe_route_groups(experts.data_ptr(), weights.data_ptr(), _ptr(row_gate), logits.data_ptr(),
                                                   correction.data_ptr(), rows, E, int(gate_row), int(top), int(groups),
                                                   int(keep), float(scale), self._stream()), "expert routing within groups")
            return experts, weights, row_gate
        self._ok(self.moe.krk_moe_route(experts.data_ptr(), weights.data_ptr(), _ptr(row_gate), logits.data_ptr(), _ptr(b),
                                        rows, E, int(gate_row), int(top), self._stream(), 2 if sigmoid else int(over_all)),
                 "expert routing")
        return experts, weights, row_gate

    def moe_route_softmax_groups(self, x, w, correction, top, groups, keep, identity, gate_row=False):
        """(experts int32 [rows, top], weights float32 [rows, top], row gate or None, passed float32 [rows] or None): softmax
        scores over all outputs, the choice by score + correction among the outputs of the ``keep`` best of ``groups``
        groups of neighbours (a group's score: its largest), the weights the chosen scores. The last ``identity`` outputs
        hand their input through: such a choice is expert -1 with weight 0, and its weight is in ``passed``. ``gate_row`` as
        in ``moe_route``."""
        outputs = w.shape[0] - int(gate_row)
        rows = x.shape[0]
        if correction.dtype != torch.float32 or correction.numel() != outputs:
            raise KernelError("the routing correction is one float32 number per output of the router")
        experts = torch.empty((rows, top), dtype=torch.int32, device=x.device)
        weights = torch.empty((rows, top), dtype=torch.float32, device=x.device)
        row_gate = torch.empty(rows, dtype=torch.float32, device=x.device) if gate_row else None
        passed = torch.empty(rows, dtype=torch.float32, device=x.device) if identity else None
        logits = self.linear(x, w, out_float32=True)
        self._ok(self.moe.krk_moe_route_softmax_groups(experts.data_ptr(), weights.data_ptr(), _ptr(row_gate), _ptr(passed),
                                                       logits.data_ptr(), correction.data_ptr(), rows, outputs,
                                                       outputs - int(identity), int(gate_row), int(top), int(groups), int(keep),
                                                       self._stream()), "expert routing by softmax within groups")
        return experts, weights, row_gate, passed

    def up_act(self, h, w_up, activation):
        """act(up h), without a gate; the squared relu of few bfloat16 rows runs in the product's epilogue."""
        if activation == "relu2" and self._use_skinny(h, w_up):
            return self._skinny(self._resolve(h), w_up, w_up.dtype, gate_act=4)
        return self.act_rows(self.linear(h, w_up), activation)

    def moe_experts(self, x, w_gate_up, w_down, experts, weights, intermediate, activation, add=None, add_gate=None,
                    batch=None, gated=True, add_input=None, act_params=None, weigh_input=False):
        """add * add_gate + add_input * x + sum_j weights[r, j] * expert_{experts[r, j]}(x[r]) over the choices that are not
        -1; w_gate_up [E, 2F, K] ([E, F, K] without ``gated``), w_down [E, C, F]; ``add_gate`` (None: 1) and ``add_input``
        (None: 0): one float32 number per row. ``act_params``: limit and slope of "swish_clamped". ``weigh_input``: the sum is
        over expert(weights[r, j] * x[r]) instead."""
        rows, top = experts.shape
        E, C, F = w_down.shape
        K = x.shape[1]
        ptr, stride = self._rows_view(x)
        out = torch.empty((rows, C), dtype=x.dtype, device=x.device)
        act = _ACTIVATIONS[activation]
        if activation == "swish_clamped" and (act_params is None or not gated):
            raise KernelError("the clamped activation needs its limit and slope, and experts with a gate")
        limit, slope = act_params if act_params is not None else (0.0, 1.0)
        w_in, w_out = (weights, None) if weigh_input else (None, weights)  # which end of an expert the weights multiply
        single = batch is not None and batch.is_decode  # such a step may be replayed from a graph: nothing comes to the host
        if single or rows * top <= max(self.MOE_PAIR_ROWS * top, 2 * E):
            pairs = torch.empty((rows * top, F), dtype=x.dtype, device=x.device)
            self._ok(self.moe.krk_moe_gate_up_pairs(pairs.data_ptr(), ptr, stride, w_gate_up.data_ptr(), experts.data_ptr(),
                                                    rows, top, F, K, act, int(gated), _ptr(w_in), float(limit), float(slope),
                                                    _code(x.dtype), self._stream()), "experts' gate/up")
            self._ok(self.moe.krk_moe_down_pairs(out.data_ptr(), _ptr(add), _ptr(add_gate), pairs.data_ptr(), w_down.data_ptr(),
                                                 experts.data_ptr(), _ptr(w_out), rows, top, C, F, ptr, stride,
                                                 _ptr(add_input), _code(x.dtype), self._stream()), "experts' down")
            return out
        # many rows: ordered by expert on the device; the experts' row counts come to the host (a step of many
        # tokens is never replayed from a graph)
        offsets = torch.empty(E + 1, dtype=torch.int32, device=x.device)
        place = torch.empty(rows * top, dtype=torch.int32, device=x.device)
        self._ok(self.moe.krk_moe_sort(offsets.data_ptr(), place.data_ptr(), experts.data_ptr(), rows, top, E,
                                       self._stream()), "expert ordering")
        if self._use_grouped(x, K, F, C, gated, activation):
            return self._grouped_experts(x, w_gate_up, w_down, experts, w_in, w_out, activation, (limit, slope), add, add_gate,
                                         gated, add_input, offsets, place)
        bounds = offsets.tolist()
        most = max(bounds[e + 1] - bounds[e] for e in range(E))
        cap = -(-most // 16) * 16
        batched = x.dtype == torch.bfloat16 and E * cap <= 4 * rows * top
        if not batched:
            cap = 0
        n_rows = E * cap if batched else rows * top
        xg = torch.empty((n_rows, K), dtype=x.dtype, device=x.device)
        self._ok(self.moe.krk_moe_gather(xg.data_ptr(), ptr, stride, place.data_ptr(), experts.data_ptr(), offsets.data_ptr(),
                                         cap, rows, top, K, _ptr(w_in), None, _code(x.dtype), self._stream()), "expert gather")
        if batched:
            # bfloat16: every expert's rows start at a multiple of cap (the most rows any expert got), and the
            # library's batched product takes all experts at once; the rows beyond an expert's own are never read back
            gu = torch.bmm(xg.view(E, cap, K), w_gate_up.transpose(1, 2))
            h = self.gated_act(gu.view(E * cap, 2 * F), F, activation, act_params=act_params) if gated else self.act_rows(gu.view(E * cap, F), activation)
            yg = torch.bmm(h.view(E, cap, F), w_down.transpose(1, 2)).view(E * cap, C)
        else:
            yg = torch.empty((n_rows, C), dtype=x.dtype, device=x.device)
            for e in range(E):
                a, b = bounds[e], bounds[e + 1]
                if b > a:
                    h = self.gate_up_act(xg[a:b], w_gate_up[e], F, activation, act_params) if gated else self.up_act(xg[a:b], w_gate_up[e], activation)
                    yg[a:b] = self.linear(h, w_down[e])
        self._ok(self.moe.krk_moe_combine(out.data_ptr(), _ptr(add), _ptr(add_gate), yg.data_ptr(), place.data_ptr(), experts.data_ptr(),
                                          offsets.data_ptr(), cap, _ptr(w_out), rows, top, C, ptr, stride,
                                          _ptr(add_input), _code(x.dtype), self._stream()), "experts' sum")
        return out

    @staticmethod
    def _use_grouped(x, K, F, C, gated, activation) -> bool:
        """Whether the experts' products of many rows run as two grouped launches (sizes and alignment)."""
        return ((not gated or activation in ("swish_clamped", "silu")) and x.dtype == torch.bfloat16 and K % 8 == 0 and F % 8 == 0 and C % 8 == 0 and min(K, F) >= 64)

    def _grouped_experts(self, x, w_first, w_down, experts, w_in, w_out, activation, act_params, add, add_gate, gated, add_input,
                         offsets, place):
        """``moe_experts`` for many rows with the experts' row counts left on the device: rows ordered by expert, the first
        product (weights of the input and the activation in its epilogue), the second, and the weighted sum."""
        rows, top = experts.shape
        E, C, F = w_down.shape
        K = x.shape[1]
        ptr, stride = self._rows_view(x)
        pairs = rows * top
        empty = lambda n: torch.empty((pairs, n), dtype=x.dtype, device=x.device)
        xg, h, yg = empty(K), empty(F), empty(C)
        # blocks of up to 256 rows: experts of more than 128 rows on the average, and blocks enough for two rounds over the
        # SMs all the same (4,096 rows of 16 experts of 512: 33 against 28 us; 12,288 of 64 of 1,408: 199 against 258 us)
        tall = lambda n, cols: int(pairs > 128 * E and E * -(-n // cols) >= 296)
        row_w = torch.empty(pairs, dtype=torch.float32, device=x.device) if w_in is not None else None  # in the rows' new order
        self._ok(self.moe.krk_moe_gather(xg.data_ptr(), ptr, stride, place.data_ptr(), experts.data_ptr(), offsets.data_ptr(), 0,
                                         rows, top, K, _ptr(w_in), _ptr(row_w), _code(x.dtype), self._stream()), "expert gather")
        self._ok(self.moe.krk_grouped_gemm(h.data_ptr(), xg.data_ptr(), w_first.data_ptr(), offsets.data_ptr(), pairs, E, F, K,
                                           _ACTIVATIONS[activation], int(gated), tall(F, 128 if gated else 256), _ptr(row_w), float(act_params[0]),
                                           float(act_params[1]), self.error.data_ptr(), self._stream()), "experts' first product")
        self._ok(self.moe.krk_grouped_gemm(yg.data_ptr(), h.data_ptr(), w_down.data_ptr(), offsets.data_ptr(), pairs, E, C, F, -1,
                                           0, tall(C, 256), None, 0.0, 0.0, self.error.data_ptr(), self._stream()), "experts' second product")
        out = torch.empty((rows, C), dtype=x.dtype, device=x.device)
        self._ok(self.moe.krk_moe_combine(out.data_ptr(), _ptr(add), _ptr(add_gate), yg.data_ptr(), place.data_ptr(),
                                          experts.data_ptr(), offsets.data_ptr(), 0, _ptr(w_out), rows, top, C, ptr, stride,
                                          _ptr(add_input), _code(x.dtype), self._stream()), "experts' sum")
        return out

    def gate_up_act(self, h, w_gate_up, intermediate, activation, act_params=None):
        """act(gate h) * (up h) with W = cat(gate, up); silu on few bfloat16 rows runs in the product's epilogue."""
        if act_params is not None:
            if activation == "swish_clamped" and act_params[1] == 1.702 and self._use_skinny(h, w_gate_up):
                # few rows: in the product's epilogue (its clamped swish has the slope 1.702 built in)
                return self._skinny(self._resolve(h), w_gate_up, w_gate_up.dtype, swiglu_rows=intermediate, gate_act=3,
                                    act_limit=act_params[0])
            return self.gated_act(self.linear(h, w_gate_up), intermediate, activation, act_params=act_params)
        if activation == "silu" and self._use_skinny(h, w_gate_up):
            return self.gate_up_swiglu(h, w_gate_up, intermediate)
        if activation == "gelu_tanh" and self._use_skinny(h, w_gate_up):  # few rows: in the product's epilogue
            return self._skinny(self._resolve(h), w_gate_up, w_gate_up.dtype, swiglu_rows=intermediate, gate_act=2)
        return self.gated_act(self.linear(h, w_gate_up), intermediate, activation)

    def rotate_norm_write(self, proj, q_col, k_col, v_col, heads, kv_heads, dim, vdim, inv_freq, rot_dims, value_eps,
                          batch, cache, value_mix=None):
        """Rotate q in place, rotate k into the cache, write v (divided by its root mean square if
        ``value_eps`` is a number) into the cache; columns are offsets into ``proj``'s rows. ``value_mix``
        (v_first rows, lambda): (1 - lambda) v + lambda v_first is what is written."""
        ptr, stride = self._rows_view(proj)
        if cache.k.dtype != proj.dtype or cache.head_dim != dim or cache.v_dim != vdim or cache.kv_heads != kv_heads:
            raise KernelError("the cache does not fit the heads it is to receive")
        mix_ptr, mix_stride, lam = None, 0, 0.0
        if value_mix is not None:
            if value_eps is not None or value_mix[0].dtype != proj.dtype or value_mix[0].shape != (proj.shape[0], kv_heads * vdim):
                raise KernelError("blended values come without a value norm, in the path's dtype, one row per row of the step")
            (mix_ptr, mix_stride), lam = self._rows_view(value_mix[0]), float(value_mix[1])
        self._ok(self.mix.krk_rotate_norm_write(
            ptr, stride, q_col, k_col, v_col, heads, kv_heads, dim, vdim, inv_freq.data_ptr(), rot_dims,
            int(value_eps is not None), float(value_eps or 0.0), batch.row_seq.data_ptr(), batch.row_pos.data_ptr(),
            batch.seq_slot.data_ptr(), cache.table.data_ptr(), cache.width, cache.k.data_ptr(), cache.v.data_ptr(),
            proj.shape[0], int(getattr(cache, "keep_pages", 0)), mix_ptr, mix_stride, lam, _code(proj.dtype),
            self._stream()), "rotation + value norm + cache write")

    def sink_attention_step(self, proj, q_col, k_col, v_col, heads, kv_heads, dim, vdim, inv_freq, rot_dims, value_eps, sink,
                            scale, window, batch, cache, out, out_col, out_scale) -> bool:
        """Rotation, value norm, cache write and attention of a single-token step as one launch (plus the merge of
        the blocks' shares). False if the step or the sizes are not of that kind: nothing was done then."""
        if not self.fuse_single_token_attention:
            return False
        if not (batch.is_decode and proj.shape[0] == batch.n_seqs) or heads // kv_heads > 8 or vdim > 128:
            return False
        return self.sink_attention(proj, q_col, heads, dim, vdim, sink, scale, window, batch, cache, out, out_col, out_scale,
                                   fuse=(k_col, v_col, inv_freq, rot_dims, value_eps))

    def sink_attention(self, proj, q_col, heads, dim, vdim, sink, scale, window, batch, cache, out, out_col, out_scale,
                       fuse=None, keep_first=0, gate=None, gate_rows=None, slopes=None, softcap=None):
        """``slopes`` (float32, one per query head) and ``softcap``: a scaled score s becomes softcap * tanh(s / softcap) -
        slope * distance, either left out where None. ``keep_first``: a windowed query also sees the sequence's first keys. ``gate`` (column, "head" or "element"):
        the result is multiplied by the sigmoid of those columns of ``gate_rows`` (default: of ``proj``)."""
        ptr, stride = self._rows_view(proj)
        optr, ostride = self._rows_view(out)
        keep_first = int(keep_first) if window else 0
        keep_pages = int(getattr(cache, "keep_pages", 0))
        g_ptr, g_stride, g_col, g_mode = None, 0, 0, 0
        if gate is not None:
            g_rows = proj if gate_rows is None else gate_rows
            if g_rows.dtype != proj.dtype or g_rows.shape[0] != proj.shape[0]:
                raise KernelError("the gate's rows have the queries' dtype and number")
            (g_ptr, g_stride), g_col, g_mode = self._rows_view(g_rows), int(gate[0]), {"head": 1, "element": 2}[gate[1]]
        if slopes is not None and (slopes.dtype != torch.float32 or slopes.numel() != heads):
            raise KernelError("the distance bias takes one float32 slope per query head")
        shape = (_ptr(slopes), float(softcap or 0.0))
        extras = (keep_first, keep_pages, g_ptr, g_stride, g_col, g_mode, *shape)
        tensor_cores = (proj.dtype == torch.bfloat16 and dim == vdim == cache.v_dim and dim % 16 == 0 and dim <= 256
                        and dim in self.attn)  # whole pages on the tensor cores, kernels compiled per head size
        if batch.is_decode and proj.shape[0] == batch.n_seqs:
            # one token per sequence: a block per (sequence, kv head), its warps splitting the window's keys. The
            # choice depends on the step's shape alone, so a sequence's results do not depend on its batch
            # blocks per (sequence, kv head) by the number of such items alone, never by lengths, so that a
            # captured step stays valid: enough to give every SM a block while items are few
            items = batch.n_seqs * cache.kv_heads
            esz = proj.element_size()
            if tensor_cores and not fuse and hasattr(self.attn[dim], "krk_sink_window_decode"):
                # bfloat16, key and value heads of one size: whole pages on the tensor cores, an item's blocks a cluster
                row_tiles = -(-(heads // cache.kv_heads) // 16)
                tiles = items * row_tiles
                pages = -(-min(int(window or 1 << 30), cache.width * 64) // 64) + 1 + -(-keep_first // 64)
                splits = 8 if tiles <= 37 else 4 if tiles <= 74 else 2 if tiles <= 192 else 1
                while splits > pages:
                    splits //= 2
                rc = self.attn[dim].krk_sink_window_decode(
                    optr + out_col * esz, ostride, float(out_scale), ptr + q_col * esz, stride, heads, cache.kv_heads, _ptr(sink),
                    batch.seq_slot.data_ptr(), batch.seq_start.data_ptr(), cache.table.data_ptr(), cache.width, cache.k.data_ptr(),
                    cache.v.data_ptr(), batch.n_seqs, float(scale), int(window or 0), keep_first, keep_pages,
                    None if g_ptr is None else g_ptr + g_col * esz, g_stride, g_mode, *shape, splits, self._stream())
                if rc != -2:  # -2: odd strides or offsets, or too large for it; the kernel below takes them
                    self._ok(rc, "tensor-core single-token windowed attention")
                    return True
            splits = 8 if items <= 18 else 4 if items <= 37 else 2 if items <= 74 else 1
            key = ("sink", batch.n_seqs, heads, vdim, splits)
            scratch = self._partials.get(key)
            if scratch is None and splits > 1:
                scratch = self._partials[key] = torch.empty(batch.n_seqs * heads * splits * (vdim + 2),
                                                            dtype=torch.float32, device=self.device)
            rc = self.mix.krk_sink_attention_single(
                optr, ostride, out_col, float(out_scale), ptr, stride, q_col, heads, cache.kv_heads, dim, vdim,
                _ptr(sink), batch.seq_slot.data_ptr(), batch.seq_start.data_ptr(), cache.table.data_ptr(), cache.width,
                cache.k.data_ptr(), cache.v.data_ptr(), cache.v_dim, batch.n_seqs, float(scale), int(window or 0), splits,
                _ptr(scratch), *((1, fuse[0], fuse[1], fuse[2].data_ptr(), fuse[3], int(fuse[4] is not None),
                                  float(fuse[4] or 0.0)) if fuse else (0, 0, 0, None, 0, 0, 0.0)),
                *extras, _code(proj.dtype), self._stream())
            if rc != -2:  # -2: heads too large for it; the general kernel takes them
                self._ok(rc, "single-token windowed attention with a sink")
                return True
            if fuse:
                return False
        elif fuse:
            return False
        if tensor_cores and not batch.is_decode and hasattr(self.attn[dim], "krk_sink_window_prefill"):
            # many tokens per sequence: the tensor-core walk over whole pages
            esz = proj.element_size()
            rc = self.attn[dim].krk_sink_window_prefill(
                optr + out_col * esz, ostride, float(out_scale), ptr + q_col * esz, stride, heads, cache.kv_heads,
                _ptr(sink), batch.seq_slot.data_ptr(), batch.seq_start.data_ptr(), batch.seq_qlen.data_ptr(),
                batch.cu_q.data_ptr(), cache.table.data_ptr(), cache.width, cache.k.data_ptr(), cache.v.data_ptr(),
                batch.n_seqs, batch.max_q_len, float(scale), int(window or 0), keep_first, keep_pages,
                None if g_ptr is None else g_ptr + g_col * esz, g_stride, g_mode, *shape, self._stream())
            if rc != -2:  # -2: odd strides or offsets; the general kernel takes them
                self._ok(rc, "tensor-core windowed attention with a sink")
                return
        self._ok(self.mix.krk_sink_attention(
            optr, ostride, out_col, float(out_scale), ptr, stride, q_col, heads, cache.kv_heads, dim, vdim, _ptr(sink),
            batch.row_seq.data_ptr(), batch.row_pos.data_ptr(), batch.seq_slot.data_ptr(), cache.table.data_ptr(),
            cache.width, cache.k.data_ptr(), cache.v.data_ptr(), cache.v_dim, proj.shape[0], float(scale), int(window or 0),
            *extras, _code(proj.dtype), self._stream()), "windowed attention with a sink")

    # -- pair-hash embedding, per-head norms with pair rotation, mixed head scores over blocks of keys ------------
    def embed_bigram(self, table, pairs, state, buckets, mul_prev, mul_cur, batch):
        """float32 rows table[id] + pairs[(id_prev * mul_prev + id * mul_cur) % buckets] (row ``buckets`` at position 0);
        ``state`` int32 [slots, 1] holds every sequence's last token and is brought up to date."""
        if state.dtype != torch.int32 or not state.is_contiguous() or pairs.dtype != table.dtype or pairs.shape[0] != buckets + 1:
            raise KernelError("the pair embedding keeps one int32 per slot and a second table of buckets + 1 rows")
        rows = batch.n_rows
        out = torch.empty((rows, table.shape[1]), dtype=torch.float32, device=table.device)
        self._ok(self.mix.krk_embed_bigram(out.data_ptr(), table.data_ptr(), pairs.data_ptr(), batch.tokens.data_ptr(),
                                           state.data_ptr(), rows, table.shape[1], table.shape[0], int(buckets), int(mul_prev),
                                           int(mul_cur), batch.row_seq.data_ptr(), batch.row_pos.data_ptr(),
                                           batch.cu_q.data_ptr(), batch.seq_slot.data_ptr(), self.error.data_ptr(),
                                           _code(table.dtype), self._stream()), "pair-hash embedding")
        return out

    def bias_norm_rotate_write(self, proj, q_col, k_col, v_col, heads, kv_heads, dim, vdim, bias, qk_gain, eps, inv_freq,
                               rot_dims, pairs, batch, cache, unit=False, temperature=None):
        """On a stacked q | k | v product: float32 ``bias`` over all three (None: none); with ``qk_gain`` (float32, the q
        weight then the k weight, ``dim`` each) every q and k head is divided by its root mean square and multiplied by
        it (``unit``: divided only); ``temperature`` (coef, every): a q head at position p is multiplied by
        1 + coef * ln(floor((p + 1) / every) + 1); the first ``rot_dims`` elements are rotated (``pairs``: 2i with 2i + 1, else i with i + rot_dims/2); q in
        place, k and v into their pages."""
        ptr, stride = self._rows_view(proj)
        if cache.k.dtype != proj.dtype or cache.head_dim != dim or cache.v_dim != vdim or cache.kv_heads != kv_heads:
            raise KernelError("the cache does not fit the heads it is to receive")
        n = (heads + kv_heads) * dim + kv_heads * vdim
        if (bias is not None and (bias.numel() != n or bias.dtype != torch.float32)) or (
                qk_gain is not None and (qk_gain.numel() != 2 * dim or qk_gain.dtype != torch.float32)):
            raise KernelError("float32 biases cover q, k and v; the float32 gains are one head's q weight and k weight")
        self._ok(self.mix.krk_bias_norm_rotate_write(
            ptr, stride, q_col, k_col, v_col, heads, kv_heads, dim, vdim, _ptr(bias), _ptr(qk_gain), float(eps), int(unit),
            float(temperature[0]) if temperature else 0.0, int(temperature[1]) if temperature else 0, inv_freq.data_ptr(), int(rot_dims), int(bool(pairs)), batch.row_seq.data_ptr(), batch.row_pos.data_ptr(),
            batch.seq_slot.data_ptr(), cache.table.data_ptr(), cache.width, cache.k.data_ptr(), cache.v.data_ptr(),
            proj.shape[0], int(getattr(cache, "keep_pages", 0)), _code(proj.dtype), self._stream()),
            "biases + head norms + rotation + cache write")

    # bytes up to which a prompt step's tiles leave shares to be merged (measured: 51 MB of shares at 12 heads gain
    # 12 % of the attention's time, 136 MB at 32 heads lose 30 %)
    MIXED_PREFILL_SCRATCH = 64 << 20
    MIXED_SPLITS_MAX = 32  # blocks that share one sequence's keys in a single-token step

    def mixed_attention(self, proj, q_col, heads, dim, vdim, sink, talk, scale, chunk, batch, cache, out, out_col, out_scale,
                        gate=None):
        """Attention over the keys of the query's own block of ``chunk`` positions (None: all earlier keys), the heads'
        scores mixed by ``talk`` [heads, heads] before the softmax (None: not mixed), ``sink`` as in ``sink_attention``,
        ``gate`` (column, "head"). Up to 32 heads, value heads up to 256."""
        ptr, stride = self._rows_view(proj)
        optr, ostride = self._rows_view(out)
        g_col, g_mode = (int(gate[0]), 1) if gate is not None else (0, 0)
        if gate is not None and gate[1] != "head":
            raise KernelError("this attention takes a gate per head only")
        if getattr(cache, "keep_pages", 0) or cache.window:
            raise KernelError("this attention reads a cache that keeps every key")
        if talk is not None and (talk.dtype != torch.float32 or talk.shape != (heads, heads) or not talk.is_contiguous()):
            raise KernelError("the heads' mixing matrix is float32 [heads, heads]")
        chunk = int(chunk or 0)
        if batch.is_decode and proj.shape[0] == batch.n_seqs:
            # by the step's shape alone, never by lengths, so that a captured step stays valid
            most = -(-chunk // 32) if chunk else self.MIXED_SPLITS_MAX
            splits = max(1, min(self.MIXED_SPLITS_MAX, most, 148 // batch.n_seqs))
            key = ("mixed", batch.n_seqs, heads, vdim, splits)
            scratch = self._partials.get(key)
            if scratch is None:
                scratch = self._partials[key] = torch.empty(batch.n_seqs * heads * splits * (vdim + 2), dtype=torch.float32,
                                                            device=self.device)
            self._ok(self.mix.krk_mixed_attention_single(
                optr, ostride, out_col, float(out_scale), ptr, stride, q_col, heads, cache.kv_heads, dim, vdim, _ptr(sink),
                _ptr(talk), batch.seq_slot.data_ptr(), batch.seq_start.data_ptr(), cache.table.data_ptr(), cache.width,
                cache.k.data_ptr(), cache.v.data_ptr(), batch.n_seqs, float(scale), chunk, splits, scratch.data_ptr(),
                ptr, stride, g_col, g_mode, _code(proj.dtype), self._stream()), "single-token attention with mixed scores")
            self.launches += 1
            return
        if (proj.dtype == torch.bfloat16 and dim == vdim and dim in self.attn and hasattr(self.attn[dim], "krk_mixed_prefill")):
            # many tokens per sequence in bfloat16: scores and P.V on the tensor cores (compiled per head size)
            esz = proj.element_size()
            # Few tiles of unequal length (one prompt of a few thousand tokens: a tile sees 1 to chunk / 64 pages) leave
            # SMs idle while the longest runs: then every tile's pages are dealt out over 2 or 4 blocks and a merge
            # kernel adds their shares. By the step's shape; a step of many tokens is never replayed from a graph.
            rows = proj.shape[0]
            tiles = -(-batch.max_q_len // 16) * batch.n_seqs
            pages = -(-min(chunk or batch.max_kv_len, batch.max_kv_len) // 64)
            splits = 1 if tiles >= 592 or pages < 4 else (2 if tiles >= 296 else 4)
            splits = min(splits, pages)
            part = None
            while splits > 1 and rows * heads * splits * (dim + 2) * 4 > self.MIXED_PREFILL_SCRATCH:
                splits //= 2  # the shares are written and read once: beyond this size that costs more than it gains
            if splits > 1:
                need = rows * heads * splits * (dim + 2)
                part = self._partials.get("mixed_prefill")
                if part is None or part.numel() < need:
                    part = self._partials["mixed_prefill"] = torch.empty(need, dtype=torch.float32, device=self.device)
            rc = self.attn[dim].krk_mixed_prefill(
                optr + out_col * esz, ostride, float(out_scale), ptr + q_col * esz, stride, heads, cache.kv_heads, _ptr(sink),
                _ptr(talk), batch.seq_slot.data_ptr(), batch.seq_start.data_ptr(), batch.seq_qlen.data_ptr(),
                batch.cu_q.data_ptr(), cache.table.data_ptr(), cache.width, cache.k.data_ptr(), cache.v.data_ptr(),
                batch.n_seqs, batch.max_q_len, float(scale), chunk, ptr + g_col * esz, stride, g_mode, self._stream(),
                splits, _ptr(part))
            if rc != -2:  # -2: a shape it does not take; the general kernel does
                self._ok(rc, "tensor-core attention with mixed scores")
                if splits > 1:
                    self._ok(self.mix.krk_mixed_attention_merge(optr, ostride, out_col, float(out_scale), part.data_ptr(), heads,
                                                               vdim, splits, rows, ptr, stride, g_col, g_mode,
                                                               _code(proj.dtype), self._stream()),
                             "merge of a prompt's key splits")
                return
        self._ok(self.mix.krk_mixed_attention(
            optr, ostride, out_col, float(out_scale), ptr, stride, q_col, heads, cache.kv_heads, dim, vdim, _ptr(sink),
            _ptr(talk), batch.row_seq.data_ptr(), batch.row_pos.data_ptr(), batch.seq_slot.data_ptr(),
            cache.table.data_ptr(), cache.width, cache.k.data_ptr(), cache.v.data_ptr(), proj.shape[0], float(scale), chunk,
            ptr, stride, g_col, g_mode, _code(proj.dtype), self._stream()), "attention with mixed scores")

    def norm_sum(self, outs, gains, eps, scale):
        """scale * sum_b rmsnorm(outs[b]) * gains[b]: up to four [rows, C] inputs of the path's dtype, float32 gains [n, C]."""
        first = outs[0]
        n = len(outs)
        if any(o.shape != first.shape or o.dtype != first.dtype or not o.is_contiguous() for o in outs) or (
                gains.dtype != torch.float32 or gains.shape != (n, first.shape[1]) or not gains.is_contiguous()):
            raise KernelError("the summed norms read contiguous rows of one shape and dtype and float32 gains [n, C]")
        out = torch.empty_like(first)
        ptrs = [o.data_ptr() for o in outs] + [None] * (4 - n)
        self._ok(self.mix.krk_norm_sum(out.data_ptr(), *ptrs, n, gains.data_ptr(), first.shape[0], first.shape[1], float(eps),
                                       float(scale), _code(first.dtype), self._stream()), "norms of several outputs, summed")
        return out

    def act_rows(self, z, activation, params=(0.0, 0.0)):
        """An activation without a gate over [rows, I]; "xielu" takes (softplus(p), 1/2 + softplus(q))."""
        ptr, stride = self._rows_view(z)
        out = torch.empty(z.shape, dtype=z.dtype, device=z.device)
        self._ok(self.mix.krk_act_rows(out.data_ptr(), ptr, stride, z.shape[0], z.shape[1], _ACTIVATIONS[activation],
                                       float(params[0]), float(params[1]), _code(z.dtype), self._stream()), "activation")
        return out

    def token_shift(self, h, last_state, mu, batch, store=False):
        """[mixes, rows, hidden]: h + (h_prev - h) * mu, the row before a step's first coming from ``last_state``;
        with ``store`` every sequence's last row of the step then takes its place there."""
        if last_state.dtype != torch.float32 or not last_state.is_contiguous() or mu.dtype != torch.float32:
            raise KernelError("the token shift keeps a contiguous float32 row per slot and reads float32 blend weights")
        ptr, stride = self._rows_view(h)
        rows, C = h.shape
        out = torch.empty((mu.shape[0], rows, C), dtype=h.dtype, device=h.device)
        self._ok(self.scan.krk_token_shift(out.data_ptr(), ptr, stride, last_state.data_ptr(), mu.data_ptr(), mu.shape[0],
                                          C, rows, batch.row_seq.data_ptr(), batch.cu_q.data_ptr(),
                                          batch.seq_slot.data_ptr(), _code(h.dtype), self._stream(), int(store)), "token shift")
        return out

    def linear_recurrence(self, kind, r, k, v, gate, lora, w2, w0, heads, dim, norm_w, eps, state, batch, out, out_col,
                          out_scale, rate=None, rate_bias=None, decay_scale=1.0, bonus=None, last_rows=None):
        """The scan of a matrix-state mixer over a step's rows ("wkv" or "delta"); see csrc/recurrent.cu."""
        views = [self._rows_view(t) for t in (r, k, v, gate)]
        rate_v = self._rows_view(rate) if rate is not None else (None, 0)
        lora_v = self._rows_view(lora)
        optr, ostride = self._rows_view(out)
        last_ptr, last_stride, C, last_state = None, 0, 0, None
        if last_rows is not None:
            (last_ptr, last_stride), C, last_state = self._rows_view(last_rows[0]), last_rows[0].shape[1], last_rows[1]
        if state.dtype != torch.float32 or not state.is_contiguous() or not w2.is_contiguous() or w2.dtype != r.dtype:
            raise KernelError("the recurrence keeps a contiguous float32 state and reads W2 in the path's dtype")
        rows = r.shape[0]
        prep = o_raw = None
        if not batch.is_decode and dim % 4 == 0 and self.split_recurrence:
            # steps of many tokens: decays and gates over all rows at once, the scan between them (float32 scratch)
            prep = torch.empty(rows * heads * 6 * dim, dtype=torch.float32, device=r.device)
            o_raw = torch.empty(rows * heads * dim, dtype=torch.float32, device=r.device)
        rc = self.scan.krk_linear_recurrence(
            {"wkv": 0, "delta": 1}[kind], views[0][0], views[0][1], views[1][0], views[1][1], views[2][0], views[2][1],
            views[3][0], views[3][1], rate_v[0], rate_v[1], lora_v[0], lora_v[1], w2.data_ptr(), w0.data_ptr(),
            _ptr(rate_bias), _ptr(bonus), norm_w.data_ptr(), state.data_ptr(), last_ptr, last_stride, C,
            _ptr(last_state), optr, ostride, out_col, float(out_scale), float(eps), float(decay_scale), heads, dim,
            lora.shape[1], batch.n_seqs, batch.cu_q.data_ptr(), batch.seq_qlen.data_ptr(), batch.seq_slot.data_ptr(),
            rows, _ptr(prep), _ptr(o_raw), _code(r.dtype), self._stream())
        self._ok(rc, f"{kind} recurrence (heads of up to 256 channels)")

    # -- matrix states without a removal term -------------------------------------------------
    MEMORY_CHUNK_MIN = 128  # tokens of a step's longest sequence from which a bfloat16 scan runs in chunks

    def _memory_chunk(self, views, dtype, dim, vdim, gated, batch) -> int:
        """Tokens per chunk where a step's scan runs in chunks on the tensor cores, else 0."""
        if batch.is_decode or dtype != torch.bfloat16 or batch.max_q_len < self.MEMORY_CHUNK_MIN or any(
                p % 16 or s % 8 for p, s in views[:3]):
            return 0
        return int(self.memory.krk_memory_chunk_tokens(dim, vdim, int(gated)))

    def _memory_step(self, views, z, w2, bias, constant, heads, dim, vdim, norm_w, eps, state, nm, batch, rows, dtype, out,
                     out_col, out_scale) -> bool:
        """A single-token step as one launch; False where the step or the sizes are not of that kind."""
        if not batch.is_decode or rows != batch.n_seqs or vdim > 1024 or (vdim % 4 and vdim > 256):
            return False
        self._check_memory_state(state, nm, heads, dim, vdim)
        optr, ostride = self._rows_view(out)
        # blocks per (sequence, head) by the number of such items alone, so that a captured step stays valid
        items = batch.n_seqs * heads
        split = 8 if items <= 18 else 4 if items <= 37 else 2 if items <= 74 else 1
        while split > 1 and vdim < 16 * split:
            split //= 2
        self._ok(self.memory.krk_memory_step(optr, ostride, int(out_col), float(out_scale), *views[0], *views[1], *views[2],
                                             *views[3], float(dim) ** -0.5, *z, _ptr(w2), bias.data_ptr(), float(constant),
                                             0 if w2 is None else w2.shape[1], state.data_ptr(), _ptr(nm), norm_w.data_ptr(),
                                             float(eps), heads, dim, vdim, batch.n_seqs, split, batch.seq_slot.data_ptr(),
                                             _code(dtype), self._stream()), "single-token matrix-state step")
        return True

    @staticmethod
    def _check_memory_state(state, nm, heads, dim, vdim) -> None:
        if state.dtype != torch.float32 or not state.is_contiguous() or state.shape[1:] != (heads, dim, vdim):
            raise KernelError("the scan keeps a contiguous float32 state [slots, heads, dim, vdim]")
        if nm is not None and (nm.dtype != torch.float32 or not nm.is_contiguous() or nm.shape[1:] != (heads, dim + 1)):
            raise KernelError("the gated scan keeps a contiguous float32 [slots, heads, dim + 1] beside its state")

    def _memory_scan(self, views, chunk, dtype, decays, gates, heads, dim, vdim, norm_w, eps, state, nm, batch, rows, out,
                     out_col, out_scale):
        optr, ostride = self._rows_view(out)
        self._check_memory_state(state, nm, heads, dim, vdim)
        gated = nm is not None
        y = torch.empty((rows, heads * vdim), dtype=torch.float32, device=self.device)
        den = torch.empty((rows, heads), dtype=torch.float32, device=self.device) if gated else None
        tables = (batch.cu_q.data_ptr(), batch.seq_qlen.data_ptr(), batch.seq_slot.data_ptr())
        if chunk:
            chunks = batch.n_seqs * -(-batch.max_q_len // chunk) * heads
            cs = torch.empty((chunks, dim * (vdim + int(gated))), dtype=torch.float32, device=self.device)
            cd = torch.empty((chunks, dim), dtype=torch.float32, device=self.device)
            self._ok(self.memory.krk_memory_chunks(y.data_ptr(), _ptr(den), *views[0], *views[1], *views[2], float(dim) ** -0.5, _ptr(decays),
                                                   _ptr(gates), state.data_ptr(), _ptr(nm), cs.data_ptr(), cd.data_ptr(), heads,
                                                   dim, vdim, batch.n_seqs, batch.max_q_len, *tables, self._stream()),
                     "matrix-state scan in chunks")
            self.launches += 2
        else:
            self._ok(self.memory.krk_memory_scan(y.data_ptr(), _ptr(den), *views[0], *views[1], *views[2], float(dim) ** -0.5, _ptr(decays),
                                                 _ptr(gates), state.data_ptr(), _ptr(nm), heads, dim, vdim, batch.n_seqs, *tables,
                                                 _code(dtype), self._stream()),
                     "matrix-state scan (up to 1,024 key channels a head)")
        self._ok(self.memory.krk_memory_finish(optr, ostride, int(out_col), float(out_scale), y.data_ptr(), _ptr(den), _ptr(gates), *views[3],
                                               norm_w.data_ptr(), heads, vdim, float(eps), rows, _code(dtype), self._stream()),
                 "matrix-state head norm and gate")

    def gla_scan(self, q, k, v, gate, lora, w2, bias, tau, heads, dim, vdim, norm_w, eps, state, batch, out, out_col, out_scale):
        """Gated linear attention over a step's rows, from and to ``state`` [slots, heads, dim, vdim]; see
        csrc/matrix_memory.cu. ``norm_w`` [vdim]."""
        views = [self._rows_view(t) for t in (q, k, v, gate)]
        lptr, lstride = self._rows_view(lora)
        rows, R = lora.shape
        if w2.dtype != q.dtype or not w2.is_contiguous() or bias.dtype != torch.float32:
            raise KernelError("the decays read their second matrix in the path's dtype and a float32 bias")
        if self._memory_step(views, (lptr, lstride), w2, bias, tau, heads, dim, vdim, norm_w, eps, state, None, batch, rows,
                             q.dtype, out, out_col, out_scale):
            return
        chunk = self._memory_chunk(views, q.dtype, dim, vdim, False, batch) if R <= 192 else 0  # a chunk's rows in shared memory
        decays = torch.empty((rows, heads * dim), dtype=torch.float32, device=q.device)
        if chunk:
            self._ok(self.memory.krk_memory_chunk_decays(decays.data_ptr(), lptr, lstride, w2.data_ptr(), bias.data_ptr(),
                                                         float(tau), heads * dim, R, batch.n_seqs, batch.max_q_len,
                                                         batch.cu_q.data_ptr(), batch.seq_qlen.data_ptr(), self._stream()),
                     "log decays summed within chunks")
        else:
            self._ok(self.memory.krk_memory_decays(decays.data_ptr(), lptr, lstride, w2.data_ptr(), bias.data_ptr(), float(tau),
                                                   rows, heads * dim, R, _code(q.dtype), self._stream()), "log decays")
        self._memory_scan(views, chunk, q.dtype, decays, None, heads, dim, vdim, norm_w, eps, state, None, batch, rows, out,
                          out_col, out_scale)

    def mlstm_scan(self, q, k, v, gate, if_rows, if_bias, cap, heads, dim, vdim, norm_w, eps, state, nm, batch, out, out_col,
                   out_scale):
        """The matrix LSTM over a step's rows; ``if_rows`` [rows, 2 * heads]: input then forget gates before bias and cap;
        ``nm`` [slots, heads, dim + 1]: the vector beside the matrix and the running maximum. ``norm_w`` [heads * vdim]."""
        views = [self._rows_view(t) for t in (q, k, v, gate)]
        zptr, zstride = self._rows_view(if_rows)
        rows = q.shape[0]
        if self._memory_step(views, (zptr, zstride), None, if_bias, cap, heads, dim, vdim, norm_w, eps, state, nm, batch, rows,
                             q.dtype, out, out_col, out_scale):
            return
        gates = torch.empty((rows, heads, 4), dtype=torch.float32, device=q.device)
        self._ok(self.memory.krk_memory_gates(gates.data_ptr(), zptr, zstride, if_bias.data_ptr(), float(cap), nm.data_ptr(), heads,
                                              dim, batch.n_seqs, batch.max_q_len, batch.cu_q.data_ptr(), batch.seq_qlen.data_ptr(),
                                              batch.seq_slot.data_ptr(), _code(q.dtype), self._stream()), "matrix LSTM gates")
        chunk = self._memory_chunk(views, q.dtype, dim, vdim, True, batch)
        self._memory_scan(views, chunk, q.dtype, None, gates, heads, dim, vdim, norm_w, eps, state, nm, batch, rows, out, out_col,
                          out_scale)

    # -- state-space mixer ------------------------------------------------------------------
    SSD_CHUNK = 128  # tokens per chunk where one sequence's step is long enough to be scanned in chunks

    def causal_conv_silu(self, x, w, b, tail, batch):
        """silu(b + short causal convolution over each sequence's rows); ``tail`` [slots, taps - 1, channels] holds
        every sequence's last inputs and is brought up to date. x may be a column slice; w [taps, channels] float32."""
        ptr, stride = self._rows_view(x)
        rows, ch = x.shape
        taps = w.shape[0]
        if w.shape[1] != ch or not w.is_contiguous():
            raise KernelError("the convolution's weights come tap-major, [taps, channels], contiguous")
        if tail.dtype != x.dtype or not tail.is_contiguous() or tail.shape[1:] != (max(taps - 1, 1), ch):
            raise KernelError("the convolution's stored inputs have the path's dtype and [taps - 1, channels] per slot")
        out = torch.empty((rows, ch), dtype=x.dtype, device=x.device)
        self._ok(self.scan.krk_causal_conv_silu(out.data_ptr(), ptr, stride, w.data_ptr(), b.data_ptr(), tail.data_ptr(),
                                               taps, ch, rows, batch.n_seqs, batch.row_seq.data_ptr(),
                                               batch.cu_q.data_ptr(), batch.seq_qlen.data_ptr(), batch.seq_slot.data_ptr(),
                                               _code(x.dtype), self._stream()), "causal convolution + silu")
        self.launches += int(taps > 1)
        return out

    def ssd_scan(self, x, B, C, dt, dt_bias, a_log, skip, heads, P, N, groups, state, batch):
        """The scan of a state-space mixer over a step's rows (csrc/ssd.cu): float32 y [rows, heads * P]; ``state``
        [slots, heads, N, P] float32 is read and left as the sequences' new state."""
        views = [self._rows_view(t) for t in (x, B, C, dt)]
        rows = x.shape[0]
        if state.dtype != torch.float32 or not state.is_contiguous() or state.shape[1:] != (heads, N, P):
            raise KernelError("the scan keeps a contiguous float32 state [slots, heads, N, P]")
        y = torch.empty((rows, heads * P), dtype=torch.float32, device=x.device)
        chunk, cs, cd = 0, None, None
        if not batch.is_decode and batch.max_q_len >= 2 * self.SSD_CHUNK:
            chunk = self.SSD_CHUNK
            n_chunks = -(-batch.max_q_len // chunk)
            cs = torch.empty((batch.n_seqs * n_chunks * heads, N * P), dtype=torch.float32, device=x.device)
            cd = torch.empty(batch.n_seqs * n_chunks * heads, dtype=torch.float32, device=x.device)
            self.launches += 2
        self._ok(self.scan.krk_ssd_scan(y.data_ptr(), views[0][0], views[0][1], views[1][0], views[1][1], views[2][0],
                                        views[2][1], views[3][0], views[3][1], dt_bias.data_ptr(), a_log.data_ptr(),
                                        skip.data_ptr(), state.data_ptr(), heads, P, N, groups, batch.n_seqs,
                                        batch.max_q_len, batch.cu_q.data_ptr(), batch.seq_qlen.data_ptr(),
                                        batch.seq_slot.data_ptr(), chunk, _ptr(cs), _ptr(cd), _code(x.dtype),
                                        self._stream()), "state-space scan (a head's state must fit a block's registers)")
        return y

    def gated_group_norm(self, y, gate_rows, weight, parts, eps, out, out_col, out_scale):
        """out[:, out_col:...] = group_norm(y * silu(gate_rows)) * weight * out_scale; y float32, ``parts`` equal parts
        each divided by its own root mean square."""
        zptr, zstride = self._rows_view(gate_rows)
        optr, ostride = self._rows_view(out)
        rows, inner = y.shape
        if y.dtype != torch.float32 or not y.is_contiguous() or gate_rows.dtype != out.dtype:
            raise KernelError("the gated norm reads float32 rows and a gate of the path's dtype")
        self._ok(self.scan.krk_gated_group_norm(optr, ostride, int(out_col), float(out_scale), y.data_ptr(), zptr, zstride,
                                               weight.data_ptr(), rows, inner, int(parts), float(eps), _code(out.dtype),
                                               self._stream()), "gated group norm")

    # -- token selection ------------------------------------------------------------
    def select_tokens(self, logits, temperature, seed, requests, step, feed=None, out=None):
        """One token per row. ``feed``: the batch description of a single-token step; the
        kernel then also writes the chosen tokens into it and moves its positions on by
        one, so that the next step can run without the host."""
        n, vocab = logits.shape
        tokens = out if out is not None else torch.empty(n, dtype=torch.int32, device=logits.device)
        logits = logits.contiguous()
        f = (None, None, None) if feed is None else (feed.tokens.data_ptr(), feed.row_pos.data_ptr(),
                                                     feed.seq_start.data_ptr())
        if self._select_scratch is None or self._select_scratch.numel() < n:
            self._select_scratch = torch.zeros(max(n, 256), dtype=torch.int64, device=self.device)
        self._ok(self.core.krk_select_tokens(tokens.data_ptr(), logits.data_ptr(), n, vocab, temperature,
                                             seed & 0xFFFFFFFF, requests.data_ptr(), step & 0xFFFFFFFF, *f,
                                             self._select_scratch.data_ptr(), self._stream()), "token selection")
        return tokens


_cached: dict = {}


def load_kernels(head_dims=(), device="cuda:0") -> Kernels:
    """The process-wide Kernels object of a device, with the given head sizes loaded."""
    key = str(torch.device(device))
    k = _cached.get(key)
    if k is None:
        k = _cached[key] = Kernels(head_dims, device)
    for d in head_dims:
        k._attn_lib(int(d))
    return k
