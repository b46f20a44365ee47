"""Kernel-backed op set (sm_100a).  Every method launches hand-written kernels from ``libblaze_kernels.so``
through its C ABI; nothing here falls back to the PyTorch oracle.

The op boundaries are those of the reference's forward pass (``crates/blaze/src/model.rs:2330-2551``), fused
differently: norm → (quantised) activation handed straight to the next GEMM, RoPE + q/k norm + FP8 page write in
one kernel, one attention kernel for prefill / decode / verify rows.
"""
from __future__ import annotations

import os

import ctypes
from typing import Dict, Optional, Tuple

import torch

from .. import quant
from .._native import kernels
from ..linear import Linear, QuantAct
from ..quant import Format

_c = ctypes
VP = ctypes.c_void_p


class CudaError(RuntimeError):
    pass


def _ptr(t: Optional[torch.Tensor]) -> VP:
    return VP(0) if t is None else VP(t.data_ptr())


class _Symbols:
    """Entry points of a kernel library for declaring their types; those the library does not have are ignored here (calling one
    raises)."""

    class _Missing:
        restype = argtypes = None

    def __init__(self, lib):
        self._lib = lib

    def __getattr__(self, name):
        try:
            return getattr(self._lib, name)
        except AttributeError:
            return self._Missing()


class RoutedRows:
    """What routed experts leave behind: ``rows`` in the padded row space, the ``row_map [T, k]`` of each token's rows with their
    ``weights`` (None: the rows count as they are), and rows that are added to the sums (``extra``, may be None; times the sigmoid of
    ``gate``, logits ``[T]``, where there is one)."""

    def __init__(self, rows, row_map, weights, extra, gate=None):
        self.rows, self.row_map, self.weights, self.extra, self.gate = rows, row_map, weights, extra, gate


class CudaOps:
    is_cuda = True
    name = "sm100a"

    def __init__(self, device, sources=None):
        self.device = torch.device(device)
        self.lib = kernels(sources)
        self.launches = 0
        self._held_stream = None
        self._held_depth = 0
        self.attn_prof = None      # optional int64 [8*3*16] wait-cycle counters of the decode attention kernel
        self._scratch: Dict[str, torch.Tensor] = {}
        self._retired: list = []
        self._sm = torch.cuda.get_device_properties(self.device).multi_processor_count
        lib = _Symbols(self.lib)           # a library of one model family has some of the entry points only
        lib.blz_gemm_tc.restype = _c.c_int
        lib.blz_gemm_tc.argtypes = [_c.c_int, VP, _c.c_longlong, VP, _c.c_longlong, VP, _c.c_longlong, _c.c_int, _c.c_int,
                                    _c.c_int, VP, VP, VP, VP, VP, _c.c_int, _c.c_int, _c.c_int, VP, _c.c_int, _c.c_int, _c.c_int, _c.c_float, VP]
        lib.blz_gemm_wait_flags.restype = _c.c_int
        lib.blz_gemm_wait_flags.argtypes = [VP, VP, _c.c_int, _c.c_int]
        lib.blz_gemm_argmax_parts.argtypes = [VP, VP]
        lib.blz_argmax_parts.argtypes = [VP, VP, _c.c_int, _c.c_int, VP, VP, _c.c_int, VP]
        lib.blz_gemm_wide.restype = _c.c_int
        lib.blz_gemm_wide.argtypes = [_c.c_int, VP, _c.c_longlong, VP, _c.c_longlong, VP, _c.c_longlong, _c.c_int, _c.c_int,
                                      _c.c_int, VP, VP, VP, VP, VP, _c.c_int, _c.c_int, _c.c_int, VP, _c.c_longlong, VP,
                                      _c.c_int, _c.c_int, _c.c_int, _c.c_float, VP]
        lib.blz_gemm_sk.restype = _c.c_int
        lib.blz_gemm_sk.argtypes = [_c.c_int, VP, _c.c_longlong, VP, _c.c_longlong, VP, _c.c_longlong, _c.c_int, _c.c_int,
                                    _c.c_int, VP, VP, VP, VP, VP, _c.c_int, _c.c_int, _c.c_float, VP]
        lib.blz_gemm_fp8_block.restype = _c.c_int
        lib.blz_gemm_fp8_block.argtypes = [VP, _c.c_longlong, VP, _c.c_longlong, VP, _c.c_longlong, _c.c_int, _c.c_int, _c.c_int,
                                           VP, _c.c_longlong, VP, VP, _c.c_int, VP]
        lib.blz_quant_fp8_block.restype = _c.c_int
        lib.blz_quant_fp8_block.argtypes = [VP, _c.c_longlong, VP, VP, _c.c_longlong, _c.c_int, _c.c_int, VP]
        # FP8 checkpoints with 128x128 fp32 block scales: "exact" keeps the stored codes and scales and promotes every K block
        # in fp32 (blz_gemm_fp8_block); "mx" re-quantises the weight once to e4m3 with e8m0 scales per 32 elements and runs the
        # hardware block-scaled MMA (faster, but only exact when the stored scales are powers of two)
        self._fp8_block_exact = os.environ.get("BLAZE_FP8_BLOCK", "exact") != "mx"
        lib.blz_gemm_sk_default_ks.restype = _c.c_int
        lib.blz_gemm_sk_default_ks.argtypes = [_c.c_int] * 4
        # decode-sized GEMMs (few output tiles) take the cluster split-K kernel; BLAZE_GEMM_SK=0 keeps them on the
        # one-CTA-per-tile kernel (A/B timing)
        self._sk_ok = os.environ.get("BLAZE_GEMM_SK", "1") != "0"
        self.SK_MAX_ROWS = 512
        self.tuning = None         # optional tune.Tuning: per-shape kernel choices measured on this device
        lib.blz_gemm_wide_ksplit.restype = _c.c_int
        lib.blz_gemm_wide_ksplit.argtypes = [_c.c_int, _c.c_int, _c.c_int]
        self._wide_ok = os.environ.get("BLAZE_GEMM_WIDE", "1") != "0"
        # tile-major weight storage measured no faster than row-major on B200 and keeps a second copy of the weights: opt-in
        self._tiled_ok = os.environ.get("BLAZE_TILED_WEIGHTS", "0") == "1"
        self._wide_ws = self._wide_ctr = None
        lib.blz_embed.argtypes = [VP, VP, VP, _c.c_int, _c.c_int, _c.c_int, VP]
        lib.blz_rmsnorm.argtypes = [VP, VP, VP, VP, VP, VP, VP, _c.c_int, _c.c_int, _c.c_float, _c.c_int, _c.c_int, _c.c_int, VP]
        lib.blz_swiglu.argtypes = [VP, VP, VP, VP, VP, _c.c_int, _c.c_int, _c.c_int, _c.c_int, VP]
        lib.blz_attn_prep.argtypes = [VP, VP, VP, VP, VP, VP, VP, VP, VP, _c.c_int, _c.c_int, _c.c_int, _c.c_int, _c.c_int,
                                      _c.c_float, _c.c_float, _c.c_int, _c.c_int, _c.c_float, _c.c_float, _c.c_longlong,
                                      _c.c_longlong, _c.c_int, _c.c_longlong, _c.c_int, _c.c_int, VP]
        lib.blz_attn_tc.argtypes = [VP, VP, VP, VP, VP, VP, VP, VP, VP, _c.c_int, _c.c_int, _c.c_int, _c.c_int, _c.c_int,
                                    _c.c_longlong, _c.c_longlong, _c.c_float, _c.c_float, _c.c_float, _c.c_int, VP, VP, _c.c_int, VP]
        lib.blz_attn_decode_tree.argtypes = [VP, VP, VP, VP, VP, VP, VP, _c.c_int, _c.c_int, _c.c_int, _c.c_int, _c.c_int,
                                             _c.c_longlong, _c.c_longlong, _c.c_float, _c.c_float, _c.c_float, _c.c_int, _c.c_int, _c.c_int,
                                             _c.c_int, _c.c_int, VP, VP, _c.c_int, VP, VP, VP]
        lib.blz_kv_move_rows.argtypes = [VP, VP, VP, VP, _c.c_int, _c.c_int, _c.c_int, _c.c_longlong, _c.c_longlong, VP]
        lib.blz_mul_sigmoid.argtypes = [VP, VP, _c.c_longlong, VP]
        lib.blz_add.argtypes = [VP, VP, VP, _c.c_longlong, VP]
        lib.blz_add_sigmoid_scaled.argtypes = [VP, VP, VP, VP, _c.c_int, _c.c_int, VP]
        lib.blz_gather_rows.argtypes = [VP, VP, VP, _c.c_int, _c.c_int, VP]
        lib.blz_argmax.argtypes = [VP, VP, VP, _c.c_int, _c.c_int, _c.c_longlong, _c.c_int, VP]
        lib.blz_moe_route.argtypes = [VP, _c.c_longlong, VP, VP, VP] + [_c.c_int] * 7 + [VP]
        lib.blz_moe_plan.argtypes = [VP, VP, VP, VP, VP, _c.c_int, _c.c_int, VP]
        lib.blz_moe_gemm.restype = _c.c_int
        lib.blz_moe_gemm.argtypes = [_c.c_int, VP, _c.c_longlong, VP, _c.c_longlong, VP, _c.c_longlong, _c.c_int, _c.c_int, _c.c_int,
                                     _c.c_int, VP, VP, VP, VP, VP, VP, _c.c_int, VP]
        lib.blz_gemm_narrow.restype = _c.c_int
        lib.blz_gemm_narrow.argtypes = [_c.c_int, VP, _c.c_longlong, VP, _c.c_longlong, VP, _c.c_longlong, _c.c_int, _c.c_int, _c.c_int,
                                        VP, VP, VP, VP, VP, _c.c_int, _c.c_int, _c.c_float, VP]
        # dense layers with few rows (single-user decoding, verify steps) and a large weight take the features-on-lanes kernel
        # with the K range split over a cluster (blz_gemm_narrow).  Measured on B200, NVFP4, captured-graph timing, against the
        # one-CTA-per-tile kernel: 1-32 rows 24576x4096 21 -> 16 us, 4096x12288 19 -> 16 us, 17408x5120 18 -> 16 us, 6144x4096
        # equal, 4096x4096 11.3 -> 12.0 us (loses); at 64 rows only the 24576-wide layer still wins, at 128 rows none does: both
        # kernels sit on a floor of about 10 us (launch, set-up, first load, reduction) at these sizes.  0 = never.
        self.NARROW_ROWS = int(os.environ.get("BLAZE_GEMM_NARROW_ROWS", "64"))
        self.NARROW_ALWAYS = os.environ.get("BLAZE_GEMM_NARROW_ALWAYS", "0") == "1"
        lib.blz_swiglu_live.argtypes = [VP, VP, VP, VP, VP, _c.c_int, _c.c_int, _c.c_int, _c.c_int, VP, VP]
        # routed rows per expert below this: the expert GEMMs put the features on the tensor-core lanes and only the live rows
        # on its columns (blz_moe_gemm); above it the 128-row tiles of the grouped GEMM are full enough (BLAZE_MOE_NARROW=0: never)
        self.MOE_NARROW_ROWS = 48 if os.environ.get("BLAZE_MOE_NARROW", "1") != "0" else 0
        lib.blz_moe_scatter.argtypes = [_c.c_int, VP, VP, VP, VP, VP, VP, VP, VP, VP, VP, _c.c_int, _c.c_int, _c.c_int, _c.c_int,
                                        _c.c_int, VP, _c.c_int, VP]
        lib.blz_moe_combine.argtypes = [VP, VP, VP, VP, _c.c_int, _c.c_int, _c.c_int, VP]
        self._route_counts = None
        lib.blz_gdn_conv.argtypes = [VP, _c.c_longlong, VP, VP, VP, VP, VP, VP, VP, _c.c_int, _c.c_int, _c.c_int, VP]
        lib.blz_gdn_recurrent.argtypes = [VP, VP, VP, _c.c_longlong, VP, VP, VP, VP, VP, VP, VP, VP, _c.c_int, _c.c_int, _c.c_int,
                                          _c.c_int, _c.c_int, VP]
        lib.blz_gdn_conv_runs.argtypes = [VP, _c.c_longlong, VP, VP, VP, VP, VP, VP, VP, _c.c_int, _c.c_int, _c.c_int, _c.c_int, VP]
        lib.blz_gdn_recurrent_upto.argtypes = [VP, VP, VP, _c.c_longlong, VP, VP, VP, VP, VP, VP, VP, VP, _c.c_int, _c.c_int, _c.c_int,
                                               _c.c_int, _c.c_int, _c.c_int, VP]
        lib.blz_gdn_chunk.argtypes = [VP, VP, VP, _c.c_longlong, VP, VP, VP, VP, VP, VP, VP, VP, _c.c_int, _c.c_int, _c.c_int,
                                      _c.c_int, _c.c_int, _c.c_int, VP]
        # Gated DeltaNet: sequences with at least this many new tokens in a step take the chunked tensor-core kernel (0 = never)
        self.GDN_CHUNK_MIN = int(os.environ.get("BLAZE_GDN_CHUNK_MIN", "64"))
        lib.blz_gdn_chunk_split.argtypes = [VP, VP, VP, _c.c_longlong, VP, VP, VP, VP, VP, VP, VP, VP, _c.c_int, _c.c_int, _c.c_int,
                                            _c.c_int, _c.c_int, _c.c_int, _c.c_int, _c.c_int, VP, VP]
        lib.blz_gdn_chunk_ws_bytes.restype = _c.c_longlong
        lib.blz_gdn_chunk_ws_bytes.argtypes = [_c.c_int, _c.c_int]
        # chunk-parallel preparation + sequential scan (two kernels) instead of the one fused kernel; 0 keeps the fused one
        self.GDN_SPLIT = os.environ.get("BLAZE_GDN_SPLIT", "1") != "0"
        self.GDN_SPLIT_MAX_WS = 4 << 30
        lib.blz_gated_rmsnorm.argtypes = [VP, VP, _c.c_longlong, VP, VP, _c.c_int, _c.c_int, _c.c_int, _c.c_float, _c.c_int, VP]
        lib.blz_status_take.restype = _c.c_int
        lib.blz_status_peek_async.restype = _c.c_int
        lib.blz_status_peek_async.argtypes = [VP, VP]
        # static residual streams, differential attention, 32-bit products
        lib.blz_streams.argtypes = [VP, VP, VP, _c.c_int, _c.c_float, VP, VP, VP, VP, VP, _c.c_float, VP, VP, _c.c_int, _c.c_int, _c.c_int,
                                    _c.c_int, _c.c_int, _c.c_int, VP]
        lib.blz_residual_norm.argtypes = [VP, _c.c_int, _c.c_float, VP, VP, _c.c_float, VP, VP, _c.c_int, _c.c_int, _c.c_int, VP]
        lib.blz_norm_rows.argtypes = [VP, VP, VP, VP, _c.c_int, _c.c_int, _c.c_float, _c.c_int, _c.c_int, VP]
        lib.blz_gemm_simple.argtypes = [VP, _c.c_longlong, VP, _c.c_longlong, VP, _c.c_longlong, VP, _c.c_int, _c.c_int, _c.c_int, _c.c_int,
                                        _c.c_int, VP]
        lib.blz_clamped_glu.argtypes = [VP, VP, _c.c_int, _c.c_int, _c.c_float, _c.c_int, VP]
        lib.blz_diff_store.argtypes = [VP, _c.c_longlong, VP, _c.c_longlong, _c.c_longlong, VP] + [_c.c_int] * 6 + [VP]
        common = [VP, _c.c_longlong, VP, VP, _c.c_longlong, _c.c_longlong, VP, _c.c_int, VP, VP, VP]
        shape = [_c.c_int] * 7 + [_c.c_float] * 4
        lib.blz_diff_plain.argtypes = common + [VP] + shape + [_c.c_int, VP]
        lib.blz_diff_tc.argtypes = common + shape + [_c.c_int, _c.c_int, VP]
        lib.blz_diff_short.argtypes = common + shape + [_c.c_int, _c.c_int, _c.c_int, VP, VP, VP]

        # one softmax map with sink and gate; recurrences
        LL = _c.c_longlong
        lib.blz_attn_prep_pages.argtypes = [VP] + [LL] * 4 + [VP, VP, LL, LL, VP, VP, VP] + [_c.c_int] * 8 + [_c.c_float, _c.c_int, VP]
        common = [VP, LL, VP, LL, VP, LL, LL, VP, _c.c_int, VP, VP, VP, VP, VP, LL]
        shape = [_c.c_int] * 7 + [_c.c_float] * 2
        lib.blz_soft_plain.argtypes = common + [VP] + shape + [_c.c_int, VP]
        lib.blz_soft_tc.argtypes = common + shape + [_c.c_int, _c.c_int, VP, VP]
        lib.blz_soft_short.argtypes = common + shape + [_c.c_int, _c.c_int, _c.c_int, VP, VP, VP]
        lib.blz_short_conv.argtypes = [VP, LL] + [VP] * 8 + [_c.c_int] * 5 + [VP]
        runs = [_c.c_int] * 5 + [VP] + [_c.c_int] * 2 + [VP, LL, _c.c_int, VP]
        lib.blz_delta_rule.argtypes = [VP, LL, VP, LL, VP, LL] + [VP] * 8 + [_c.c_int] + runs
        lib.blz_state_space.argtypes = [VP, LL, VP, LL] + [VP] * 9 + runs
        lib.blz_rec_ws_bytes.restype = LL
        lib.blz_rec_ws_bytes.argtypes = [_c.c_int] * 5
        lib.blz_gated_linear.argtypes = [VP, LL, VP, LL, VP, LL] + [VP] * 8 + [_c.c_int] * 4 + [VP] + [_c.c_int] * 2 + [VP, LL, _c.c_int, VP]
        # residual with normed branches, input convolution, feed-forwards without a gate
        lib.blz_branch_norm.argtypes = [VP, LL, VP, VP, _c.c_int, VP, VP, _c.c_float, VP, VP] + [_c.c_int] * 3 + [VP]
        lib.blz_embed_norm.argtypes = [VP, VP, _c.c_int, VP, _c.c_float, VP] + [_c.c_int] * 3 + [VP]
        lib.blz_input_conv.argtypes = [VP] * 8 + [_c.c_int] * 5 + [VP]
        lib.blz_relu2.argtypes = [VP, _c.c_int, VP, LL, _c.c_int, VP]
        lib.blz_poly_norm.argtypes = [VP, VP, VP, _c.c_int, _c.c_int, _c.c_float, _c.c_int, VP]
        lib.blz_gemm_simple_experts.argtypes = [VP, LL, VP, VP, LL] + [_c.c_int] * 3 + [VP, VP, _c.c_int, VP]
        # mixer and feed-forward side by side, position vectors, sigmoid attention, minGRU
        lib.blz_branch_step.argtypes = [VP] * 6 + [LL, VP, VP, _c.c_int, VP, VP, LL] + [VP] * 5 + [LL] + [_c.c_float] * 2 + [_c.c_int] * 3 + [VP]
        lib.blz_embed_positions.argtypes = [VP] * 4 + [_c.c_int, _c.c_float, VP, VP, LL] + [_c.c_int] * 3 + [VP]
        lib.blz_conv_prep_pages.argtypes = ([VP] + [LL] * 4 + [VP, VP, LL, LL] + [VP] * 8 + [_c.c_int] * 9 + [_c.c_float] * 3 +
                                            [_c.c_int] * 2 + [VP])
        common = [VP, LL, VP, LL, VP, LL, LL, VP, _c.c_int, VP, VP, VP, VP, _c.c_int]
        lib.blz_sigmoid_plain.argtypes = common + [VP] + shape + [_c.c_int, VP]
        lib.blz_sigmoid_tc.argtypes = common + shape + [_c.c_int, _c.c_int, VP]
        lib.blz_sigmoid_short.argtypes = common + shape + [_c.c_int, _c.c_int, _c.c_int, VP, VP, VP]
        lib.blz_min_gru.argtypes = [VP, VP, VP, LL, VP, VP, LL, VP, VP, VP, VP] + [_c.c_int] * 4 + [VP, _c.c_int, VP]
        lib.blz_min_gru_ws_bytes.restype = LL
        lib.blz_min_gru_ws_bytes.argtypes = [_c.c_int] * 3
        # latent attention
        lib.blz_latent_prep.argtypes = [VP, LL, LL, LL, VP, VP, LL, VP, VP, VP, VP, VP] + [_c.c_int] * 5 + [_c.c_float, _c.c_int, VP]
        lib.blz_latent_rot.argtypes = [VP] * 5 + [_c.c_int] * 7 + [VP]
        lib.blz_latent_map.argtypes = [VP] * 5 + [_c.c_int] * 6 + [VP, VP, _c.c_int, _c.c_int, VP]
        lib.blz_head_gemm.argtypes = [VP, LL, LL, VP, VP, LL, LL] + [_c.c_int] * 4 + [VP, VP, _c.c_int, _c.c_int, VP]
        lib.blz_latent_rows_block.restype = _c.c_int
        lib.blz_latent_rows_block.argtypes = [_c.c_int] * 3 + [VP]
        lib.blz_latent_rows.argtypes = [VP, VP, VP, LL, VP, _c.c_int, VP, VP, VP, VP] + [_c.c_int] * 5 + [_c.c_float] + [_c.c_int] * 5 + [VP, VP, VP]
        lib.blz_latent_gather.argtypes = [VP, LL, VP, _c.c_int, VP, _c.c_int, _c.c_int, VP]
        lib.blz_expand_store.argtypes = [VP, LL, VP, LL, VP, VP] + [_c.c_int] * 6 + [VP]
        lib.blz_shared_plain.argtypes = [VP, LL, VP, LL, VP, LL, VP, _c.c_int, VP, VP, VP, VP, VP] + [_c.c_int] * 6 + [_c.c_float, _c.c_int, VP]
        lib.blz_group_norm.argtypes = [VP, VP, LL, VP, VP, LL] + [_c.c_int] * 4 + [_c.c_float] * 2 + [_c.c_int] * 3 + [VP]

    # ------------------------------------------------------------------ plumbing
    def _stream(self) -> VP:
        s = self._held_stream
        return s if s is not None else VP(torch.cuda.current_stream(self.device).cuda_stream)

    def hold_stream(self) -> None:
        """Look the current stream up once for the launches that follow (a step of the engine issues hundreds, and the
        look-up costs more host time than the launch itself); ``release_stream`` ends it.  Calls nest."""
        if self._held_depth == 0:
            self._held_stream = VP(torch.cuda.current_stream(self.device).cuda_stream)
        self._held_depth += 1

    def release_stream(self) -> None:
        self._held_depth = max(self._held_depth - 1, 0)
        if self._held_depth == 0:
            self._held_stream = None

    def _check(self, code: int, what: str) -> None:
        self.launches += 1
        if code != 0:
            raise CudaError(f"{what} failed with cudaError {code}")

    def take_status(self) -> int:
        """Read and clear the device status word (non-zero = a bounded device wait ran out)."""
        return int(self.lib.blz_status_take())

    def status_peek(self, host_word: torch.Tensor) -> None:
        """Queue a copy of the status word into ``host_word`` (pinned int32) behind the work already on the stream."""
        rc = self.lib.blz_status_peek_async(VP(host_word.data_ptr()), self._stream())
        if rc != 0:
            raise CudaError(f"blz_status_peek_async failed: {rc}")

    def _buf(self, key: str, nbytes: int) -> torch.Tensor:
        """Scratch that only grows.  A buffer that is outgrown is kept alive: captured graphs of smaller steps still hold
        its address, and handing that memory back to the allocator would let other tensors land under their writes."""
        b = self._scratch.get(key)
        if b is None or b.numel() < nbytes:
            if b is not None:
                self._retired.append(b)
            b = torch.empty(max(nbytes, 1), dtype=torch.uint8, device=self.device)
            self._scratch[key] = b
        return b

    # ------------------------------------------------------------------ weights → kernel layouts
    @staticmethod
    def tile_major(w: torch.Tensor) -> Tuple[torch.Tensor, int]:
        """Row-major weight bytes [N, row bytes] -> [ceil(N/128), kt, 128, 128] (zero padded): every 128-row x 128-byte
        operand tile becomes one contiguous 16 KB run, so a CTA streaming a weight tile reads DRAM pages end to end
        instead of touching a new page for every 128 bytes."""
        b = w.contiguous().view(torch.uint8).view(w.shape[0], -1)
        N, KB = b.shape
        NP, KP = (N + 127) // 128 * 128, (KB + 127) // 128 * 128
        if (NP, KP) != (N, KB):
            pad = torch.zeros(NP, KP, dtype=torch.uint8, device=b.device)
            pad[:N, :KB] = b
            b = pad
        kt = KP // 128
        t = b.view(NP // 128, 128, kt, 128).permute(0, 2, 1, 3).contiguous()
        # store each tile as the 128-byte-swizzled shared-memory image the tensor core reads (16-byte chunk c of row r
        # sits at chunk c ^ (r % 8)), so that the kernel fetches a whole 16 KB tile with ONE bulk copy
        v = t.view(NP // 128, kt, 16, 8, 8, 16)
        r = torch.arange(8, device=b.device).view(8, 1)
        c = torch.arange(8, device=b.device).view(1, 8)
        src = (c ^ r).view(1, 1, 1, 8, 8, 1).expand(NP // 128, kt, 16, 8, 8, 16)
        return torch.gather(v, 4, src).contiguous().view(NP // 128, kt, 128, 128), kt

    @staticmethod
    def swiglu_order(n_rows: int) -> torch.Tensor:
        """Row order that turns stacked ``[gate (I rows); up (I rows)]`` into groups of 16 gate rows followed by the 16 up
        rows of the same features, so that one 32-column group of the GEMM output holds both halves of 16 activations."""
        I = n_rows // 2
        g = torch.arange(I).view(I // 16, 16)
        return torch.cat([g, g + I], dim=1).reshape(-1)

    def pack(self, lin: Linear, tiled: Optional[bool] = None, swiglu: bool = False, exact_fp8: bool = True):
        """``tiled`` (default: off unless BLAZE_TILED_WEIGHTS=1): store the weight tile-major (see ``tile_major``); the grouped
        expert GEMM asks for row-major.  ``swiglu``: interleave the gate and up rows for the GEMM's SwiGLU epilogue (the
        packed weight is then only valid for ``linear_swiglu``)."""
        if lin.cuda_pack is not None:
            if bool(lin.cuda_pack.get("swiglu")) != bool(swiglu):
                raise CudaError("this weight was packed for the other epilogue (plain / SwiGLU)")
            return lin.cuda_pack
        pk = self._pack(lin, self.swiglu_order(lin.N).to(self.device) if swiglu else None, exact_fp8=exact_fp8)
        pk["swiglu"] = bool(swiglu)
        if tiled is None:
            tiled = self._tiled_ok
        pk["kt"] = 0
        if tiled:
            pk["w"], pk["kt"] = self.tile_major(pk["w"])
        lin.cuda_pack = pk
        return pk

    def _pack(self, lin: Linear, order: Optional[torch.Tensor] = None, exact_fp8: bool = True):
        """``order``: optional permutation of the output rows applied to the weight, its scales, alpha and bias.
        ``exact_fp8`` = False: an FP8 block-scale weight is re-expressed in MXFP8 (what the grouped expert GEMM consumes)."""
        dev = self.device

        def perm(t):
            return t if (order is None or t is None) else t.to(dev)[order]

        if lin.fmt == Format.DENSE and lin.w.dtype == torch.float32:
            if order is not None:
                raise CudaError("32-bit weights are not interleaved: their gated activation is an op of its own")
            return {"kind": 5, "w": lin.w.to(dev).contiguous(), "sf": None, "alpha": None,
                    "bias": None if lin.bias is None else lin.bias.to(dev, torch.float32).contiguous()}
        if lin.fmt == Format.DENSE:
            pk = {"kind": 0, "w": perm(lin.w.to(dev, torch.bfloat16)).contiguous(), "sf": None, "alpha": None}
        elif lin.fmt == Format.NVFP4:
            rows = (lin.N + 255) // 256 * 256
            sf = torch.zeros(rows, lin.K // 16, dtype=torch.uint8, device=dev)
            sf[:lin.N] = perm(lin.sf.to(dev).view(torch.uint8))
            pk = {"kind": 1, "w": perm(lin.w.to(dev)).contiguous(), "sf": quant.swizzle_sf_128x4(sf),
                  "alpha": perm(lin.alpha.to(dev, torch.float32)).contiguous()}
        elif lin.fmt == Format.FP8_BLOCK and self._fp8_block_exact and exact_fp8 and order is None and tuple(lin.block) == (128, 128) \
                and lin.K % 128 == 0 and tuple(lin.sf.shape) == ((lin.N + 127) // 128, lin.K // 128):
            pk = {"kind": 4, "w": lin.w.to(dev).view(torch.uint8).contiguous(), "sf": lin.sf.to(dev, torch.float32).contiguous(),
                  "alpha": None}
        elif lin.fmt in (Format.MXFP8, Format.FP8_BLOCK):
            if lin.fmt == Format.FP8_BLOCK:
                # 128x128 fp32 block scales have no native MMA mode: re-express the weight as e4m3 with one e8m0
                # scale per 32 elements (exact when the block scales are powers of two).
                q, e8 = quant.mxfp8_quantize(lin.dequant().to(dev))
            else:
                q, e8 = lin.w.to(dev), lin.sf.to(dev)
            rows = (lin.N + 255) // 256 * 256
            sf = torch.full((rows, lin.K // 32), 127, dtype=torch.uint8, device=dev)
            sf[:lin.N] = perm(e8.view(torch.uint8))
            alpha = None if lin.fmt == Format.FP8_BLOCK else perm(lin.alpha.to(dev, torch.float32)).contiguous()
            pk = {"kind": 2, "w": perm(q.view(torch.uint8)).contiguous(), "sf": quant.swizzle_sf_128x4(sf), "alpha": alpha}
        else:  # per-channel / per-tensor FP8
            pk = {"kind": 3, "w": perm(lin.w.to(dev).view(torch.uint8)).contiguous(), "sf": None,
                  "alpha": perm(lin.alpha.to(dev, torch.float32)).contiguous()}
        pk["bias"] = None if lin.bias is None else perm(lin.bias.to(dev, torch.bfloat16)).contiguous()
        return pk

    # ------------------------------------------------------------------ activation quantisation
    def _alloc_qact(self, fmt: Format, T: int, K: int) -> QuantAct:
        dev = self.device
        if fmt == Format.NVFP4:
            data = torch.empty(T, K // 2, dtype=torch.uint8, device=dev)
            sf = torch.empty(((T + 127) // 128) * ((K + 63) // 64) * 512, dtype=torch.uint8, device=dev)
            rs = torch.empty(T, dtype=torch.float32, device=dev)
        else:
            data = torch.empty(T, K, dtype=torch.uint8, device=dev)
            sf = torch.empty(((T + 127) // 128) * ((K + 127) // 128) * 512, dtype=torch.uint8, device=dev)
            rs = None
        return QuantAct(fmt, data, sf, rs, T, K)

    def _qmode(self, lin: Optional[Linear]) -> int:
        """Activation format the producer's epilogue should emit for ``lin``: 0 bf16, 1 NVFP4, 2 MXFP8.  (The exact FP8
        block-scale GEMM quantises its bf16 input itself, to e4m3 with one fp32 scale per 1x128 group.)"""
        if lin is None or not lin.act_quant:
            return 0
        if lin.fmt == Format.NVFP4:
            return 1
        if lin.fmt == Format.MXFP8:
            return 2
        if lin.fmt == Format.FP8_BLOCK:
            pk = lin.cuda_pack
            return 0 if (pk["kind"] == 4 if pk is not None else self._fp8_block_exact) else 2
        return 0

    def quantize_fp8_block(self, x: torch.Tensor):
        """bf16 ``[T, K]`` -> (e4m3 codes ``[T, K]``, fp32 scales ``[K / 128, T4]``) with one scale per row and 128 columns."""
        T, K = x.shape
        ld = (T + 3) // 4 * 4
        q = torch.empty(T, K, dtype=torch.uint8, device=self.device)
        sc = torch.empty(K // 128, ld, dtype=torch.float32, device=self.device)
        if x.stride(1) != 1:
            x = x.contiguous()
        self._check(self.lib.blz_quant_fp8_block(_ptr(x), x.stride(0), _ptr(q), _ptr(sc), ld, T, K, self._stream()), "quant_fp8_block")
        return q, sc

    def quantize_rows(self, x: torch.Tensor, lin: Linear) -> QuantAct:
        """bf16 ``[T, K]`` → the activation format ``lin`` consumes."""
        mode = self._qmode(lin)
        T, K = x.shape
        qa = self._alloc_qact(Format.NVFP4 if mode == 1 else Format.MXFP8, T, K)
        self._check(self.lib.blz_swiglu(_ptr(x), VP(0), _ptr(qa.data), _ptr(qa.sf), _ptr(qa.row_scale), T, K, mode, 1,
                                        self._stream()), "quantize_rows")
        return qa

    # ------------------------------------------------------------------ basics
    def embed(self, table, tokens):
        T, H = tokens.numel(), table.shape[1]
        out = torch.empty(T, H, dtype=table.dtype, device=self.device)
        self._check(self.lib.blz_embed(_ptr(table), _ptr(tokens), _ptr(out), T, H * table.element_size() // 2, table.shape[0],
                                       self._stream()), "embed")
        return out

    def norm(self, x, residual, w, eps, zero_centered=False, quant_for: Optional[Linear] = None, zero_src: bool = False):
        T, H = x.shape
        mode = self._qmode(quant_for)
        new_res = residual if residual is not None else x
        if mode == 0:
            out = torch.empty_like(x)
            self._check(self.lib.blz_rmsnorm(_ptr(x), _ptr(residual), _ptr(w), _ptr(out), VP(0), VP(0), VP(0), T, H, eps,
                                             int(zero_centered), 0, int(zero_src), self._stream()), "rmsnorm")
            return out, new_res
        qa = self._alloc_qact(Format.NVFP4 if mode == 1 else Format.MXFP8, T, H)
        self._check(self.lib.blz_rmsnorm(_ptr(x), _ptr(residual), _ptr(w), VP(0), _ptr(qa.data), _ptr(qa.sf),
                                         _ptr(qa.row_scale), T, H, eps, int(zero_centered), mode, int(zero_src), self._stream()), "rmsnorm_q")
        return qa, new_res

    WIDE_WS_BYTES = 40 << 20

    def linear_swiglu(self, lin: Linear, x, quant_for: Optional[Linear] = None):
        """``silu(x @ Wg^T) * (x @ Wu^T)`` for a stacked ``[gate; up]`` weight with the activation computed in the GEMM's
        epilogue (the ``[T, 2I]`` intermediate never reaches memory); quantised for ``quant_for`` when that GEMM wants it."""
        exact8 = lin.fmt == Format.FP8_BLOCK and (lin.cuda_pack["kind"] == 4 if lin.cuda_pack is not None else self._fp8_block_exact)
        if lin.fmt == Format.DENSE and (lin.w.dtype == torch.float32 or lin.N % 32 or lin.K % 16):
            return self._glu(self.linear(lin, x), -1.0)
        if lin.N % 32 or (lin.N // 2) % 8 or exact8:
            return self.silu_mul(self.linear(lin, x), quant_for=quant_for)
        act = self.linear(lin, x, swiglu=True)
        return self.quantize_rows(act, quant_for) if self._qmode(quant_for) else act

    def _linear_simple(self, lin, pk, x, f32: bool, out=None):
        """``x @ W^T`` on the CUDA cores: 32-bit weights, and bf16 rows too ragged for the TMA kernels."""
        in32 = pk["kind"] == 5
        if x.dtype != (torch.float32 if in32 else torch.bfloat16):
            raise CudaError(f"{x.dtype} activations for {pk['w'].dtype} weights")
        if x.stride(1) != 1:
            x = x.contiguous()
        M = x.shape[0]
        if out is None:
            out = torch.empty(M, lin.N, dtype=torch.float32 if f32 else torch.bfloat16, device=self.device)
        if M == 0:
            return out
        bias = pk["bias"].float() if pk["bias"] is not None else None
        self._check(self.lib.blz_gemm_simple(_ptr(x), x.stride(0), _ptr(pk["w"]), lin.K, _ptr(out), out.stride(0), _ptr(bias), M, lin.N, lin.K,
                                             int(in32), int(f32), self._stream()), "gemm_simple")
        return out

    def linear_glu(self, lin: Linear, x, limit: float):
        """``g * sigmoid(1.702 g) * (u + 1)`` with ``g = min(x @ Wg^T, limit)`` and ``u`` = ``x @ Wu^T`` clamped to ``+-limit``, for a
        stacked ``[gate; up]`` weight: in the GEMM's epilogue (fp32 accumulators) where the shape allows."""
        if lin.w.dtype != torch.float32 and lin.N % 32 == 0 and lin.K % 16 == 0:
            return self.linear(lin, x, swiglu=True, glu_limit=limit)
        return self._glu(self.linear(lin, x), limit)

    def _glu(self, gu, limit: float):
        """The gated activation as an op of its own (``limit`` < 0: SwiGLU)."""
        T, I = gu.shape[0], gu.shape[1] // 2
        out = torch.empty(T, I, dtype=gu.dtype, device=self.device)
        if T:
            self._check(self.lib.blz_clamped_glu(_ptr(gu), _ptr(out), T, I, limit, int(gu.dtype == torch.float32), self._stream()), "clamped_glu")
        return out

    def linear_argmax(self, lin: Linear, x, index_offset: int = 0, want_values: bool = False):
        """``argmax(x @ W^T)`` per row without writing the logits: the GEMM epilogue keeps the best (value, column) of each
        128-column tile and a small kernel merges the tiles (ties to the lower column, like ``argmax``)."""
        if self.pack(lin)["kind"] == 5 or lin.K % 16:
            return self.argmax(self.linear(lin, x, out_dtype=torch.float32), index_offset, want_values)
        M = x.rows if isinstance(x, QuantAct) else x.shape[0]
        tiles = (lin.N + 127) // 128
        val = self._buf("amax_val", tiles * max(M, 1) * 4).view(torch.float32)
        idx = self._buf("amax_idx", tiles * max(M, 1) * 4).view(torch.int32)
        out = torch.empty(M, dtype=torch.int64, device=self.device)
        vals = torch.empty(M, dtype=torch.float32, device=self.device) if want_values else None
        if M == 0:
            return (out, vals) if want_values else out
        self.linear(lin, x, out_dtype=torch.float32, wide=False, argmax_parts=(val, idx))
        self._check(self.lib.blz_argmax_parts(_ptr(val), _ptr(idx), tiles, M, _ptr(out), _ptr(vals), index_offset,
                                              self._stream()), "argmax_parts")
        return (out, vals) if want_values else out

    def _linear_fp8_block(self, lin, pk, x, f32, out, swiglu, argmax_parts, wide, sk):
        if swiglu or argmax_parts is not None or wide or (sk is not None and sk is not False):
            raise CudaError("the FP8 block-scale GEMM has the plain epilogue only (bf16 / fp32 output, optional bias)")
        q = sc = None
        if isinstance(x, QuantAct):
            if x.wait is not None:
                raise CudaError("an activation with a pending peer wait cannot feed the FP8 block-scale GEMM")
            if x.fmt == Format.FP8_BLOCK:
                q, sc = x.data, x.sf              # already in 1x128 groups (quantize_fp8_block)
            else:
                x = x.dense
        M = q.shape[0] if q is not None else x.shape[0]
        if out is None:
            out = torch.empty(M, lin.N, dtype=torch.float32 if f32 else torch.bfloat16, device=self.device)
        if M == 0:
            return out
        if q is None:
            q, sc = self.quantize_fp8_block(x)
        self._check(self.lib.blz_gemm_fp8_block(_ptr(q), lin.K, _ptr(pk["w"]), lin.K, _ptr(out), out.stride(0), M, lin.N, lin.K,
                                                _ptr(sc), sc.stride(0), _ptr(pk["sf"]), _ptr(pk["bias"]), int(f32), self._stream()),
                    "gemm_fp8_block")
        return out

    def linear(self, lin: Linear, x, out_dtype=None, out: Optional[torch.Tensor] = None, bn: int = 0, max_ctas: int = 0,
               wide: Optional[bool] = None, ksplit: int = 0, swiglu: bool = False, argmax_parts=None, sk=None,
               glu_limit: Optional[float] = None, relu2: bool = False):
        """``wide``: None = choose; False = the 128-column kernel (needed by the fused all-reduce epilogue); True = insist on
        the wide-N kernel (raises when the shape is not covered).  ``sk``: None = choose; False = never; True or a K-slice
        count 1..8 = the cluster split-K kernel (bf16 output, row-major weights).  ``swiglu`` with ``glu_limit``: the clamped
        gated activation instead of SwiGLU.  ``relu2``: squared ReLU of the result."""
        pk = self.pack(lin, swiglu=swiglu)
        kind = pk["kind"]
        act, limit = (3 if relu2 else int(swiglu)) if glu_limit is None else 2, float(glu_limit or 0.0)
        if relu2:
            wide = sk = False
        if kind == 5 or (kind == 0 and lin.K % 16):
            if swiglu or argmax_parts is not None:
                raise CudaError("the CUDA-core GEMM has the plain epilogue only")
            return self._linear_simple(lin, pk, x, kind == 5 or out_dtype == torch.float32, out)
        f32 = out_dtype == torch.float32
        n_out = lin.N // 2 if swiglu else lin.N
        sfa = rs = None
        if kind == 4:
            return self._linear_fp8_block(lin, pk, x, f32, out, swiglu, argmax_parts, wide, sk)
        if kind in (1, 2):
            if not isinstance(x, QuantAct):
                x = self.quantize_rows(x.contiguous(), lin)
            a, sfa, rs, M = x.data, x.sf, x.row_scale, x.rows
            lda = a.shape[1]
        elif kind == 3:
            xt = x.dense if isinstance(x, QuantAct) else x
            q, s = quant.fp8_rowwise_quantize(xt)
            a, rs, M = q.view(torch.uint8).contiguous(), s.float().contiguous(), xt.shape[0]
            lda = a.shape[1]
        else:
            # rows may be a run of columns of a wider matrix where TMA can start and step on 16 bytes
            a = x if x.stride(1) == 1 and x.stride(0) % 8 == 0 and x.data_ptr() % 16 == 0 else x.contiguous()
            M, lda = a.shape[0], a.stride(0) * 2
        if argmax_parts is not None:
            out = argmax_parts[0]            # the logits are not written; any valid pointer will do
            ld_out = n_out
        elif out is None:
            out = torch.empty(M, n_out, dtype=torch.float32 if f32 else torch.bfloat16, device=self.device)
        if argmax_parts is None:
            ld_out = out.stride(0)
        if M == 0:
            return out
        w = pk["w"]
        kt = pk.get("kt", 0)
        ldb = 128 if kt else w.shape[1] * w.element_size()
        pending = getattr(x, "wait", None) if isinstance(x, QuantAct) else None
        if pending is not None:
            # the peers may still be writing these rows: the 128-column kernel waits for their flags after it has sent
            # its first weight tiles
            if wide:
                raise CudaError("an activation with a pending peer wait needs the 128-column GEMM")
            wide = False
            rc = self.lib.blz_gemm_wait_flags(VP(pending[0]), VP(pending[1]), pending[2], pending[3])
            if rc != 0:
                raise CudaError(f"blz_gemm_wait_flags failed: {rc}")
            x.wait = None
        big = self.NARROW_ALWAYS or (lin.N * lin.K >= 6144 * 4096 if M <= 32 else lin.N >= 16384)
        narrow = (M <= self.NARROW_ROWS and big and kind in (0, 1, 2) and lin.N % 128 == 0 and not f32 and argmax_parts is None
                  and pending is None and not kt and (wide is None or relu2) and bn == 0 and (sk is None or sk is False)
                  and (not swiglu or ld_out % 8 == 0) and (sfa is None or sfa.numel() >= 512))
        if narrow:
            self._check(self.lib.blz_gemm_narrow(kind, _ptr(a), lda, _ptr(w), ldb, _ptr(out), ld_out, M, lin.N, lin.K, _ptr(rs),
                                                 _ptr(pk["alpha"]), _ptr(pk["bias"]), _ptr(sfa), _ptr(pk["sf"]), 0, act, limit,
                                                 self._stream()), f"gemm_narrow kind {kind}")
            return out
        sk_able = not f32 and argmax_parts is None and pending is None and not kt
        if sk is None:
            sk = False
            if self._sk_ok and sk_able and wide is None and bn == 0 and M <= self.SK_MAX_ROWS:
                # Measured on B200 (NVFP4, 256 rows, captured-graph timing): splitting K over a cluster pays when the K range
                # is long and the tiles are few (4096 x 12288: 23.7 -> 22.2 us); for the other decode shapes the exchange of
                # fp32 partials through distributed shared memory (about 5 us per 64 KB tile) costs what the split saves.
                # A tuning table measured on this device (tune.tune_linear) overrides the rule.
                tiles = ((M + 127) // 128) * ((lin.N + 127) // 128)
                sk = lin.K >= 8192 and tiles <= 2 * self._sm // 2
                if self.tuning is not None:
                    from ..tune import bucket
                    hit = self.tuning.get(f"gemm{kind}", lin.N, lin.K, bucket(M))
                    if hit is not None:
                        sk = False if hit.get("kernel") != "sk" else (hit.get("ks") or True)
        if sk is not False and sk is not None:
            if not sk_able:
                raise CudaError("the split-K GEMM writes bf16 from row-major weights and has no arg-max / peer-wait epilogue")
            ks = 0 if sk is True else int(sk)
            self._check(self.lib.blz_gemm_sk(kind, _ptr(a), lda, _ptr(w), ldb, _ptr(out), ld_out, M, lin.N, lin.K,
                                             _ptr(rs), _ptr(pk["alpha"]), _ptr(pk["bias"]), _ptr(sfa), _ptr(pk["sf"]),
                                             ks, act, limit, self._stream()), f"gemm_sk kind {kind}")
            return out
        if wide is None:
            # Measured on B200 (Qwen3-8B shapes, captured-graph timing): 256-feature tiles win for block-scaled prefill GEMMs
            # (NVFP4 2048x24576x4096: 156 -> 119 us); the swapped orientation wins for the very wide bf16 head
            # (256x151936x4096: 346 -> 315 us) but not for the per-layer decode GEMMs, which stay on the 128-column kernel.
            wide = self._wide_ok and bn == 0 and ((M <= 256 and kind == 0 and lin.N >= 32768 and not swiglu)
                                                  or (kind in (1, 2) and lin.N % 256 == 0 and M > 256))
        if wide:
            swap = M <= 256
            ks, ws, ctr = 1, None, None
            if swap:
                tok = 64 if M <= 64 else (128 if M <= 128 else 256)
                tiles = (lin.N + 127) // 128
                k_tiles = (lin.K + (64 if kind == 0 else 256 if kind == 1 else 128) - 1) // (64 if kind == 0 else 256 if kind == 1 else 128)
                ks = ksplit or 1          # the split along K is opt-in: its workspace round trip costs more than it saves so far
                while ks > 1 and tiles * ks * 128 * tok * 4 > self.WIDE_WS_BYTES:
                    ks -= 1
                if ks > 1:
                    if self._wide_ws is None:
                        self._wide_ws = torch.empty(self.WIDE_WS_BYTES, dtype=torch.uint8, device=self.device)
                        self._wide_ctr = torch.zeros(8192, dtype=torch.int32, device=self.device)
                    if tiles > self._wide_ctr.numel():
                        ks = 1
                    ws, ctr = self._wide_ws, self._wide_ctr
            self._check(self.lib.blz_gemm_wide(kind, _ptr(a), lda, _ptr(w), ldb, _ptr(out), out.stride(0), M, lin.N, lin.K,
                                               _ptr(rs), _ptr(pk["alpha"]), _ptr(pk["bias"]), _ptr(sfa), _ptr(pk["sf"]),
                                               int(f32), int(swap), ks, _ptr(ws), self.WIDE_WS_BYTES if ws is not None else 0,
                                               _ptr(ctr), max_ctas, kt, act, limit, self._stream()), f"gemm_wide kind {kind}")
            return out
        if argmax_parts is not None:
            rc = self.lib.blz_gemm_argmax_parts(_ptr(argmax_parts[0]), _ptr(argmax_parts[1]))
            if rc != 0:
                raise CudaError(f"blz_gemm_argmax_parts failed: {rc}")
        self._check(self.lib.blz_gemm_tc(kind, _ptr(a), lda, _ptr(w), ldb, _ptr(out), ld_out, M, lin.N, lin.K,
                                         _ptr(rs), _ptr(pk["alpha"]), _ptr(pk["bias"]), _ptr(sfa), _ptr(pk["sf"]),
                                         int(f32), bn, max_ctas, VP(0), 0, kt, act, limit, self._stream()), f"gemm kind {kind}")
        return out

    def silu_mul(self, gu, quant_for: Optional[Linear] = None):
        T, I2 = gu.shape
        I = I2 // 2
        mode = self._qmode(quant_for)
        if mode == 0:
            out = torch.empty(T, I, dtype=torch.bfloat16, device=self.device)
            self._check(self.lib.blz_swiglu(_ptr(gu), _ptr(out), VP(0), VP(0), VP(0), T, I, 0, 0, self._stream()), "swiglu")
            return out
        qa = self._alloc_qact(Format.NVFP4 if mode == 1 else Format.MXFP8, T, I)
        self._check(self.lib.blz_swiglu(_ptr(gu), VP(0), _ptr(qa.data), _ptr(qa.sf), _ptr(qa.row_scale), T, I, mode, 0,
                                        self._stream()), "swiglu_q")
        return qa

    def mul_sigmoid(self, x, gate):
        x = x.contiguous()
        self._check(self.lib.blz_mul_sigmoid(_ptr(x), _ptr(gate.contiguous()), x.numel(), self._stream()), "mul_sigmoid")
        return x

    def add(self, a, b):
        out = torch.empty_like(a)
        self._check(self.lib.blz_add(_ptr(a), _ptr(b), _ptr(out), a.numel(), self._stream()), "add")
        return out

    def add_sigmoid_scaled(self, a, b, gate_logit):
        out = torch.empty_like(a)
        self._check(self.lib.blz_add_sigmoid_scaled(_ptr(a), _ptr(b), _ptr(gate_logit.contiguous()), _ptr(out), a.shape[0],
                                                    a.shape[1], self._stream()), "add_sigmoid_scaled")
        return out

    def gather_rows(self, x, rows):
        R, H = rows.numel(), x.shape[1]
        out = torch.empty(R, H, dtype=x.dtype, device=self.device)
        self._check(self.lib.blz_gather_rows(_ptr(x), _ptr(rows), _ptr(out), R, H, self._stream()), "gather_rows")
        return out

    def all_reduce(self, x, group=None):
        if group is None or group.world == 1:
            return x
        return group.all_reduce(x)

    # ------------------------------------------------------------------ attention
    def rope_tables(self, model, batch):
        return None   # angles are computed inside the prep kernel

    def attn_prep_store(self, qkv, attn, model, batch, kv, layer_idx, rope):
        cfg = model.cfg
        T = qkv.shape[0]
        D = cfg.head_dim
        if kv.layout != "umma":
            raise CudaError("the CUDA attention path needs the FP8 'umma' KV layout (kv_dtype='fp8')")
        q = torch.empty(T, attn.heads, D, dtype=torch.bfloat16, device=self.device)
        gate = torch.empty(T, attn.heads, D, dtype=torch.bfloat16, device=self.device) if cfg.attn_output_gate else None
        # M-RoPE: three position streams [3, T]; frequency i reads stream 0 / 1 / 2 by the model's section sizes
        pos, pos_stride, m0, m1 = batch.positions, 0, 0, 0
        sec = cfg.rope.mrope_section
        if getattr(batch, "positions3", None) is not None:
            pos, pos_stride = batch.positions3, batch.positions3.stride(0)
            if sec:
                m0, m1 = int(sec[0]), int(sec[0]) + int(sec[1])
            else:
                m0 = m1 = cfg.rotary_dim // 2          # no sections: every frequency follows the first stream
        self._check(self.lib.blz_attn_prep(_ptr(qkv), _ptr(q), _ptr(gate), _ptr(kv.kv[layer_idx]), _ptr(pos),
                                           _ptr(batch.slot_mapping), _ptr(model.inv_freq), _ptr(attn.q_norm), _ptr(attn.k_norm),
                                           T, attn.heads, attn.kv_heads, D, cfg.rotary_dim, cfg.rms_norm_eps,
                                           model.rope_scale, int(cfg.attn_output_gate), int(cfg.zero_centered_norm),
                                           1.0, 1.0, kv.kv[layer_idx].stride(0), kv.kv[layer_idx].stride(1),
                                           int(getattr(model, "kv_rotate", False)), pos_stride, m0, m1, self._stream()),
                    "attn_prep")
        return q, gate

    def kv_move_rows(self, pool, src, dst, seg, D):
        """Move KV rows between flat slots of one layer's pool (kernel page layout); ``seg`` = per-sequence move ranges."""
        self._check(self.lib.blz_kv_move_rows(_ptr(pool), _ptr(src), _ptr(dst), _ptr(seg), seg.numel() - 1, pool.shape[1], D,
                                              pool.stride(0), pool.stride(1), self._stream()), "kv_move_rows")

    def attention(self, q, model, batch, kv, layer_idx, scale, splits: int = 0, max_ctas: int = 0, allowed=None):
        """Sequences with few query rows (decode, verify) go to the decode kernel, the rest to the row-block kernel."""
        if allowed is not None:
            # a sparse selection (a context beyond an indexer's budget): the kernels read every key of a sequence, so these
            # steps take the masked torch attention over the pages on this device (correct, not fast)
            from . import ref
            kl, vl = kv.logical_kv(layer_idx)
            o = ref.paged_attention(q, kl, vl, kv.block_table, batch.h_slots, batch.h_q_start, batch.h_ctx_len, scale,
                                    tree_mask=getattr(batch, "tree_mask", None), allowed=allowed)
            return o.reshape(q.shape[0], -1).contiguous()
        T, Hq, D = q.shape
        Hkv = kv.kv_heads
        group = Hq // Hkv
        out = torch.empty(T, Hq, D, dtype=torch.bfloat16, device=self.device)
        B = batch.slots.numel()
        tiles = max((batch.max_ctx + 127) // 128, 1)
        # the decode kernel runs once per row tier: plain decode rows (<= 8 rows per kv head) take its two-CTAs-per-SM
        # configuration, short multi-token sequences (verify rows, prompt tails) the wider one
        tiers = []
        if D != 128:
            # the decode kernel is built for head_dim 128: every sequence is a row-block item here (engine.attn_all_items)
            if batch.item_seq is None or batch.tiny_rows_max or batch.small_rows_max:
                raise CudaError(f"head_dim {D}: the batch must send every sequence to the row-block attention kernel")
            if getattr(batch, "tree_mask", None) is not None:
                raise CudaError(f"head_dim {D}: draft trees are verified by the decode kernel, which covers head_dim 128 only")
        if batch.tiny_rows_max:
            tiers.append((1, batch.tiny_rows_max, batch.num_tiny))
        if batch.small_rows_max:
            tiers.append((batch.tiny_rows_max + 1 if batch.tiny_rows_max else 1, batch.small_rows_max, batch.num_small))
        if not tiers and not batch.num_large and D == 128:
            tiers.append((1, group * batch.max_q_len, B))
        for lo, hi, count in tiers:
            nmax = 16
            rb = (hi + nmax - 1) // nmax
            work = max(count, 1) * Hkv * rb
            sp = splits if splits > 0 else (1 if work >= 3 * self._sm else max(1, min(8, tiles, (3 * self._sm) // max(work, 1))))
            po = pm = None
            if sp > 1:
                n = B * Hkv * rb * sp * nmax
                po = self._buf("attn_part_o", n * D * 4).view(torch.float32)
                pm = self._buf("attn_part_ml", n * 2 * 4).view(torch.float32)
            self._check(self.lib.blz_attn_decode_tree(_ptr(q), _ptr(out), _ptr(kv.kv[layer_idx]), _ptr(kv.block_table),
                                                 _ptr(batch.slots), _ptr(batch.q_start), _ptr(batch.ctx_len), B, Hq, Hkv, D,
                                                 kv.block_table.stride(0), kv.kv[layer_idx].stride(0), kv.kv[layer_idx].stride(1),
                                                 scale, 1.0, 1.0, nmax, rb, lo, hi, sp,
                                                 _ptr(po), _ptr(pm), max_ctas, _ptr(self.attn_prof),
                                                 _ptr(getattr(batch, "tree_mask", None)), self._stream()), "attn_decode")
            if sp > 1:
                self.launches += 1
        if batch.item_seq is not None:
            n_items = batch.item_seq.numel()
            work = n_items * Hkv
            sp = splits if splits > 0 else (1 if work >= self._sm else max(1, min(8, tiles, self._sm // max(work, 1))))
            po = pm = None
            if sp > 1:
                n = work * sp * 128
                po = self._buf("attn_part_o2", n * D * 4).view(torch.float32)
                pm = self._buf("attn_part_ml2", n * 2 * 4).view(torch.float32)
            self._check(self.lib.blz_attn_tc(_ptr(q), _ptr(out), _ptr(kv.kv[layer_idx]), _ptr(kv.block_table),
                                             _ptr(batch.slots), _ptr(batch.q_start), _ptr(batch.ctx_len), _ptr(batch.item_seq),
                                             _ptr(batch.item_q0), n_items, Hq, Hkv, D, kv.block_table.stride(0), kv.kv[layer_idx].stride(0),
                                             kv.kv[layer_idx].stride(1), scale, 1.0,
                                             1.0, sp, _ptr(po), _ptr(pm), max_ctas, self._stream()), "attn_prefill")
            if sp > 1:
                self.launches += 1
        return out.view(T, Hq * D)

    # ------------------------------------------------------------------ static residual streams
    def streams_begin(self, table, tokens, scale: float, n: int):
        """All ``n`` streams equal to the scaled embedding rows (read from the table where they are needed, not copied)."""
        return (table, tokens, scale, n)

    def _streams(self, src, y, prev, nxt, norm_w, eps, T, W, want_sum: bool, keep: bool):
        from_embed = isinstance(src, tuple)
        dt = torch.float32 if (src[0] if from_embed else y).dtype == torch.float32 else torch.bfloat16
        if from_embed:
            table, tokens, scale, S = src
            streams = torch.empty(T, S, W, dtype=torch.float32, device=self.device) if keep else None
        else:
            table, tokens, scale, streams = None, None, 1.0, src
            S = src.shape[1]
        h = torch.empty(T, W, dtype=dt, device=self.device) if nxt is not None else None
        total = torch.empty(T, W, dtype=torch.float32, device=self.device) if want_sum else None
        self._check(self.lib.blz_streams(_ptr(streams), _ptr(table), _ptr(tokens), table.shape[0] if from_embed else 0, scale, _ptr(y),
                                         _ptr(prev.mix if prev is not None else None), _ptr(prev.out if prev is not None else None),
                                         _ptr(nxt.read if nxt is not None else None), _ptr(norm_w), eps, _ptr(h), _ptr(total), T, S, W,
                                         int(from_embed), int(keep), int(dt == torch.float32), self._stream()), "streams")
        return streams if keep else src, h, total

    def streams_step(self, src, y, prev, nxt, norm_w, eps):
        """Write the last sublayer's output ``y`` through ``prev``'s mix into the streams (``y`` None: there was none yet), then read
        and normalise the next sublayer's input; returns (streams, input)."""
        T, W = (src[1].numel(), src[0].shape[1]) if isinstance(src, tuple) else (src.shape[0], src.shape[2])
        streams, h, _ = self._streams(src, y, prev, nxt, norm_w, eps, T, W, False, y is not None)
        return streams, h

    def streams_sum(self, src, y, prev):
        """The sum of the streams after the sublayer whose output is ``y``, fp32 ``[T, W]``."""
        T, W = (src[1].numel(), src[0].shape[1]) if isinstance(src, tuple) else (src.shape[0], src.shape[2])
        return self._streams(src, y, prev, None, None, 0.0, T, W, True, False)[2]

    def norm_rows(self, x, rows, w, eps, dtype, centre: bool = False):
        """RMS norm (``centre``: layer norm) of fp32 rows (those named by ``rows``) to ``dtype``."""
        R = x.shape[0] if rows is None else rows.numel()
        out = torch.empty(R, x.shape[1], dtype=dtype, device=self.device)
        if R:
            rows = None if rows is None else rows.to(torch.int32)
            self._check(self.lib.blz_norm_rows(_ptr(x), _ptr(rows), _ptr(w), _ptr(out), R, x.shape[1], eps, int(centre),
                                               int(dtype == torch.float32), self._stream()), "norm_rows")
        return out

    # ------------------------------------------------------------------ differential attention
    SHORT_ROWS = 64            # sequences with new tokens * group up to this take the short-row kernel

    def diff_store(self, qkv, A, batch, kv, layer_idx):
        """The rows' keys and values into their pages."""
        a, pool = A.spec, kv.kv[layer_idx]
        if kv.layout != "tiles" or pool.dtype != qkv.dtype:
            raise CudaError(f"differential attention of {qkv.dtype} rows needs 'tiles' pages of that type")
        self._check(self.lib.blz_diff_store(_ptr(qkv), qkv.stride(0), _ptr(pool), pool.stride(0), pool.stride(1), _ptr(batch.slot_mapping),
                                            qkv.shape[0], a.heads, a.kv_heads, a.dim, a.vdim, int(qkv.dtype == torch.float32),
                                            self._stream()), "diff_store")

    def diff_attention(self, qkv, A, batch, kv, layer_idx, eps, store: bool = True):
        """Page write (``store``) and differential attention of one layer; ``[T, heads * vdim]``, every head normed and scaled."""
        a = A.spec
        T = qkv.shape[0]
        f32 = qkv.dtype == torch.float32
        pool = kv.kv[layer_idx]
        if store:
            self.diff_store(qkv, A, batch, kv, layer_idx)
        out = torch.empty(T, a.heads * a.vdim, dtype=qkv.dtype, device=self.device)
        B, bt = batch.slots.numel(), kv.block_table
        st = self._stream()
        common = (_ptr(qkv), qkv.stride(0), _ptr(out), _ptr(pool), pool.stride(0), pool.stride(1), _ptr(bt), bt.stride(0),
                  _ptr(batch.slots), _ptr(batch.q_start), _ptr(batch.ctx_len))
        shape = (T, B, a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.scale, A.lam, 1.0 - a.diff, eps)
        group = a.group
        if f32 or a.dim > 128 or a.vdim > 128 or group > 128 or a.scale <= 0:
            self._check(self.lib.blz_diff_plain(*common, _ptr(batch.seq_of_row), *shape, int(f32), st), "diff_plain")
            return out
        items, small = self._split_rows(batch, a)
        if items:
            self._check(self.lib.blz_diff_tc(*common, *shape, self.SHORT_ROWS, items, st), "diff_tc")
        if small:
            self._check(self.lib.blz_diff_short(*common, *shape, self.SHORT_ROWS, *small, st), "diff_short")
        return out

    def _split_rows(self, batch, a):
        """How a step's sequences are shared out between the page attention kernels: row blocks for the prompt kernel, and (row
        blocks, key splits, workspaces) of the short-row kernel or None."""
        group, B, limit = a.group, batch.slots.numel(), self.SHORT_ROWS
        lens = [b - s for s, b in zip(batch.h_q_start, batch.h_q_start[1:])]
        small = [n * group for n in lens if 0 < n * group <= limit]
        per = (128 // group) * (1 if a.maps == 2 else 2)
        items = sum(-(-n // per) for n in lens if n * group > limit)
        if not small:
            return items, None
        rb = (max(small) + 15) // 16
        toks = (max(small) + group - 1) // group
        keys = min(batch.max_ctx, a.window + toks - 1) if a.window else batch.max_ctx
        work = len(small) * a.kv_heads * rb
        sp = max(1, min(4 * self._sm // work, (keys + 127) // 128, 32))
        po = pm = None
        if sp > 1:
            n = B * a.kv_heads * rb * sp * 16 * a.maps
            po = self._buf("maps_part_o", n * 128 * 4).view(torch.float32)
            pm = self._buf("maps_part_ml", n * 2 * 4).view(torch.float32)
            self.launches += 1
        return items, (rb, sp, _ptr(po), _ptr(pm))

    # ------------------------------------------------------------------ post-norm residual, gated softmax attention, recurrences
    def residual_norm(self, x, alpha: float, y, w, eps):
        """``norm(alpha * x + y)`` in fp32 (in place of an fp32 ``x``), and the same in y's type."""
        T, W = y.shape
        f32 = y.dtype == torch.float32
        dst = torch.empty(T, W, dtype=torch.float32, device=self.device) if x.dtype != torch.float32 else x
        h = dst if f32 else torch.empty_like(y)
        if T:
            self._check(self.lib.blz_residual_norm(_ptr(x), int(x.dtype != torch.float32), alpha, _ptr(y), _ptr(w), eps, _ptr(dst),
                                                   VP(0) if f32 else _ptr(h), T, W, int(f32), self._stream()), "residual_norm")
        return dst, h

    def attn_prep_pages(self, proj, M, batch, kv, layer_idx, eps):
        """Rotated and normalised queries ``[T, heads * dim]`` of a mixer; its keys and values go to their pages."""
        A, a, pool, c = M.attn, M.attn.spec, kv.kv[layer_idx], M.cols
        if kv.layout != "tiles" or pool.dtype != proj.dtype:
            raise CudaError(f"attention of {proj.dtype} rows needs 'tiles' pages of that type")
        T = proj.shape[0]
        q = torch.empty(T, a.heads * a.dim, dtype=proj.dtype, device=self.device)
        rot = a.rot.dims if a.rot is not None else 0
        self._check(self.lib.blz_attn_prep_pages(_ptr(proj), proj.stride(0), c["q"], c["k"], c["v"], _ptr(q), _ptr(pool), pool.stride(0),
                                                 pool.stride(1), _ptr(batch.positions), _ptr(batch.slot_mapping), _ptr(A.freq), T, a.heads,
                                                 a.kv_heads, a.dim, a.vdim, rot, int(rot > 0 and a.rot.interleaved), int(a.unit_rms), eps,
                                                 int(proj.dtype == torch.float32), self._stream()), "attn_prep_pages")
        return q

    def soft_attention(self, proj, M, batch, kv, layer_idx, eps, out):
        """Softmax attention of a mixer (page write included), gated and scaled, into ``out`` (columns of a wider matrix)."""
        self.soft_attend(self.attn_prep_pages(proj, M, batch, kv, layer_idx, eps), proj, M, batch, kv, layer_idx, out)

    def soft_attend(self, q, proj, M, batch, kv, layer_idx, out):
        A, a, pool, bt = M.attn, M.attn.spec, kv.kv[layer_idx], kv.block_table
        T, B, f32, st = q.shape[0], batch.slots.numel(), q.dtype == torch.float32, self._stream()
        gate = VP(proj.data_ptr() + M.cols["gate"] * proj.element_size()) if a.gate else VP(0)
        common = (_ptr(q), q.stride(0), _ptr(out), out.stride(0), _ptr(pool), pool.stride(0), pool.stride(1), _ptr(bt), bt.stride(0),
                  _ptr(batch.slots), _ptr(batch.q_start), _ptr(batch.ctx_len), _ptr(A.sink), gate, proj.stride(0))
        shape = (T, B, a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.scale, a.out_scale)
        if f32 or a.dim > 128 or a.vdim > 128 or a.group > 128 or a.scale <= 0:
            self._check(self.lib.blz_soft_plain(*common, _ptr(batch.seq_of_row), *shape, int(f32), st), "soft_plain")
            return
        items, small = self._split_rows(batch, a)
        if items:
            self._check(self.lib.blz_soft_tc(*common, *shape, self.SHORT_ROWS, items, VP(0), st), "soft_tc")
        if small:
            self._check(self.lib.blz_soft_short(*common, *shape, self.SHORT_ROWS, *small, st), "soft_short")

    def short_conv(self, proj, M, batch, kv, layer_idx):
        """Causal convolution and SiLU of a mixer's recurrent inputs ``[T, conv_dim]``; advances its history."""
        R, r, T = M.rec, M.rec.spec, proj.shape[0]
        y = torch.empty(T, r.conv_dim, dtype=proj.dtype, device=self.device)
        src = VP(proj.data_ptr() + M.cols["conv"] * proj.element_size())
        self._check(self.lib.blz_short_conv(src, proj.stride(0), _ptr(y), _ptr(kv.conv_state[layer_idx]), _ptr(R.conv_w), _ptr(R.conv_b),
                                            _ptr(batch.slots), _ptr(batch.q_start), _ptr(batch.ctx_len), _ptr(batch.gdn_defer),
                                            batch.slots.numel(), r.conv_dim, r.conv, int(batch.max_q_len), int(proj.dtype == torch.float32),
                                            self._stream()), "short_conv")
        return y

    def recurrence(self, proj, low, M, batch, kv, layer_idx, eps, out, state_only: bool = False):
        """The recurrent mixer of a layer: convolution, recurrence, gated norm into ``out`` (columns of a wider matrix).  Sequences
        flagged in ``batch.gdn_defer`` leave their state untouched; ``state_only`` advances the states and writes nothing."""
        R, r, T = M.rec, M.rec.spec, proj.shape[0]
        if R.kind == "mingru":
            self.min_gru(proj, M, batch, kv, layer_idx, None if state_only else out)
            return
        y = self.short_conv(proj, M, batch, kv, layer_idx) if r.conv else None
        o = None if state_only else torch.empty(T, r.heads * r.vdim, dtype=torch.float32, device=self.device)
        self.recur(y, proj, low, M, batch, kv, layer_idx, o)
        if state_only:
            return
        self.gated_norm(o, low if low is not None else proj, M, eps, out)

    def min_gru(self, proj, M, batch, kv, layer_idx, out):
        """Elementwise gated recurrence with its output gate, into ``out`` (None: the state only)."""
        r, es = M.rec.spec, proj.element_size()
        z, u, g = [VP(proj.data_ptr() + M.cols[c] * es) for c in ("zg", "u", "g")]
        lens = [e - s for s, e in zip(batch.h_q_start, batch.h_q_start[1:])]
        kinds = (1 if 1 in lens else 0) | (2 if batch.max_q_len > 1 else 0)
        ws_bytes = int(self.lib.blz_min_gru_ws_bytes(len(lens), int(batch.max_q_len), r.width)) if kinds & 2 else 0
        ws = torch.empty(ws_bytes, dtype=torch.uint8, device=self.device) if ws_bytes else None
        self.launches += int(kinds == 3) + int(ws is not None)
        self._check(self.lib.blz_min_gru(z, u, g, proj.stride(0), _ptr(kv.rec_state[layer_idx]), _ptr(out), out.stride(0) if out is not None else 0,
                                         _ptr(batch.slots), _ptr(batch.q_start), _ptr(batch.ctx_len), _ptr(batch.gdn_defer),
                                         batch.slots.numel(), r.width, int(batch.max_q_len), kinds, _ptr(ws), int(es == 4), self._stream()),
                    "min_gru")

    def gated_norm(self, o, gates, M, eps, out):
        """The norm and gate of a recurrence's rows ``o``; ``gates`` holds the gate's columns: the low-rank outputs (delta rule with channel
        decays), or the input projection (gated linear attention has none)."""
        R, r, es = M.rec, M.rec.spec, gates.element_size()
        delta = R.kind == "delta"
        z = VP(0) if R.kind == "gated" else VP(gates.data_ptr() + (r.heads * r.dim if delta and not r.head_decay else M.cols["z"]) * es)
        self._check(self.lib.blz_group_norm(_ptr(o), z, gates.stride(0), _ptr(R.norm_w), _ptr(out), out.stride(0), o.shape[0], R.norm_groups,
                                            o.shape[1] // R.norm_groups, R.norm_w.numel(), eps, r.out_scale,
                                            int(delta and r.gate == "sigmoid"), int(not delta),
                                            int(es == 4), self._stream()), "group_norm")

    REC_MAX_WS = 4 << 30       # workspace of the streaming recurrences; steps that need more run without it

    def recur(self, y, proj, low, M, batch, kv, layer_idx, o):
        """The recurrence alone: convolved inputs ``y`` (gated linear attention: None) to fp32 rows ``o`` (None: the state only)."""
        R, r, es, f32 = M.rec, M.rec.spec, proj.element_size(), int(proj.dtype == torch.float32)
        seqs = (_ptr(batch.slots), _ptr(batch.q_start), _ptr(batch.ctx_len), _ptr(batch.gdn_defer), batch.slots.numel())
        state, st, longest, T = kv.rec_state[layer_idx], self._stream(), int(batch.max_q_len), proj.shape[0]
        delta, gated = R.kind == "delta", R.kind == "gated"
        groups = r.kv_heads if delta else r.heads if gated else r.groups
        # which kernels the step needs: single tokens, short runs, and long runs, which read what a token needs from a workspace
        # filled for all tokens at once
        lens = [e - s for s, e in zip(batch.h_q_start, batch.h_q_start[1:])]
        long_rows, ws, ws_bytes = int(self.lib.blz_rec_long_rows()), None, 0
        kinds = (1 if 1 in lens else 0) | (2 if any(1 < n < long_rows for n in lens) else 0)
        if longest >= long_rows:
            ws_bytes = int(self.lib.blz_rec_ws_bytes(2 if gated else 3 if delta and r.head_decay else int(delta), T, r.heads, groups, r.state))
            if o is not None and ws_bytes <= self.REC_MAX_WS:
                ws = torch.empty(ws_bytes, dtype=torch.uint8, device=self.device)
                kinds |= 4
            else:
                kinds |= 2
        self.launches += (0, 0, 0, 1, 1, 2, 2, 3)[kinds]
        runs = (_ptr(batch.seq_of_row), T, kinds, _ptr(ws), ws_bytes, f32, st)
        if gated:
            at = [VP(proj.data_ptr() + M.cols[c] * es) for c in ("q", "f", "v")]
            ld = proj.stride(0)
            self._check(self.lib.blz_gated_linear(at[0], ld, at[1], ld, at[2], ld, _ptr(R.A), _ptr(R.dt_bias), _ptr(state), _ptr(o), *seqs,
                                                  r.heads, r.dim, r.vdim, *runs), "gated_linear")
        elif delta:
            decay, ld = (VP(proj.data_ptr() + M.cols["decay"] * es), proj.stride(0)) if r.head_decay else (_ptr(low), low.stride(0))
            self._check(self.lib.blz_delta_rule(_ptr(y), y.stride(0), decay, ld, VP(proj.data_ptr() + M.cols["beta"] * es),
                                                proj.stride(0), _ptr(R.A), _ptr(R.dt_bias), _ptr(state), _ptr(o), *seqs, r.heads,
                                                r.kv_heads, r.dim, r.vdim, int(r.head_decay), *runs), "delta_rule")
        else:
            self._check(self.lib.blz_state_space(_ptr(y), y.stride(0), VP(proj.data_ptr() + M.cols["dt"] * es), proj.stride(0), _ptr(R.A),
                                                 _ptr(R.dt_bias), _ptr(R.D), _ptr(state), _ptr(o), *seqs, r.heads, r.groups, r.state,
                                                 r.vdim, *runs), "state_space")

    # ------------------------------------------------------------------ residual with normed branches, input convolution
    def embed_norm(self, table, tokens, w, eps):
        """Layer-normed embedding rows, fp32."""
        T, W = tokens.numel(), table.shape[1]
        x = torch.empty(T, W, dtype=torch.float32, device=self.device)
        if T:
            self._check(self.lib.blz_embed_norm(_ptr(table), _ptr(tokens), table.shape[0], _ptr(w), eps, _ptr(x), T, W,
                                                int(table.dtype == torch.float32), self._stream()), "embed_norm")
        return x

    def branch_norm(self, x, y, w, eps, copy: bool = True):
        """``x + layer_norm(y)`` in place of the fp32 rows ``x``, and the same in y's type (``copy``; else None).  ``y`` may be routed
        rows (:meth:`moe_rows`), which are summed up on the way."""
        T, W = x.shape
        routed = isinstance(y, RoutedRows)
        rows = y.rows if routed else y
        f32 = rows.dtype == torch.float32
        h = None if not copy else x if f32 else torch.empty(T, W, dtype=rows.dtype, device=self.device)
        if T:
            how = (_ptr(y.weights), _ptr(y.row_map), y.row_map.shape[1], _ptr(y.extra)) if routed else (VP(0), VP(0), 0, VP(0))
            self._check(self.lib.blz_branch_norm(_ptr(rows), rows.stride(0), *how, _ptr(w), eps, _ptr(x), VP(0) if f32 else _ptr(h), T, W,
                                                 int(f32), self._stream()), "branch_norm")
        return x, h

    def input_conv(self, x, w, batch, kv, layer_idx, dtype, state_only: bool = False):
        """``x + conv(x)`` of fp32 rows in ``dtype``, with the inputs before each sequence's rows from its state row, which advances
        (not for sequences flagged in ``batch.gdn_defer``)."""
        T, W = x.shape
        h = None if state_only else torch.empty(T, W, dtype=dtype, device=self.device)
        if h is not None and T > batch.h_q_start[-1]:
            h[batch.h_q_start[-1]:].zero_()                  # padding rows
        if T:
            self._check(self.lib.blz_input_conv(_ptr(x), _ptr(h), _ptr(kv.input_state.get(layer_idx)), _ptr(w), _ptr(batch.slots),
                                                _ptr(batch.q_start), _ptr(batch.ctx_len), _ptr(batch.gdn_defer), batch.slots.numel(), W,
                                                w.shape[0], int(batch.max_q_len), int(dtype == torch.float32), self._stream()), "input_conv")
            if batch.max_q_len > 32:
                self.launches += 1
        return h

    # ------------------------------------------------------------------ mixer and feed-forward side by side, sigmoid attention
    def embed_positions(self, table, tokens, positions, scale: float, freq, copy=None):
        """Scaled embedding rows plus their position's vector, fp32; ``copy`` (columns of a wider matrix) gets them in the table's type."""
        T, W = tokens.numel(), table.shape[1]
        x = torch.empty(T, W, dtype=torch.float32, device=self.device)
        if T:
            self._check(self.lib.blz_embed_positions(_ptr(table), _ptr(tokens), _ptr(positions), _ptr(freq), table.shape[0], scale, _ptr(x),
                                                     _ptr(copy), copy.stride(0) if copy is not None else 0, T, W,
                                                     int(table.dtype == torch.float32), self._stream()), "embed_positions")
        return x

    def branch_step(self, x, br, eps, dtype, w1=None, w2=None, copy=None):
        """Add a layer's branches (None: nothing) to the fp32 rows ``x`` in place; then their RMS norms with the weights ``w1`` and ``w2``
        (None: no such norm) in ``dtype``.  ``copy`` (columns of a wider matrix) gets the rows in ``dtype``.  (rows, norm 1, norm 2)"""
        T, W = x.shape
        h1, h2 = [None if w is None else torch.empty(T, W, dtype=dtype, device=self.device) for w in (w1, w2)]
        if not T:
            return x, h1, h2
        y1 = y2 = m1 = m2 = ffn = None
        mult = 0.0
        if br is not None:
            mult, ffn = br.mult, br.ffn
            (y1, y2), (m1, m2) = (br.rows, br.norms) if br.norms is not None else ((br.rows, None), (None, None))
        routed = (_ptr(ffn.rows), ffn.rows.stride(0), _ptr(ffn.weights), _ptr(ffn.row_map), ffn.row_map.shape[1], _ptr(ffn.extra),
                  _ptr(ffn.gate), ffn.gate.stride(0) if ffn.gate is not None else 0) if ffn is not None else (VP(0), 0, VP(0), VP(0), 0, VP(0), VP(0), 0)
        self._check(self.lib.blz_branch_step(_ptr(x), _ptr(y1), _ptr(y2), _ptr(m1), _ptr(m2), *routed, _ptr(w1), _ptr(w2), _ptr(h1), _ptr(h2),
                                             _ptr(copy), copy.stride(0) if copy is not None else 0, mult, eps, T, W,
                                             int(dtype == torch.float32), self._stream()), "branch_step")
        return x, h1, h2

    def conv_prep_pages(self, proj, M, batch, kv, layer_idx, eps, state_only: bool = False):
        """Convolved queries ``[T, heads * dim]`` of a sigmoid attention (times their position's temperature); its convolved keys and
        (normed) values go to their pages, and the convolution's history advances.  ``state_only``: only that."""
        A, a, pool, c, T = M.attn, M.attn.spec, kv.kv[layer_idx], M.cols, proj.shape[0]
        if kv.layout != "tiles" or pool.dtype != proj.dtype:
            raise CudaError(f"attention of {proj.dtype} rows needs 'tiles' pages of that type")
        q = None if state_only else torch.empty(T, a.heads * a.dim, dtype=proj.dtype, device=self.device)
        self._check(self.lib.blz_conv_prep_pages(_ptr(proj), proj.stride(0), c["q"], c["k"], c["v"], _ptr(q), _ptr(pool), pool.stride(0),
                                                 pool.stride(1), _ptr(batch.positions), _ptr(batch.slot_mapping), _ptr(A.conv_w),
                                                 _ptr(kv.qkv_state.get(layer_idx)), _ptr(batch.slots), _ptr(batch.q_start), _ptr(batch.ctx_len),
                                                 _ptr(batch.gdn_defer), batch.slots.numel(), int(batch.max_q_len), T, a.heads, a.kv_heads,
                                                 a.dim, a.vdim, max(a.conv, 1), int(a.unit_v), a.temp_coef, a.temp_every, eps, int(state_only),
                                                 int(proj.dtype == torch.float32), self._stream()), "conv_prep_pages")
        return q

    def sigmoid_attention(self, proj, M, batch, kv, layer_idx, eps, out, state_only: bool = False):
        """Sigmoid attention of a mixer (convolution, value norm and page write included) into ``out`` (columns of a wider matrix).
        ``state_only`` advances the convolution's history and does nothing else."""
        q = self.conv_prep_pages(proj, M, batch, kv, layer_idx, eps, state_only)
        if not state_only:
            self.sigmoid_attend(q, M, batch, kv, layer_idx, out)

    def sigmoid_attend(self, q, M, batch, kv, layer_idx, out):
        A, a, pool, bt = M.attn, M.attn.spec, kv.kv[layer_idx], kv.block_table
        T, B, f32, st = q.shape[0], batch.slots.numel(), q.dtype == torch.float32, self._stream()
        plain = f32 or a.dim > 128 or a.vdim > 128 or a.group > 128 or a.scale <= 0
        common = (_ptr(q), q.stride(0), _ptr(out), out.stride(0), _ptr(pool), pool.stride(0), pool.stride(1), _ptr(bt), bt.stride(0),
                  _ptr(batch.slots), _ptr(batch.q_start), _ptr(batch.ctx_len), _ptr(A.bias if plain else A.bias_ex2), A.reach)
        shape = (T, B, a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.scale, a.out_scale)
        if plain:
            self._check(self.lib.blz_sigmoid_plain(*common, _ptr(batch.seq_of_row), *shape, int(f32), st), "sigmoid_plain")
            return
        items, small = self._split_rows(batch, a)
        if items:
            self._check(self.lib.blz_sigmoid_tc(*common, *shape, self.SHORT_ROWS, items, st), "sigmoid_tc")
        if small:
            self._check(self.lib.blz_sigmoid_short(*common, *shape, self.SHORT_ROWS, *small, st), "sigmoid_short")

    # ------------------------------------------------------------------ feed-forwards without a gate
    def relu2_(self, z, row_list=None):
        """``relu(z)^2`` in place, of all rows or of those named by ``row_list`` (-1: none)."""
        n = z.shape[0] if row_list is None else row_list.numel()
        if n:
            self._check(self.lib.blz_relu2(_ptr(z), z.shape[1], _ptr(row_list), n, int(z.dtype == torch.float32), self._stream()), "relu2")
        return z

    def linear_relu2(self, lin: Linear, x):
        if lin.fmt != Format.DENSE or lin.w.dtype == torch.float32 or lin.K % 16:
            return self.relu2_(self.linear(lin, x))
        return self.linear(lin, x, relu2=True)

    def poly_norm(self, z, act, eps):
        out = torch.empty_like(z)
        if z.shape[0]:
            self._check(self.lib.blz_poly_norm(_ptr(z), _ptr(act), _ptr(out), z.shape[0], z.shape[1], eps, int(z.dtype == torch.float32),
                                               self._stream()), "poly_norm")
        return out

    # ------------------------------------------------------------------ latent attention
    LATENT_BLOCK = 64          # query rows per CTA of the kernel over the latents, at most
    LATENT_SHORT = 16          # new tokens up to which a sequence's queries are mapped to the latents instead of the latents to keys

    def latent_attention(self, proj, M, batch, kv, layer_idx, eps, out):
        """Latent attention of a mixer: its own latents go to their pages, the heads' outputs (before the output projection) to ``out``."""
        q = self.latent_queries(proj, M, batch, kv, layer_idx, eps)
        self.latent_attend(q, M, batch, kv, layer_idx, out)

    def latent_queries(self, proj, M, batch, kv, layer_idx, eps):
        """Page write, and the queries ``[T, heads * (dim + rot_dim)]`` before their rotation."""
        return self.linear(M.attn.uq, self.latent_prep(proj, M, batch, kv, layer_idx, eps))

    def latent_prep(self, proj, M, batch, kv, layer_idx, eps):
        """The queries' normed latents; the keys' (where the layer has its own) with their rotated part go to their pages."""
        A, a, T, pool = M.attn, M.attn.spec, proj.shape[0], kv.kv[layer_idx]
        if kv.layout != "tiles" or pool.dtype != proj.dtype:
            raise CudaError(f"latent attention of {proj.dtype} rows needs 'tiles' pages of that type")
        own = a.kv_from is None
        lat = torch.empty(T, a.q_rank, dtype=proj.dtype, device=self.device)
        self._check(self.lib.blz_latent_prep(_ptr(proj), proj.stride(0), M.cols["q"], M.cols.get("kv", 0), _ptr(lat),
                                             _ptr(pool) if own else VP(0), pool.stride(0), _ptr(A.q_norm), _ptr(A.c_norm), _ptr(A.freq),
                                             _ptr(batch.positions), _ptr(batch.slot_mapping), T, a.q_rank, a.kv_rank, a.rot_dim,
                                             a.rot.dims if a.rot is not None else 0, eps, int(proj.dtype == torch.float32), self._stream()),
                    "latent_prep")
        return lat

    def latent_attend(self, q, M, batch, kv, layer_idx, out):
        """Rotation and attention of the queries.  Sequences with many new tokens go by head where the prompt kernel covers the
        sizes, all the others over the latents."""
        A, a = M.attn, M.attn.spec
        T, H, f32 = q.shape[0], a.heads, q.dtype == torch.float32
        lens = [e - s for s, e in zip(batch.h_q_start, batch.h_q_start[1:])]
        wide = not f32 and a.scale > 0 and a.vdim <= 128 and a.dim + a.rot_dim <= 192
        most = self.LATENT_SHORT if wide else max(batch.max_q_len, 1)
        longest = max((n for n in lens if n <= most), default=0)
        D = (a.kv_rank + 15) // 16 * 16 + (a.rot_dim + 15) // 16 * 16
        rows, rot = (_ptr(batch.seq_of_row), _ptr(batch.q_start)), a.rot.dims if a.rot is not None else 0
        if longest:
            qe = torch.empty(T, H, D, dtype=q.dtype, device=self.device)
            self._check(self.lib.blz_latent_map(_ptr(q), _ptr(A.uk_t), _ptr(qe), _ptr(A.freq), _ptr(batch.positions), T, H, a.dim, a.rot_dim, rot,
                                                a.kv_rank, *rows, most, int(f32), self._stream()), "latent_map")
            lat = torch.empty(T, H * a.kv_rank, dtype=q.dtype, device=self.device)
            self.latent_rows(qe, M, batch, kv, layer_idx, longest, most, lat)
            self._head_gemm(lat, a.kv_rank, A.uv, out, a.vdim, batch, most)
        if any(n > most for n in lens):
            if rot:
                self._check(self.lib.blz_latent_rot(_ptr(q), _ptr(A.freq), _ptr(batch.positions), *rows, T, H, a.dim, a.rot_dim, rot, most, int(f32),
                                                    self._stream()), "latent_rot")
            self._expanded_attention(q, M, batch, kv, self._expand_latents(M, batch, kv, layer_idx, most), most, out)

    def _head_gemm(self, x, x_head: int, w, y, y_head: int, batch, most: int):
        """``y[t, h] = w[h] x[t, h]`` for the sequences with at most ``most`` new tokens; ``*_head``: columns from head to head."""
        self._check(self.lib.blz_head_gemm(_ptr(x), x.stride(0), x_head, _ptr(w), _ptr(y), y.stride(0), y_head, x.shape[0], w.shape[1], w.shape[2],
                                           w.shape[0], _ptr(batch.seq_of_row), _ptr(batch.q_start), most, int(x.dtype == torch.float32),
                                           self._stream()), "head_gemm")

    def latent_rows(self, qe, M, batch, kv, layer_idx, longest: int, most: int, lat):
        """Weighted sums of the latents for the sequences with at most ``most`` new tokens (the longest has ``longest``)."""
        A, a, pool, bt = M.attn, M.attn.spec, kv.kv[layer_idx], kv.block_table
        T, H, D = qe.shape
        B, f32, st = batch.slots.numel(), qe.dtype == torch.float32, self._stream()
        seqs = (_ptr(bt), bt.stride(0), _ptr(batch.slots), _ptr(batch.q_start), _ptr(batch.ctx_len), _ptr(A.sink))
        per_sm = _c.c_int(1)
        R = 0 if f32 or a.scale <= 0 else int(self.lib.blz_latent_rows_block(a.kv_rank, a.rot_dim, min(longest * H, self.LATENT_BLOCK),
                                                                             _c.byref(per_sm)))
        if R == 0:
            self._check(self.lib.blz_shared_plain(_ptr(qe), H * D, _ptr(lat), H * a.kv_rank, _ptr(pool), pool.stride(0), *seqs,
                                                  _ptr(batch.seq_of_row), T, B, H, D, a.kv_rank, a.window, a.scale, int(f32), st), "shared_plain")
            return
        short = sum(1 for s, e in zip(batch.h_q_start, batch.h_q_start[1:]) if 0 < e - s <= most)
        rb = (longest * H + R - 1) // R
        keys = min(batch.max_ctx, a.window + (R + H - 1) // H) if a.window else batch.max_ctx
        sp = max(1, min(per_sm.value * self._sm // (short * rb), (keys + 127) // 128, 32))
        po = pm = None
        if sp > 1:
            n = B * rb * sp * R
            po, pm = self._buf("latent_part_o", n * a.kv_rank * 4), self._buf("latent_part_ml", n * 8)
            self.launches += 1
        self._check(self.lib.blz_latent_rows(_ptr(qe), _ptr(lat), _ptr(pool), pool.stride(0), *seqs, B, H, a.kv_rank, a.rot_dim, a.window, a.scale,
                                             most, longest, R, rb, sp, _ptr(po), _ptr(pm), st), "latent_rows")

    def _expand_latents(self, M, batch, kv, layer_idx, most: int):
        """Keys and values by head, as pages, of all tokens that the sequences with more than ``most`` new tokens see."""
        A, a, pool, st = M.attn, M.attn.spec, kv.kv[layer_idx], self._stream()
        pages, _, n, _ = self._visible_pages(batch, kv, a.window, most)
        lat = torch.empty(n * 16, a.kv_rank, dtype=pool.dtype, device=self.device)
        self._check(self.lib.blz_latent_gather(_ptr(pool), pool.stride(0), _ptr(pages), n, _ptr(lat), a.kv_rank, a.rot_dim, st), "latent_gather")
        kx = self.linear(A.expand, lat)
        block = 16 * ((a.dim + a.rot_dim + 15) // 16 * 16 + (a.vdim + 15) // 16 * 16)
        out = torch.empty(n, a.heads, block, dtype=pool.dtype, device=self.device)
        self._check(self.lib.blz_expand_store(_ptr(kx), kx.stride(0), _ptr(pool), pool.stride(0), _ptr(pages), _ptr(out), n, a.heads, a.dim,
                                              a.rot_dim, a.vdim, a.kv_rank, st), "expand_store")
        return out

    def _expanded_attention(self, q, M, batch, kv, pages, most: int, out):
        """Prompt attention of the sequences with more than ``most`` new tokens over the pages of :meth:`_expand_latents`."""
        A, a, bt = M.attn, M.attn.spec, kv.block_table
        _, base, _, items = self._visible_pages(batch, kv, a.window, most)
        self._check(self.lib.blz_soft_tc(_ptr(q), q.stride(0), _ptr(out), out.stride(0), _ptr(pages), pages.stride(0), pages.stride(1), _ptr(bt),
                                         bt.stride(0), _ptr(batch.slots), _ptr(batch.q_start), _ptr(batch.ctx_len), _ptr(A.sink), VP(0), 0,
                                         q.shape[0], batch.slots.numel(), a.heads, a.heads, a.dim + a.rot_dim, a.vdim, a.window, a.scale, 1.0, most,
                                         items, _ptr(base), self._stream()), "soft_tc")

    def _visible_pages(self, batch, kv, window: int, most: int):
        """(pages, page base of each sequence, number of pages, row blocks) of the sequences with more than ``most`` new tokens: the pages
        any of their rows sees, one sequence after the other.  Kept with the batch: its layers share them."""
        key = (window, most)
        hit = batch.visible.get(key)
        if hit is not None:
            return hit
        pages, base, items = [], [], 0
        for b, slot in enumerate(batch.h_slots):
            n, ctx = batch.h_q_start[b + 1] - batch.h_q_start[b], batch.h_ctx_len[b]
            lo = (max(ctx - n - window + 1, 0) if window else 0) // 16
            base.append(len(pages) - lo)
            if n > most:
                pages.extend(kv.block_table_host[slot, lo:(ctx + 15) // 16].tolist())
                items += -(-n // 256)
        dev = torch.tensor(base + pages, dtype=torch.int32).to(self.device)
        batch.visible[key] = hit = (dev[len(base):], dev[:len(base)], len(pages), items)
        return hit

    # ------------------------------------------------------------------ head
    def argmax(self, logits, index_offset: int = 0, want_values: bool = False):
        R, V = logits.shape
        out = torch.empty(R, dtype=torch.int64, device=self.device)
        vals = torch.empty(R, dtype=torch.float32, device=self.device) if want_values else None
        self._check(self.lib.blz_argmax(_ptr(logits), _ptr(out), _ptr(vals), R, V, logits.stride(0), index_offset,
                                        self._stream()), "argmax")
        return (out, vals) if want_values else out

    # ------------------------------------------------------------------ mixture of experts
    def router_topk(self, logits, k, renorm=True, first: int = 0, local_n: int = -1, sigmoid: bool = False, n_exp: Optional[int] = None):
        """Softmax (or sigmoids) → top-k → renormalise on the device; also counts the routed rows of each local expert.  ``n_exp``: the
        experts' logits are the first ``n_exp`` columns."""
        T, E = logits.shape[0], logits.shape[1] if n_exp is None else n_exp
        logits = logits if logits.stride(1) == 1 else logits.contiguous()
        local_n = E if local_n < 0 else local_n
        w = torch.empty(T, k, dtype=torch.float32, device=self.device)
        ids = torch.empty(T, k, dtype=torch.int32, device=self.device)
        counts = torch.empty(max(local_n, 1), dtype=torch.int32, device=self.device)
        self._check(self.lib.blz_moe_route(_ptr(logits), logits.stride(0), _ptr(w), _ptr(ids), _ptr(counts), T, E, k, int(renorm), int(sigmoid),
                                           first, local_n, self._stream()), "moe_route")
        self._route_counts = (counts, first, local_n)
        return w, ids

    def pack_experts(self, ex):
        """Stack the local experts' weights into two grouped-GEMM operands (gate_up and down)."""
        if ex.cuda_pack is not None:
            return ex.cuda_pack

        relu2, fused = ex.act == "relu2", ex.act == "swiglu" and ex.fused_act
        if (relu2 or fused) and (ex.gate_up[0].w.dtype == torch.float32 or ex.gate_up[0].K % 16):
            # 32-bit, or rows too ragged for TMA: the CUDA-core product
            def plain(lins):
                w = torch.stack([l.w for l in lins]).to(self.device).contiguous()
                return {"kind": 5, "w": w, "N": lins[0].N, "K": lins[0].K, "fmt": Format.DENSE, "act_quant": False}
            ex.cuda_pack = {"gate_up": plain(ex.gate_up), "down": plain(ex.down)}
            return ex.cuda_pack

        def padded(lins, n128, k128):
            """The grouped product's tiles are 128 rows of one expert's weight: pad those that are not (zeros stay zeros)."""
            N, K = lins[0].N, lins[0].K
            NP, KP = (N + 127) // 128 * 128 if n128 else N, (K + 127) // 128 * 128 if k128 else K
            if (NP, KP) == (N, K):
                return lins
            out = []
            for l in lins:
                w = l.w.new_zeros(NP, KP)
                w[:N, :K] = l.w
                out.append(Linear.from_dense(w, dtype=l.w.dtype))
            return out

        def stack(lins):
            pk0 = self.pack(lins[0], tiled=False, exact_fp8=False)
            kind = pk0["kind"]
            w = torch.cat([self.pack(l, tiled=False, exact_fp8=False)["w"] for l in lins])
            alpha = torch.cat([self.pack(l, tiled=False, exact_fp8=False)["alpha"] for l in lins]) if pk0["alpha"] is not None else None
            sf = None
            if kind in (1, 2):
                l0 = lins[0]
                if l0.N % 128:
                    raise CudaError("grouped GEMM needs expert output dims that are multiples of 128")
                per = l0.K // (16 if kind == 1 else 32)
                if kind == 1:
                    raw = torch.cat([l.sf.to(self.device).view(torch.uint8) for l in lins])
                else:
                    raw = torch.cat([quant.unswizzle_sf_128x4(self.pack(l, tiled=False, exact_fp8=False)["sf"], (l.N + 255) // 256 * 256, per)[:l.N] for l in lins])
                rows = (raw.shape[0] + 255) // 256 * 256
                buf = torch.zeros(rows, per, dtype=torch.uint8, device=self.device)
                buf[:raw.shape[0]] = raw
                sf = quant.swizzle_sf_128x4(buf)
            for l in lins:
                l.cuda_pack = None          # the stacked copy replaces the per-expert ones
            return {"kind": kind, "w": w.contiguous(), "sf": sf, "alpha": alpha, "N": lins[0].N, "K": lins[0].K,
                    "fmt": lins[0].fmt, "act_quant": lins[0].act_quant}
        if fused:
            # [gate | up] rows, each half rounded up to 64 features, in the order of the SwiGLU epilogue
            ff, K = ex.down[0].K, ex.gate_up[0].K
            fp = (ff + 63) // 64 * 64
            ws = []
            for l in ex.gate_up:
                w = l.w.new_zeros(2 * fp, K)
                w[:ff], w[fp:fp + ff] = l.w[:ff], l.w[ff:]
                ws.append(w[self.swiglu_order(2 * fp).to(w.device)])
            downs = [l.w.new_zeros((l.N + 127) // 128 * 128, fp) for l in ex.down]
            for w, l in zip(downs, ex.down):
                w[:l.N, :ff] = l.w
            ex.cuda_pack = {n: {"kind": 0, "w": torch.cat(w).to(self.device, torch.bfloat16).contiguous(), "sf": None, "alpha": None, "N": w[0].shape[0],
                                "K": w[0].shape[1], "fmt": Format.DENSE, "act_quant": False} for n, w in (("gate_up", ws), ("down", downs))}
            return ex.cuda_pack
        up, down = (padded(ex.gate_up, True, False), padded(ex.down, True, True)) if relu2 else (ex.gate_up, ex.down)
        ex.cuda_pack = {"gate_up": stack(up), "down": stack(down)}
        return ex.cuda_pack

    def _grouped_gemm(self, pk, a, M_pad, tile_expert, n_exp, out, act: int = 0):
        kind = pk["kind"]
        if kind in (1, 2):
            data, sfa, rs = a.data, a.sf, a.row_scale
            lda = data.shape[1]
        else:
            data, sfa, rs = a, None, None
            lda = a.shape[1] * 2
        w = pk["w"]
        self._check(self.lib.blz_gemm_tc(kind, _ptr(data), lda, _ptr(w), w.shape[1] * w.element_size(), _ptr(out), out.stride(0),
                                         M_pad, pk["N"], pk["K"], _ptr(rs), _ptr(pk["alpha"]), VP(0), _ptr(sfa), _ptr(pk["sf"]),
                                         0, 128, 0, _ptr(tile_expert), n_exp, 0, act, 0.0, self._stream()), "grouped gemm")
        return out

    def moe(self, x, topk_w, topk_id, experts):
        """Routed experts held by this rank: scatter rows by expert → grouped gate_up GEMM → SwiGLU → grouped down GEMM →
        weighted combine.  ``x`` is bf16 ``[T, H]``.  Under expert parallelism the result is a partial sum."""
        r = self.moe_rows(x, topk_w, topk_id, experts)
        T, H, k = x.shape[0], x.shape[1], topk_id.shape[1]
        out = torch.empty(T, H, dtype=torch.bfloat16, device=self.device)
        self._check(self.lib.blz_moe_combine(_ptr(r.rows), _ptr(r.weights), _ptr(r.row_map), _ptr(out), T, H, k, self._stream()),
                    "moe_combine")
        return out

    def moe_rows(self, x, topk_w, topk_id, experts, shared=None, gate=None) -> RoutedRows:
        """The routed experts' outputs as rows (:meth:`branch_norm` and :meth:`branch_step` sum them up, with ``shared`` added, there times
        the sigmoid of the logits ``gate``)."""
        pk = self.pack_experts(experts)
        gu, dn = pk["gate_up"], pk["down"]
        T, H = x.shape
        k = topk_id.shape[1]
        n_exp, first = experts.count, experts.first
        counts, cf, cn = getattr(self, "_route_counts", (None, -1, -1))
        if counts is None or cf != first or cn != n_exp:
            # routing was computed elsewhere: rebuild the histogram of local experts
            le = (topk_id.long() - first).flatten()
            ok = (le >= 0) & (le < n_exp)
            counts = torch.bincount(le[ok], minlength=n_exp).to(torch.int32)
        max_tiles = (T * k + 127) // 128 + n_exp
        M_pad = max_tiles * 128
        dev = self.device
        offsets = torch.empty(n_exp, dtype=torch.int32, device=dev)
        fill = torch.empty(n_exp, dtype=torch.int32, device=dev)
        tile_expert = torch.empty(max_tiles, dtype=torch.int32, device=dev)
        tile_rows = torch.empty(max_tiles, dtype=torch.int32, device=dev)
        row_map = torch.empty(T, k, dtype=torch.int32, device=dev)
        self._check(self.lib.blz_moe_plan(_ptr(counts), _ptr(offsets), _ptr(fill), _ptr(tile_expert), _ptr(tile_rows), n_exp,
                                          max_tiles, self._stream()), "moe_plan")
        narrow = T * k <= self.MOE_NARROW_ROWS * n_exp and gu["kind"] in (0, 1, 2) and gu["N"] % 128 == 0 and dn["N"] % 128 == 0
        mode = 1 if (gu["fmt"] == Format.NVFP4 and gu["act_quant"]) else (2 if gu["kind"] == 2 else 0)
        if mode:
            proxy = Linear(gu["fmt"], gu["N"], gu["K"])
            proxy.act_quant = True
            xq = self.quantize_rows(x.contiguous(), proxy)
            a = self._alloc_qact(Format.NVFP4 if mode == 1 else Format.MXFP8, M_pad, H)
            self._check(self.lib.blz_moe_scatter(mode, _ptr(xq.data), _ptr(xq.sf), _ptr(xq.row_scale), _ptr(a.data), _ptr(a.sf),
                                                 _ptr(a.row_scale), _ptr(topk_id), _ptr(offsets), _ptr(fill), _ptr(row_map), T, H, k,
                                                 first, n_exp, VP(0), 0, self._stream()), "moe_scatter")
        else:
            a = torch.empty(M_pad, H, dtype=x.dtype, device=dev)
            self._check(self.lib.blz_moe_scatter(0, _ptr(x.contiguous()), VP(0), VP(0), _ptr(a), VP(0), VP(0), _ptr(topk_id),
                                                 _ptr(offsets), _ptr(fill), _ptr(row_map), T, H * x.element_size() // 2, k, first, n_exp,
                                                 _ptr(topk_w if experts.weigh_input else None), int(x.dtype == torch.float32),
                                                 self._stream()), "moe_scatter")
        self._route_counts = None
        weights = None if experts.weigh_input else topk_w.contiguous()
        if experts.act == "swiglu" and experts.fused_act:
            y = torch.empty(M_pad, dn["N"], dtype=x.dtype, device=dev)
            if gu["kind"] == 5:
                g = torch.empty(M_pad, gu["N"], dtype=x.dtype, device=dev)
                simple = (_ptr(tile_expert), _ptr(tile_rows), int(x.dtype == torch.float32), self._stream())
                self._check(self.lib.blz_gemm_simple_experts(_ptr(a), a.stride(0), _ptr(gu["w"]), _ptr(g), g.stride(0), max_tiles, gu["N"],
                                                             gu["K"], *simple), "gemm_simple_experts")
                g = self._glu(g, -1.0)
                self._check(self.lib.blz_gemm_simple_experts(_ptr(g), g.stride(0), _ptr(dn["w"]), _ptr(y), y.stride(0), max_tiles, dn["N"],
                                                             dn["K"], *simple), "gemm_simple_experts")
            else:
                g = torch.empty(M_pad, gu["N"] // 2, dtype=x.dtype, device=dev)
                for w, src, dst in ((gu, a, g), (dn, g, y)):
                    if narrow:
                        self._moe_gemm(w, src, max_tiles, tile_expert, tile_rows, n_exp, dst, act=int(dst is g))
                    else:
                        self._grouped_gemm(w, src, M_pad, tile_expert, n_exp, dst, act=int(dst is g))
            return RoutedRows(y, row_map, weights, shared, gate)
        g = torch.empty(M_pad, gu["N"], dtype=x.dtype, device=dev)
        if experts.act == "relu2":
            y = torch.empty(M_pad, dn["N"], dtype=x.dtype, device=dev)
            for w, src, dst in ((gu, a, g), (dn, g, y)):
                if w["kind"] == 5:
                    self._check(self.lib.blz_gemm_simple_experts(_ptr(src), src.stride(0), _ptr(w["w"]), _ptr(dst), dst.stride(0), max_tiles, w["N"],
                                                                 w["K"], _ptr(tile_expert), _ptr(tile_rows), int(x.dtype == torch.float32),
                                                                 self._stream()), "gemm_simple_experts")
                    if dst is g:
                        self.relu2_(g, row_map)
                elif narrow:
                    self._moe_gemm(w, src, max_tiles, tile_expert, tile_rows, n_exp, dst, act=3 if dst is g else 0)
                else:
                    self._grouped_gemm(w, src, M_pad, tile_expert, n_exp, dst, act=3 if dst is g else 0)
            return RoutedRows(y, row_map, weights, shared, gate)
        proxy_d = Linear(dn["fmt"], dn["N"], dn["K"])
        proxy_d.act_quant = dn["act_quant"]
        y = torch.empty(M_pad, dn["N"], dtype=torch.bfloat16, device=dev)
        if narrow:
            self._moe_gemm(gu, a, max_tiles, tile_expert, tile_rows, n_exp, g)
            act = self._silu_mul_live(g, proxy_d if dn["kind"] in (1, 2) else None, row_map)
            self._moe_gemm(dn, act, max_tiles, tile_expert, tile_rows, n_exp, y)
        else:
            self._grouped_gemm(gu, a, M_pad, tile_expert, n_exp, g)
            # only the routed rows: the padded row space is up to (1 + experts * 128 / routed rows) times larger
            act = self._silu_mul_live(g, proxy_d if dn["kind"] in (1, 2) else None, row_map)
            self._grouped_gemm(dn, act, M_pad, tile_expert, n_exp, y)
        return RoutedRows(y, row_map, weights, shared, gate)

    def _moe_gemm(self, pk, a, row_tiles, tile_expert, tile_rows, n_exp, out, act: int = 0):
        """Expert GEMM over the padded row space with the features on the MMA lanes and only each tile's live rows on its columns."""
        kind = pk["kind"]
        if isinstance(a, QuantAct):
            data, sfa, rs = a.data, a.sf, a.row_scale
            lda = data.shape[1]
        else:
            data, sfa, rs = a, None, None
            lda = a.shape[1] * 2
        w = pk["w"]
        self._check(self.lib.blz_moe_gemm(kind, _ptr(data), lda, _ptr(w), w.shape[1] * w.element_size(), _ptr(out), out.stride(0),
                                          row_tiles, pk["N"], pk["K"], n_exp, _ptr(rs), _ptr(pk["alpha"]), _ptr(sfa), _ptr(pk["sf"]),
                                          _ptr(tile_expert), _ptr(tile_rows), act, self._stream()), f"moe_gemm kind {kind}")

    def _silu_mul_live(self, gu, quant_for, row_list):
        """``silu_mul`` over the padded row space of the routed rows: only the rows named in ``row_list`` (-1 = none) are
        touched, one CTA each."""
        T, I2 = gu.shape
        I = I2 // 2
        n = row_list.numel()
        mode = self._qmode(quant_for)
        if mode == 0:
            out = torch.empty(T, I, dtype=torch.bfloat16, device=self.device)
            self._check(self.lib.blz_swiglu_live(_ptr(gu), _ptr(out), VP(0), VP(0), VP(0), n, I, 0, 0, _ptr(row_list), self._stream()),
                        "swiglu_live")
            return out
        qa = self._alloc_qact(Format.NVFP4 if mode == 1 else Format.MXFP8, T, I)
        self._check(self.lib.blz_swiglu_live(_ptr(gu), VP(0), _ptr(qa.data), _ptr(qa.sf), _ptr(qa.row_scale), n, I, mode, 0,
                                             _ptr(row_list), self._stream()), "swiglu_live_q")
        return qa

    # ------------------------------------------------------------------ Gated DeltaNet
    def gdn(self, mixed_qkv, z, b, a, gdn, model, batch, kv, layer_idx, state_only: bool = False):
        """Causal conv + SiLU → gated delta rule (gates computed in the kernel) → gated RMSNorm.  Sequences flagged in
        ``batch.gdn_defer`` leave their state untouched; ``state_only`` advances the states and returns nothing."""
        conv = self.gdn_conv(mixed_qkv, gdn, batch, kv, layer_idx)
        o = None if state_only else torch.empty(mixed_qkv.shape[0], gdn.v_heads, model.cfg.linear_value_head_dim, dtype=torch.bfloat16,
                                                device=self.device)
        self.gdn_rule(conv, b, a, gdn, model, batch, kv, layer_idx, o)
        return None if state_only else self.gdn_norm(o, z, gdn, model.cfg)

    def gdn_conv(self, mixed_qkv, gdn, batch, kv, layer_idx):
        T, C = mixed_qkv.shape[0], gdn.conv_w.shape[0]
        conv = torch.empty(T, C, dtype=torch.bfloat16, device=self.device)
        self._check(self.lib.blz_gdn_conv_runs(_ptr(mixed_qkv), mixed_qkv.stride(0), _ptr(conv), _ptr(kv.conv_state[layer_idx]),
                                               _ptr(gdn.conv_w), _ptr(batch.slots), _ptr(batch.q_start), _ptr(batch.ctx_len),
                                               _ptr(batch.gdn_defer), batch.slots.numel(), C, gdn.conv_w.shape[1], int(batch.max_q_len),
                                               self._stream()), "gdn_conv")
        return conv

    def gdn_rule(self, conv, b, a, gdn, model, batch, kv, layer_idx, o):
        """The gated delta rule on convolved inputs; ``o`` None: the states only."""
        cfg = model.cfg
        dk, dv = cfg.linear_key_head_dim, cfg.linear_value_head_dim
        hk, hv = gdn.k_heads, gdn.v_heads
        T, B, state_only = conv.shape[0], batch.slots.numel(), o is None
        # long token runs (prompt chunks) go through the chunked tensor-core kernel, short ones (decode, verify, replay)
        # through the token-by-token kernel; both walk the same batch and each takes its own sequences
        chunked = (self.GDN_CHUNK_MIN > 0 and not state_only and dk == 128 and dv == 128 and batch.max_q_len >= self.GDN_CHUNK_MIN)
        n_chunks = T // 128 + B                    # upper bound of the sum over sequences of ceil(new tokens / 128)
        ws_bytes = int(self.lib.blz_gdn_chunk_ws_bytes(n_chunks, hv)) if chunked and self.GDN_SPLIT else 0
        if chunked and self.GDN_SPLIT and ws_bytes <= self.GDN_SPLIT_MAX_WS:
            ws = torch.empty(ws_bytes, dtype=torch.uint8, device=self.device)
            self._check(self.lib.blz_gdn_chunk_split(_ptr(conv), _ptr(a), _ptr(b), a.stride(0), _ptr(gdn.A_log), _ptr(gdn.dt_bias),
                                                     _ptr(kv.rec_state[layer_idx]), _ptr(o), _ptr(batch.slots), _ptr(batch.q_start),
                                                     _ptr(batch.ctx_len), _ptr(batch.gdn_defer), B, hk, hv, dk, dv, self.GDN_CHUNK_MIN,
                                                     int(batch.max_q_len), n_chunks, _ptr(ws), self._stream()), "gdn_chunk_split")
            self.launches += 1                     # two kernels behind the one call
        elif chunked:
            self._check(self.lib.blz_gdn_chunk(_ptr(conv), _ptr(a), _ptr(b), a.stride(0), _ptr(gdn.A_log), _ptr(gdn.dt_bias),
                                               _ptr(kv.rec_state[layer_idx]), _ptr(o), _ptr(batch.slots), _ptr(batch.q_start),
                                               _ptr(batch.ctx_len), _ptr(batch.gdn_defer), B, hk, hv, dk, dv, self.GDN_CHUNK_MIN,
                                               self._stream()), "gdn_chunk")
        if not chunked or batch.num_rows > batch.max_q_len or B > 1:
            self._check(self.lib.blz_gdn_recurrent_upto(_ptr(conv), _ptr(a), _ptr(b), a.stride(0), _ptr(gdn.A_log), _ptr(gdn.dt_bias),
                                                        _ptr(kv.rec_state[layer_idx]), _ptr(o), _ptr(batch.slots), _ptr(batch.q_start),
                                                        _ptr(batch.ctx_len), _ptr(batch.gdn_defer), B, hk, hv, dk, dv,
                                                        self.GDN_CHUNK_MIN - 1 if chunked else 0x7fffffff, self._stream()),
                        "gdn_recurrent")

    def gdn_norm(self, o, z, gdn, cfg):
        T, hv, dv = o.shape
        y = torch.empty(T, hv * dv, dtype=torch.bfloat16, device=self.device)
        self._check(self.lib.blz_gated_rmsnorm(_ptr(o), _ptr(z), z.stride(0), _ptr(gdn.norm_w), _ptr(y), T, hv, dv,
                                               cfg.rms_norm_eps, 2 if cfg.gdn_output_gate == "sigmoid" else 0, self._stream()),
                    "gated_rmsnorm")
        return y
