"""Bindings of the layer-stack kernels (``csrc/stack*.cu``, ``csrc/latent_attn.cu``), built as their own library.

The argument classes are generated from ``csrc/stack.cuh`` (``ops.abi.generate_from``) and their sizes checked against
the loaded library; nothing here allocates on the launch path.
"""
from __future__ import annotations

import ctypes as C
from typing import Optional

import torch

from . import kernels as K
from .abi import generate_from
from .build import load_library

VP = C.c_void_p
_G = generate_from("stack.cuh", ["StackGemmArgs", "StackRowArgs", "LatentPrepArgs", "LatentAttnArgs", "LatentDecodeArgs",
                                 "RecurrenceArgs", "MoeGatherArgs", "StepArgs", "GroupPrepArgs", "TransposeArgs", "GroupDecodeArgs",
                                 "StateChunkArgs", "ShortConvArgs", "TokenMixArgs", "HeadGateArgs", "StateStepArgs"])
StackGemmArgs, StackRowArgs, LatentPrepArgs = _G["StackGemmArgs"], _G["StackRowArgs"], _G["LatentPrepArgs"]
LatentAttnArgs, LatentDecodeArgs, RecurrenceArgs = _G["LatentAttnArgs"], _G["LatentDecodeArgs"], _G["RecurrenceArgs"]
MoeGatherArgs, StepArgs = _G["MoeGatherArgs"], _G["StepArgs"]
GroupPrepArgs, TransposeArgs, GroupDecodeArgs = _G["GroupPrepArgs"], _G["TransposeArgs"], _G["GroupDecodeArgs"]
StateChunkArgs, ShortConvArgs, TokenMixArgs = _G["StateChunkArgs"], _G["ShortConvArgs"], _G["TokenMixArgs"]
HeadGateArgs, StateStepArgs = _G["HeadGateArgs"], _G["StateStepArgs"]

EPI_STORE, EPI_BIAS, EPI_TRANSPOSE, EPI_CLAMPED_GLU, EPI_SILU_GLU = 0, 1, 2, 3, 4
EPI_RELU2, EPI_TANH, EPI_DECAY_SOFT, EPI_DECAY_EXP = 5, 6, 7, 8
PRO_RESIDUAL, PRO_NORM, PRO_LOAD, PRO_MERGE, PRO_EXPERTS, PRO_MIX = 0, 1, 2, 3, 4, 5
TEPI_STORE, TEPI_CONV, TEPI_GATE, TEPI_GLU, TEPI_RECUR, TEPI_CONV_SILU, TEPI_RELU2 = 0, 1, 2, 3, 4, 5, 6
NORM = {"rms": 0, "layer": 1}
STATE_DELTA, STATE_BONUS, STATE_NORMALIZED = 0, 1, 2
GATE_SIGMOID, GATE_SILU = 0, 1
MAX_SPLITS = 8                                        # context splits of the grouped one-token attention (a cluster)

# library entry points of the family and the argument struct each reads
ENTRIES = {"nrt_stack_gemm": ("StackGemmArgs", "nrt_stack_gemm_args_size"), "nrt_stack_gemm_f32": ("StackGemmArgs", "nrt_stack_gemm_args_size"),
           "nrt_stack_rows": ("StackRowArgs", "nrt_stack_row_args_size"), "nrt_latent_prep": ("LatentPrepArgs", "nrt_latent_prep_args_size"),
           "nrt_latent_attn_rows": ("LatentAttnArgs", "nrt_latent_attn_args_size"),
           "nrt_latent_attn_tc": ("LatentAttnArgs", "nrt_latent_attn_args_size"),
           "nrt_latent_decode": ("LatentDecodeArgs", "nrt_latent_decode_args_size"),
           "nrt_stack_conv": ("RecurrenceArgs", "nrt_recurrence_args_size"), "nrt_stack_scan": ("RecurrenceArgs", "nrt_recurrence_args_size"),
           "nrt_moe_gather": ("MoeGatherArgs", "nrt_moe_gather_args_size"), "nrt_stack_step": ("StepArgs", "nrt_step_args_size"),
           "nrt_group_prep": ("GroupPrepArgs", "nrt_group_prep_args_size"), "nrt_transpose": ("TransposeArgs", "nrt_transpose_args_size"),
           "nrt_group_decode": ("GroupDecodeArgs", "nrt_group_decode_args_size"),
           "nrt_state_chunk": ("StateChunkArgs", "nrt_state_chunk_args_size"), "nrt_state_step": ("StateStepArgs", "nrt_state_step_args_size"),
           "nrt_short_conv": ("ShortConvArgs", "nrt_short_conv_args_size"), "nrt_token_mix": ("TokenMixArgs", "nrt_token_mix_args_size"),
           "nrt_head_gate": ("HeadGateArgs", "nrt_head_gate_args_size")}

_lib = None


def lib() -> C.CDLL:
    """The layer-stack library; refuses one whose argument structs differ from these bindings."""
    global _lib
    if _lib is None:
        L = load_library(group="stack")
        for entry, (struct, size) in ENTRIES.items():
            if not hasattr(L, entry):
                raise RuntimeError(f"the layer-stack library exports no {entry}")
            if getattr(L, size)() != C.sizeof(_G[struct]):
                raise RuntimeError(f"{struct}: library has {getattr(L, size)()} bytes, bindings {C.sizeof(_G[struct])}")
        if L.nrt_ep_args_size() != C.sizeof(K.EpArgs):
            raise RuntimeError("EpArgs layout drift")
        _lib = L
    return _lib


def _stream() -> VP:
    return VP(torch.cuda.current_stream().cuda_stream)


def weight_map(w: torch.Tensor, k: int) -> K.TensorMap:
    """bf16 weights [z, n, ld] with ``k`` live columns -> boxes of 128 features x 64 columns."""
    z, n, ld = w.shape
    return K.TensorMap(w, (k, n, z), (ld * 2, n * ld * 2), (64, 128, 1), 1, library=lib())


def token_map(t: torch.Tensor, k: int, zcount: int, zstride: int, rows: int, ld: int, box_rows: int, offset: int = 0) -> K.TensorMap:
    """bf16 rows, element (row, z, c) at offset + row * ld + z * zstride + c, ``k`` live columns per group."""
    view = t.view(-1)[offset:]
    return K.TensorMap(view, (k, zcount, rows), ((zstride if zcount > 1 else ld) * 2, ld * 2), (64, 1, box_rows), 1, library=lib())


def value_map(v: torch.Tensor, keys: int, features: int, box: int) -> K.TensorMap:
    """Feature-major values [features, keys] -> boxes of ``box`` features x 64 keys."""
    return K.TensorMap(v, (keys, features), (keys * 2,), (64, box), 1, library=lib())


def gemm(epi: int, ntok: int, w: K.TensorMap, w2: Optional[K.TensorMap], x: K.TensorMap, args: StackGemmArgs, items_fastest: bool) -> None:
    K.check(lib().nrt_stack_gemm(epi, ntok, C.byref(w.buf), C.byref(w2.buf) if w2 is not None else None, C.byref(x.buf),
                                 C.byref(args), int(items_fastest), _stream()), "stack gemm")


def gemm_f32(epi: int, args: StackGemmArgs) -> None:
    K.check(lib().nrt_stack_gemm_f32(epi, C.byref(args), _stream()), "stack gemm (float)")


def rows(args: StackRowArgs) -> None:
    K.check(lib().nrt_stack_rows(C.byref(args), _stream()), "stack rows")


def latent_prep(args: LatentPrepArgs) -> None:
    K.check(lib().nrt_latent_prep(C.byref(args), _stream()), "latent prep")


def latent_attn_rows(args: LatentAttnArgs) -> None:
    K.check(lib().nrt_latent_attn_rows(C.byref(args), _stream()), "latent attention (rows)")


def latent_attn_tc(q: K.TensorMap, k: K.TensorMap, v: K.TensorMap, args: LatentAttnArgs) -> None:
    K.check(lib().nrt_latent_attn_tc(C.byref(q.buf), C.byref(k.buf), C.byref(v.buf), C.byref(args), _stream()), "latent attention (chunk)")


def latent_decode(args: LatentDecodeArgs, pdl: bool) -> None:
    K.check(lib().nrt_latent_decode(C.byref(args), _stream(), int(pdl)), "latent attention (step)")


def conv(args: RecurrenceArgs) -> None:
    K.check(lib().nrt_stack_conv(C.byref(args), _stream()), "short convolution")


def scan(args: RecurrenceArgs) -> None:
    K.check(lib().nrt_stack_scan(C.byref(args), _stream()), "recurrence scan")


def scan_tokens() -> int:
    return lib().nrt_stack_scan_tokens()


def group_prep(args: GroupPrepArgs) -> None:
    K.check(lib().nrt_group_prep(C.byref(args), _stream()), "grouped attention prep")


def transpose(args: TransposeArgs) -> None:
    K.check(lib().nrt_transpose(C.byref(args), _stream()), "transpose")


def group_decode(args: GroupDecodeArgs, pdl: bool) -> None:
    K.check(lib().nrt_group_decode(C.byref(args), _stream(), int(pdl)), "grouped attention (step)")


def short_conv(args: ShortConvArgs) -> None:
    K.check(lib().nrt_short_conv(C.byref(args), _stream()), "short convolution with SiLU")


def token_mix(args: TokenMixArgs) -> None:
    K.check(lib().nrt_token_mix(C.byref(args), _stream()), "token mixes")


def state_chunk(kind: int, args: StateChunkArgs) -> None:
    K.check(lib().nrt_state_chunk(kind, C.byref(args), _stream()), "matrix-state recurrence (chunk)")


STATE_BLOCK = 8                                       # tokens per block record of the chunk recurrence


def state_block_floats(kind: int, dim: int) -> int:
    """Scratch floats of the chunk recurrence per (block of tokens, head)."""
    return lib().nrt_state_block_floats(kind, dim)


def state_sum_floats(kind: int, heads: int, dim: int, vdim: int) -> int:
    """Scratch floats of the chunk recurrence for the pieces' sums."""
    f = lib().nrt_state_sum_floats
    f.restype = C.c_longlong
    return f(kind, heads, dim, vdim)


def state_step(args: StateStepArgs, pdl: bool) -> None:
    K.check(lib().nrt_state_step(C.byref(args), _stream(), int(pdl)), "matrix-state recurrence (step)")


def head_gate(args: HeadGateArgs) -> None:
    K.check(lib().nrt_head_gate(C.byref(args), _stream()), "read-out norm and gate")


def route(args: K.RouterArgs, groups: int, keep: int) -> None:
    K.check(lib().nrt_stack_route(C.byref(args), groups, keep, _stream()), "expert choice")


def moe_count(args: K.EpArgs) -> None:
    K.check(lib().nrt_ep_count(C.byref(args), _stream(), 0), "expert counts")


def moe_gather(args: MoeGatherArgs) -> None:
    K.check(lib().nrt_moe_gather(C.byref(args), _stream()), "expert gather")


def step(pro: int, epi: int, args: StepArgs, router: Optional[K.RouterArgs], groups: int, keep: int, pdl: bool) -> None:
    K.check(lib().nrt_stack_step(pro, epi, C.byref(args), C.byref(router) if router is not None else None, groups, keep, _stream(),
                                 int(pdl)), "stack step")
