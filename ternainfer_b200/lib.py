"""ctypes bindings of ``libternaspmm.so`` and the dense decoders' libraries (built in-tree under ``csrc/``).

The reference binds its library with ``ctypes.CDLL('./kernels/libternaspmm.so')``
and passes every pointer as ``c_void_p`` (model.py:21, :76-89 of
Gu-J/TernaInfer); this module does the same against the B200 library and
declares argument types so that mistakes fail in Python rather than on the GPU.
There is no fallback: if the library is missing, loading raises.
The libraries of the dense decoders (include/decoder_ops.h) are loaded one by
one, at the first call into each; their calls take argument structs and return
a status, which ``check`` turns into an exception.
"""
from __future__ import annotations

import ctypes
import fcntl
import os
import subprocess

_HERE = os.path.dirname(os.path.abspath(__file__))
_CSRC = os.path.join(_HERE, "csrc")
_LIB = None

_P = ctypes.c_void_p
_I = ctypes.c_int
_SPMM_ARGS = [_P, _P, _P, _P, _P, _P, _P, _P, _I, _I, _I, _I, _I, _P, _P]


class ListItem(ctypes.Structure):
    """``ternaspmm_list_item`` of include/ternaspmm.h."""
    _fields_ = [(n, _P) for n in ("x", "bitmap", "tile_offsets", "quarter_offsets", "sign_words", "out", "s", "ws",
                                  "residual")] + \
               [(n, _I) for n in ("ws_num", "M", "N", "K", "seg1", "seg2", "seg3", "prefill_form")]


class Gate(ctypes.Structure):
    """``decoder_gate``: activation of a gated feed-forward."""
    _fields_ = [("kind", _I), ("alpha", ctypes.c_float), ("limit", ctypes.c_float)]


def _struct(name, fields):
    """``fields``: 'type: names' lines in the order of the C struct."""
    kinds = {"p": _P, "i": _I, "l": ctypes.c_longlong, "f": ctypes.c_float, "g": Gate}
    flat = [(n, kinds[line[0]]) for line in fields for n in line[2:].split()]
    return type(name, (ctypes.Structure,), {"_fields_": flat})


# the argument structs of include/decoder_ops.h
EmbedArgs = _struct("EmbedArgs", ["p tokens pos prev embed bigram x", "l mul_prev mul_cur buckets", "i B T S D V"])
HyperArgs = _struct("HyperArgs", ["p x y mix out in_ w rows h y2 slots slot_w mu prev mixed pos", "f m w_offset eps",
                                  "i D S n_rows top n_mu"])
ShiftArgs = _struct("ShiftArgs", ["p h prev mu mixed pos", "i B T D n_mu"])
LinearArgs = _struct("LinearArgs", ["p x w bias out x2 w2 out2 zero", "i M N K relu2 seg_rows n_seg N2", "g gate"])
DeltaArgs = _struct("DeltaArgs", ["p proj zw w2 w0 a_bias norm pos state o y", "i B T H dk dv rank", "l ld",
                                  "i off_r off_k off_v off_a off_g off_w1", "f eps"])
AttnArgs = _struct("AttnArgs", ["p proj ck cv q_norm k_norm bias slope pos y", "i B T H G dim vdim", "l ld",
                                "i off_q off_k off_v off_g", "i chunk slots", "f scale eps"])
WkvArgs = _struct("WkvArgs", ["p r k v g t1 zw w2 w0 u norm pos state part o y", "i B T H dk dv rank", "l ld ld_t", "i n_seg seg_len", "f eps"])
LatentPrepArgs = _struct("LatentPrepArgs", ["p z cq cache q_norm kv_norm trig pos", "i B T slots ld r_at R rot dims q_rank", "l ld_z",
                                            "i off_q off_kv", "f eps"])
RotateArgs = _struct("RotateArgs", ["p src dst trig pos", "i B T H rot dims", "l ld_src ld_dst", "i head_src head_dst off_src off_dst"])
AbsorbArgs = _struct("AbsorbArgs", ["p q w_uk_t qa trig pos", "i B T H dim rot dims R r_at ld"])
LatentAttnArgs = _struct("LatentAttnArgs", ["p qa cache sink pos out w_uv part ml y", "i B T H R ld vdim slots splits cluster", "f scale"])
LatentPromptArgs = _struct("LatentPromptArgs", ["p q kv cache sink y", "i B T H dim rot vdim slots ld r_at start off_v", "l ld_kv", "f scale"])
MoeArgs = _struct("MoeArgs", ["p logits router_bias chosen weight counts rank slots ticket x sorted w_up act w_down w_rest rest bias out",
                              "i M E top K ff D K_rest", "g gate"])
GroupGemmArgs = _struct("GroupGemmArgs", ["p a w bias counts out", "i rows groups N K", "g gate"])


def library_path() -> str:
    return os.path.join(_CSRC, "libternaspmm.so")


def build_library(target: str = "all", verbose: bool = False) -> str:
    """Compile the libraries for sm_100a with nvcc (``make -C csrc``)."""
    subprocess.run(["make", "-C", _CSRC, "verbose" if verbose else target], check=True, stdout=None if verbose else subprocess.DEVNULL)
    return library_path()


def build_decoder_library(*names: str):
    """Compile the dense decoders' libraries of these names (all without any), as far as they are not up to date; safe to
    call from several processes."""
    files = [f"lib{n}.so" for n in names or DECODER_LIBRARIES]
    with open(os.path.join(_CSRC, "Makefile")) as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)
        subprocess.run(["make", "-j", str(len(files)), "-C", _CSRC] + files, check=True, stdout=subprocess.DEVNULL)


class DecoderOpsError(RuntimeError):
    """A call into a dense decoders' library was refused; the library has written the reason to stderr."""


def check(status: int):
    if status:
        raise DecoderOpsError({1: "shape not supported", 2: "bad pointer", 3: "launch failed", 4: "a wait inside a kernel ran out"}.get(status, str(status)))


_L = ctypes.c_longlong


def _calls(*calls):
    """name -> argument types: a struct first (by reference), or the list as it is."""
    return {name: ([ctypes.POINTER(args[0])] + args[1:] if isinstance(args[0], type(ctypes.Structure)) else args) if args else []
            for name, args in calls}


# library -> entry points and their argument types; everything returns int but for the names in _LONG
DECODER_LIBRARIES = {
    "decoderops": _calls(("decoder_embed", [EmbedArgs, _I, _I, _P]), ("decoder_hyper", [HyperArgs, _I, _I, _P]),
                         ("decoder_token_shift", [ShiftArgs, _I, _I, _P]), ("decoder_rows_linear", [LinearArgs, _I, _I, _P]),
                         ("decoder_gated", [_P, _P, _P, _L, _I, ctypes.POINTER(Gate), _I, _I, _P]),
                         ("decoder_head_argmax", [_P, _P, _I, _I, _I, _P, _P, _P, _P]), ("decoder_head_scratch_bytes", []),
                         ("decoder_relu2", [_P, _L, _I, _I, _P]), ("decoder_tanh_cols", [_P, _L, _I, _I, _L, _P, _I, _I, _P])),
    "deltaops": _calls(("decoder_delta", [DeltaArgs, _I, _I, _P]), ("decoder_attn", [AttnArgs, _I, _I, _I, _P]), ("decoder_status", [])),
    "latentops": _calls(("decoder_wkv", [WkvArgs, _I, _I, _P]), ("decoder_latent_prep", [LatentPrepArgs, _I, _I, _P]),
                        ("decoder_rotate", [RotateArgs, _I, _I, _P]), ("decoder_absorb", [AbsorbArgs, _I, _P]),
                        ("decoder_latent_attn", [LatentAttnArgs, _I, _I, _P]), ("decoder_latent_step", [LatentAttnArgs, _I, _P]),
                        ("decoder_latent_step_width", []), ("decoder_latent_prompt", [LatentPromptArgs, _P]),
                        ("decoder_moe_route", [MoeArgs, _I, _P]), ("decoder_moe_plain", [MoeArgs, _I, _I, _P]),
                        ("decoder_moe_up_step", [MoeArgs, _I, _P]), ("decoder_moe_down_step", [MoeArgs, _I, _P]),
                        ("decoder_group_gemm", [GroupGemmArgs, _P]), ("decoder_latent_status", [])),
}
_LONG = ("decoder_head_scratch_bytes",)
DECODER_SYMBOLS = tuple(s for calls in DECODER_LIBRARIES.values() for s in calls)


class _DecoderLibrary:
    """The entry points of all dense decoders' libraries; each library is loaded at the first call into it."""

    def __getattr__(self, symbol):
        for name, calls in DECODER_LIBRARIES.items():
            if symbol in calls:
                path = os.path.join(_CSRC, f"lib{name}.so")
                if not os.path.exists(path):
                    raise OSError(f"{path} not found: build it with `make -C {_CSRC} lib{name}.so` (or __graft_entry__.build())")
                lib = ctypes.CDLL(path)
                for s, args in calls.items():
                    fn = getattr(lib, s)
                    fn.argtypes, fn.restype = args, _L if s in _LONG else _I
                    setattr(self, s, fn)
                return getattr(self, symbol)
        raise AttributeError(symbol)


_DECODER_LIB = _DecoderLibrary()


def load_decoder_library() -> _DecoderLibrary:
    """The dense decoders' entry points; calling one raises ``OSError`` if its library has not been built."""
    return _DECODER_LIB


def load_library() -> ctypes.CDLL:
    """Load the shared library; raises ``OSError`` if it has not been built."""
    global _LIB
    if _LIB is not None:
        return _LIB
    path = library_path()
    if not os.path.exists(path):
        raise OSError(f"{path} not found: build it with `make -C {_CSRC}` (or __graft_entry__.build())")
    lib = ctypes.CDLL(path)
    for name in ("bitlinear_TernaSpMM", "bitlinear_TernaSpMM_decode", "bitlinear_TernaSpMM_prefill"):
        fn = getattr(lib, name)
        fn.argtypes = _SPMM_ARGS
        fn.restype = None
    lib.bitlinear_TernaSpMM_benchmark.argtypes = [_I, _I, _I] + _SPMM_ARGS
    lib.bitlinear_TernaSpMM_benchmark.restype = None
    lib.checkLastCudaError.argtypes = [_I]
    lib.checkLastCudaError.restype = None
    lib.reorder_WT_h.argtypes = [_P, _P, _I, _I]
    lib.reorder_WT_h.restype = None
    lib.convert_reorderd.argtypes = [_P, _I, _I, _I, _I, _I, _I, _I, _I,
                                     ctypes.POINTER(_P), ctypes.POINTER(_P), ctypes.POINTER(_P),
                                     ctypes.POINTER(_P), ctypes.POINTER(_I)]
    lib.convert_reorderd.restype = _I
    lib.gpu_sleep.argtypes = [ctypes.c_double, _P]
    lib.gpu_sleep.restype = None
    lib.ternaspmm_last_status.argtypes = []
    lib.ternaspmm_last_status.restype = _I
    lib.ternaspmm_set_wait_limit_ms.argtypes = [_I]
    lib.ternaspmm_set_wait_limit_ms.restype = None
    lib.ternaspmm_last_launch_shape.argtypes = [_P]
    lib.ternaspmm_last_launch_shape.restype = None
    lib.ternaspmm_debug_inject_host_failure.argtypes = [_I]
    lib.ternaspmm_debug_inject_host_failure.restype = None
    lib.ternaspmm_list_plan.argtypes = [_P, _I, ctypes.POINTER(ctypes.c_longlong), ctypes.POINTER(ctypes.c_longlong)]
    lib.ternaspmm_list_plan.restype = _I
    lib.ternaspmm_list_create.argtypes = [_P, _I, _P, _P, _P]
    lib.ternaspmm_list_create.restype = _P
    lib.ternaspmm_list_run.argtypes = [_P, _P]
    lib.ternaspmm_list_run.restype = None
    lib.ternaspmm_list_destroy.argtypes = [_P]
    lib.ternaspmm_list_destroy.restype = None
    lib.ternaspmm_lm_head_argmax.argtypes = [_P, _P, _I, _I, _I, _P, _P, _I, _P, _P]
    lib.ternaspmm_lm_head_argmax.restype = None
    lib.ternaspmm_lm_head_argmax_noalloc.argtypes = [_P, _P, _I, _I, _I, _P, _P, _I, _P]
    lib.ternaspmm_lm_head_argmax_noalloc.restype = None
    lib.ternaspmm_lm_head_scratch_bytes.argtypes = []
    lib.ternaspmm_lm_head_scratch_bytes.restype = ctypes.c_longlong
    lib.ternaspmm_accumulate_i32.argtypes = [_P, _P, _P, _P, _P, _P, _I, _I, _I, _P]
    lib.ternaspmm_accumulate_i32.restype = None
    lib.ternaspmm_linear_segments.argtypes = [_P] * 8 + [_I] * 8 + [_P]
    lib.ternaspmm_linear_segments.restype = None
    for name in ("ternaspmm_rmsnorm_quant", "ternaspmm_relu2_gate_rmsnorm_quant"):
        fn = getattr(lib, name)
        fn.argtypes = [_P, _P, ctypes.c_float, _I, _I, _P, _P, _P]
        fn.restype = None
    lib.ternaspmm_rmsnorm.argtypes = [_P, _P, ctypes.c_float, _I, _I, _P, _P]
    lib.ternaspmm_debug_int8_mma_rate.argtypes = [_I, _P]
    lib.ternaspmm_debug_int8_mma_rate.restype = ctypes.c_double
    lib.ternaspmm_rmsnorm.restype = None
    lib.ternaspmm_quant.argtypes = [_P, _I, _I, _P, _P, _P]
    lib.ternaspmm_quant.restype = None
    lib.ternaspmm_scale_quant_sumsq.argtypes = [_P, _P, _I, _I, _I, _P, _P, _P, _P]
    lib.ternaspmm_scale_quant_sumsq.restype = None
    lib.ternaspmm_partial_f32.argtypes = [_P] * 7 + [_I, _I, _I, _P]
    lib.ternaspmm_partial_f32.restype = None
    lib.ternaspmm_tp_finish.argtypes = [_P, _P, ctypes.c_float, _I, _I, _I, _P, _P, _P]
    lib.ternaspmm_tp_finish.restype = None
    lib.ternaspmm_tp_allreduce_finish.argtypes = [_P, _P, _P, _I, _I, _P, _P, ctypes.c_float, _I, _I, _I, _P, _P]
    lib.ternaspmm_tp_allreduce_finish.restype = None
    lib.bitlinear_TernaSpMM_ws.argtypes = [_P] * 8 + [_I] * 4 + [_P, _P, ctypes.c_longlong, _I, _P]
    lib.bitlinear_TernaSpMM_ws.restype = None
    lib.bitlinear_TernaSpMM_residual.argtypes = [_P] * 8 + [_I] * 4 + [_P, _P]
    lib.bitlinear_TernaSpMM_residual.restype = None
    lib.ternaspmm_pack_i8.argtypes = [_P, _I, _I, _P, _P, _P, _P]
    lib.ternaspmm_pack_i8.restype = ctypes.c_longlong
    lib.ternaspmm_unpack_i8.argtypes = [_P, _P, _P, _I, _I, _P]
    lib.ternaspmm_unpack_i8.restype = _I
    lib.ternaspmm_transcode_reference_layout.argtypes = [_P, _P, _P, _I, _I, _P, _P, _P]
    lib.ternaspmm_transcode_reference_layout.restype = _I
    _LIB = lib
    return lib


EXPORTED_SYMBOLS = (
    "bitlinear_TernaSpMM", "bitlinear_TernaSpMM_decode", "bitlinear_TernaSpMM_prefill",
    "bitlinear_TernaSpMM_benchmark", "checkLastCudaError", "reorder_WT_h", "convert_reorderd",
    "gpu_sleep", "ternaspmm_last_status", "ternaspmm_set_wait_limit_ms", "ternaspmm_last_launch_shape",
    "ternaspmm_debug_inject_host_failure", "ternaspmm_debug_int8_mma_rate", "ternaspmm_lm_head_argmax", "ternaspmm_lm_head_scratch_bytes",
    "ternaspmm_lm_head_argmax_noalloc",
    "ternaspmm_list_plan", "ternaspmm_list_create", "ternaspmm_list_run", "ternaspmm_list_destroy",
    "ternaspmm_accumulate_i32", "ternaspmm_linear_segments", "bitlinear_TernaSpMM_residual", "bitlinear_TernaSpMM_ws", "ternaspmm_quant",
    "ternaspmm_scale_quant_sumsq", "ternaspmm_partial_f32", "ternaspmm_tp_finish", "ternaspmm_tp_allreduce_finish", "ternaspmm_rmsnorm_quant", "ternaspmm_relu2_gate_rmsnorm_quant", "ternaspmm_rmsnorm", "ternaspmm_pack_i8",
    "ternaspmm_unpack_i8", "ternaspmm_transcode_reference_layout",
)
