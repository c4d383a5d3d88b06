"""The compiled kernels as Python callables (ctypes over the library's ``extern "C"`` launchers).

Every launcher returns 0 or an error code; :func:`call` turns a code into an exception that names
the launcher.  Pointers are passed as integers (``tensor.data_ptr()``), and the last argument of
every launcher is the CUDA stream, taken from torch's current stream, so kernels run (and are
captured into CUDA graphs) in order with torch's own work.

The library is loaded on first use and the process fails loudly when it cannot be built or loaded:
there is no CPU path and no library fallback behind these functions.
"""
from __future__ import annotations

import ctypes
import threading
from typing import Dict

import torch

from .build import KernelBuildError, ensure_built

_P, _I, _F, _L, _U = ctypes.c_void_p, ctypes.c_int, ctypes.c_float, ctypes.c_longlong, ctypes.c_ulonglong
_CODES = {"p": _P, "i": _I, "f": _F, "l": _L, "u": _U}

# name -> argument codes (the trailing stream is added for all but the ones marked no_stream)
_SIGNATURES: Dict[str, str] = {
    "tb_embed_f32": "pppii", "tb_embed_bf16": "pppii",
    "tb_add_rmsnorm_f32": "pppppippfpiipi", "tb_add_rmsnorm_bf16": "pppppippfpiipi",
    "tb_add_rmsnorm_router_f32": "pppppippfppppiiii", "tb_add_rmsnorm_router_bf16": "pppppippfppppiiii",
    "tb_rope_cache_f32": "ppppippppiiiii", "tb_rope_cache_bf16": "ppppippppiiiii",
    "tb_attention_f32": "ppppppppppiiiiiiiif", "tb_attention_bf16": "ppppppppppiiiiiiiif",
    "tb_gemm_simt_f32": "pppppliiiiiiii".replace(" ", ""), "tb_gemm_simt_bf16": "pppppliiiiiiii",
    "tb_gemm_skinny_bf16": "pppppliiiiiiiiipii",
    "tb_attention_decode_f32": "ppppppppiiiiiiif", "tb_attention_decode_bf16": "ppppppppiiiiiiif",
    "tb_attention_prefill_bf16": "pppppppppiiiiiif",
    "tb_attention_tc_bf16": "pppppppppiiiiiiiif",
    "tb_gemm_tc_bf16": "ppppiiiiiiii", "tb_gather_rows_bf16": "pppii",
    "tb_attention_decode_mma_bf16": "pppppppppiiiiiiiif",
    "tb_attention_decode_rope_bf16": "pppppppppppiiiiiiiiiif",
    "tb_router_f32": "pppppppppiiii", "tb_router_bf16": "pppppppppiiii",
    "tb_router_rows_bf16": "pppppppppiiii",
    "tb_moe_dispatch": "ppppiii",
    "tb_moe_combine_f32": "ppppiii", "tb_moe_combine_bf16": "ppppiii",
    "tb_sample": "plpiififpp",
    "tb_kernel_status_async": "p",
    "tb_random_fill_f32": "plulf", "tb_random_fill_bf16": "plulf",
    "tb_embed_scaled_f32": "pppiif", "tb_embed_scaled_bf16": "pppiif",
    "tb_post_add_rmsnorm_f32": "pppppipfppfpii", "tb_post_add_rmsnorm_bf16": "pppppipfppfpii",
    "tb_gemm_simt_glu_f32": "pppppliiiiiiiffi", "tb_gemm_simt_glu_bf16": "pppppliiiiiiiffi",
    "tb_gemm_simt_batched_f32": "pppllliiiiiii", "tb_gemm_simt_batched_bf16": "pppllliiiiiii",
    "tb_gemm_skinny_glu_bf16": "pppppliiiiiiiipiiffi",
    "tb_gemm_tc_glu_bf16": "ppppiiiiiiiffi",
    "tb_post_add_rmsnorm_router_f32": "pppppipfpfpppppiiiii", "tb_post_add_rmsnorm_router_bf16": "pppppipfpfpppppiiiii",
    "tb_add_rmsnorm_router_scored_f32": "pppppippfpppppiiii", "tb_add_rmsnorm_router_scored_bf16": "pppppippfpppppiiii",
    "tb_router_rows_scored_bf16": "pppppppppiiii",
    "tb_router_scored_f32": "pppppppppiiii", "tb_router_scored_bf16": "pppppppppiiii",
    "tb_moe_identity_rows_f32": "pppppiiii", "tb_moe_identity_rows_bf16": "pppppiiii",
    "tb_mlstm_scan_f32": "pppppppiiiiiff", "tb_mlstm_scan_bf16": "pppppppiiiiiff",
    "tb_mlstm_chunk_f32": "pppppppiiiiiff", "tb_mlstm_chunk_bf16": "pppppppiiiiiff",
    "tb_mlstm_out_f32": "ppippiiifii", "tb_mlstm_out_bf16": "ppippiiifii",
    "tb_latent_prep_f32": "pippfpppppippiiiii", "tb_latent_prep_bf16": "pippfpppppippiiiii",
    "tb_latent_attention_mma_bf16": "ppppppppppppiiiiiiiiiiifppi",
    "tb_latent_attention_f32": "pppppppppppiiiiiiiiiifppi", "tb_latent_attention_bf16": "pppppppppppiiiiiiiiiifppi",
    "tb_embed_bigram_f32": "pppppppppiifiii", "tb_embed_bigram_bf16": "pppppppppiifiii",
    "tb_scale_f32": "plf",
    "tb_qknorm_rope_cache_f32": "pippfpppippppiiiiiii", "tb_qknorm_rope_cache_bf16": "pippfpppippppiiiiiii",
    "tb_attention_window_f32": "pppppppppppiiiiiiiiiiiiffippp", "tb_attention_window_bf16": "pppppppppppiiiiiiiiiiiiffippp",
    "tb_pair_add_rmsnorm_f32": "ppppppippifii", "tb_pair_add_rmsnorm_bf16": "ppppppippifii",
    "tb_conv_roll_f32": "piplppiii", "tb_conv_roll_bf16": "piplppiii",
    "tb_causal_conv_f32": "pipplpipppiiiiii", "tb_causal_conv_bf16": "pipplpipppiiiiii",
    "tb_head_prep_f32": "pipplpppfppppppppppppiiiiiiiiipp", "tb_head_prep_bf16": "pipplpppfppppppppppppiiiiiiiiipp",
    "tb_attention_window_mma_bf16": "pppppppppppiiiiiiiiiiiiffippp",
    "tb_delta_prep_f32": "pipppppppppppiiiiiiiiiii",
    "tb_delta_prep_bf16": "pipppppppppppiiiiiiiiiii",
    "tb_delta_scan": "ppppppiiiiiii",
    "tb_bias_glu_f32": "pppiii", "tb_bias_glu_bf16": "pppiii",
    "tb_router_sigmoid_f32": "ppppppppiiii", "tb_router_sigmoid_bf16": "ppppppppiiii",
    "tb_router_rows_sigmoid_bf16": "ppppppppiiii",
    "tb_moe_scaled_rows_f32": "ppppiii", "tb_moe_scaled_rows_bf16": "ppppiii",
    "tb_relu2_f32": "pl", "tb_relu2_bf16": "pl",
    "tb_post_add_layernorm_f32": "pppppippfipppfipii", "tb_post_add_layernorm_bf16": "pppppippfipppfipii",
    "tb_renew_layernorm_f32": "pppppifppfpiipppppi", "tb_renew_layernorm_bf16": "pppppifppfpiipppppi",
    "tb_moe_dispatch_shared": "ppppiii",
    "tb_moe_terms_f32": "pppppppiii", "tb_moe_terms_bf16": "pppppppiii",
    "tb_head_prep_keyed_f32": "pipifpppppppppiiiiii", "tb_head_prep_keyed_bf16": "pipifpppppppppiiiiii",
    "tb_attention_window_heads_f32": "pppppppppppiiiiiiiiiiiiffipppifi",
    "tb_attention_window_heads_bf16": "pppppppppppiiiiiiiiiiiiffipppifi",
    "tb_attention_window_mma_heads_bf16": "pppppppppppiiiiiiiiiiiiffipppifi",
    "tb_shift_mix_f32": "pppllpppipppii", "tb_shift_mix_bf16": "pppllpppipppii",
    "tb_decay_tanh_f32": "pipiii", "tb_decay_tanh_bf16": "pipiii",
    "tb_decay_prep_f32": "pppppiii", "tb_decay_prep_bf16": "pppppiii",
    "tb_decay_scan_f32": "pplppippiiii", "tb_decay_scan_bf16": "pplppippiiii",
    "tb_decay_step_f32": "ppipippppfplpippiiiii", "tb_decay_step_bf16": "ppipippppfplpippiiiii",
    "tb_qknorm_rope_cache_biased_f32": "pippppfpppippppiiiiiii", "tb_qknorm_rope_cache_biased_bf16": "pippppfpppippppiiiiiii",
    "tb_attention_window_biased_f32": "pppppppppppiiiiiiiiiiiiffipifipi",
    "tb_attention_window_biased_bf16": "pppppppppppiiiiiiiiiiiiffipifipi",
    "tb_attention_window_mma_biased_bf16": "pppppppppppiiiiiiiiiiiiffipifipi",
    "tb_split_rows_f32": "pipiii", "tb_split_rows_bf16": "pipiii",
    "tb_decay_scan_rect": "pplpppiiiii",
    "tb_gated_linear_prep_f32": "pipppiiiiiff", "tb_gated_linear_prep_bf16": "pipppiiiiiff",
    "tb_gated_linear_step_f32": "pipipppplpippiiiiiifff", "tb_gated_linear_step_bf16": "pipipppplpippiiiiiifff",
    "tb_split_delta_prep_f32": "pipippppiii", "tb_split_delta_prep_bf16": "pipippppiii",
    "tb_split_delta_step_f32": "pipippppfplpippiiiii", "tb_split_delta_step_bf16": "pipippppfplpippiiiii",
    "tb_split_delta_scan": "pplpppiiii",
    "tb_stream_step_f32": "ppppipplpipppppii", "tb_stream_step_bf16": "ppppipplpipppppii",
    "tb_embed_learned_f32": "pppppiifppp", "tb_embed_learned_bf16": "pppppiifppp",
    "tb_post_add_layernorm_router_f32": "pppppippfipppfipiippppiii",
    "tb_post_add_layernorm_router_bf16": "pppppippfipppfipiippppiii",
}
class TapeArg(ctypes.Union):
    _fields_ = [("p", ctypes.c_void_p), ("i", ctypes.c_int), ("f", ctypes.c_float), ("l", ctypes.c_longlong),
                ("u", ctypes.c_ulonglong)]


TAPE_MAX_ARGS = 32


class TapeEntry(ctypes.Structure):
    """One recorded launcher call (csrc/tape.h)."""
    _fields_ = [("fn", ctypes.c_int), ("n_args", ctypes.c_int), ("ptr_mask", ctypes.c_uint), ("reserved", ctypes.c_int),
                ("args", TapeArg * TAPE_MAX_ARGS)]


class TapeMap(ctypes.Structure):
    """Addresses [base, base + size) of the recorded layer move by delta for the layer being run."""
    _fields_ = [("base", ctypes.c_ulonglong), ("size", ctypes.c_ulonglong), ("delta", ctypes.c_longlong)]


_NO_STREAM = {"tb_decay_scan_rect_record_size": "ii", "tb_split_delta_record_size": "i",
              "tb_decay_state_size": "iii", "tb_decay_record_size": "i",
              "tb_attention_window_mma_tile_tokens": "ii", "tb_delta_state_size": "iiiii", "tb_delta_record_size": "i", "tb_delta_scan_lanes": "i", "tb_delta_value_pitch": "i", "tb_mlstm_state_size": "ii", "tb_latent_attention_tile_tokens": "i", "tb_attention_tile_tokens": "ii", "tb_gemm_tc_status": "", "tb_attention_prefill_tile_tokens": "",
              "tb_attention_tc_tile_tokens": ""}

_lock = threading.Lock()
_lib = None


class KernelError(RuntimeError):
    pass


def library() -> ctypes.CDLL:
    global _lib
    if _lib is not None:
        return _lib
    with _lock:
        if _lib is None:
            path = ensure_built()
            try:
                lib = ctypes.CDLL(path)
            except OSError as e:  # pragma: no cover
                raise KernelBuildError(f"cannot load {path}: {e}") from e
            for name, codes in _SIGNATURES.items():
                fn = getattr(lib, name)
                fn.argtypes = [_CODES[c] for c in codes] + [_P]
                fn.restype = _I
            for name, codes in _NO_STREAM.items():
                fn = getattr(lib, name)
                fn.argtypes = [_CODES[c] for c in codes]
                fn.restype = _I
            lib.tb_tape_index.argtypes = [ctypes.c_char_p]
            lib.tb_tape_index.restype = _I
            lib.tb_tape_replay.argtypes = [ctypes.POINTER(TapeEntry), _I, ctypes.POINTER(TapeMap), _I,
                                           ctypes.POINTER(ctypes.c_int), _P]
            lib.tb_tape_replay.restype = _I
            _lib = lib
    return _lib


def library_path() -> str:
    return ensure_built()


def _error_text(code: int) -> str:
    if code == -1:
        return "bad argument"
    if code == -2:
        return "size not supported by this kernel"
    return f"CUDA error {code}"


launch_count = 0     # launchers called so far (a launcher may start more than one kernel)

_scope_stream = None  # inside stream_scope(): the handle of the stream that was current at its start


class stream_scope:
    """``with stream_scope():`` looks torch's current stream up once for all the launches inside (a model's forward
    pass is some hundred launches, and the look-up costs as much as a launch).  Whoever opens it must not
    change the current stream inside; a scope opened inside a graph capture sees the capturing stream."""

    def __enter__(self):
        global _scope_stream
        self._before = _scope_stream
        _scope_stream = torch.cuda.current_stream().cuda_stream
        return self

    def __exit__(self, *exc):
        global _scope_stream
        _scope_stream = self._before
        return False


def _stream() -> int:
    return _scope_stream if _scope_stream is not None else torch.cuda.current_stream().cuda_stream


_recorder = None      # while a layer's calls are recorded: an object with launch(name, args) and foreign(kind, *tensors)


class recording:
    """``with recording(tape):`` every launcher call that succeeds inside is also reported to ``tape.launch(name,
    args)``, and device work that does not go through a launcher reports itself with :func:`foreign`."""

    def __init__(self, tape):
        self.tape = tape

    def __enter__(self):
        global _recorder
        self._before = _recorder
        _recorder = self.tape
        return self.tape

    def __exit__(self, *exc):
        global _recorder
        _recorder = self._before
        return False


_timing = None        # while launches are timed: launcher name -> [(start event, end event)]


class timing:
    """``with timing() as t:`` every launcher call inside is bracketed by CUDA events on the launching stream;
    afterwards ``t.ms`` holds the device time per launcher name, ``t.calls`` the number of calls.  For eager steps
    (a replayed graph or tape calls no launcher from Python); costs two event records per launch."""

    def __enter__(self):
        global _timing
        self._before = _timing
        _timing = self._events = {}
        self.ms, self.calls = {}, {}
        return self

    def __exit__(self, *exc):
        global _timing
        _timing = self._before
        torch.cuda.synchronize()
        for name, pairs in self._events.items():
            self.ms[name] = sum(a.elapsed_time(b) for a, b in pairs)
            self.calls[name] = len(pairs)
        return False


def _timed(name, fn, args):
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    rc = fn(*args, _stream())
    b.record()
    if rc == 0:
        _timing.setdefault(name, []).append((a, b))
    return rc


def foreign(kind: str, *tensors) -> None:
    """Tell a recording that device work of another kind is about to run here (a library product, ...)."""
    if _recorder is not None:
        _recorder.foreign(kind, *tensors)


def try_call(name: str, *args) -> bool:
    """Like :func:`call`, but a kernel that refuses the sizes (TB_ERR_UNSUPPORTED) answers False
    instead of raising, so the caller can take the general kernel."""
    global launch_count
    fn = getattr(_lib if _lib is not None else library(), name)
    rc = fn(*args, _stream()) if _timing is None else _timed(name, fn, args)
    if rc == -2:
        return False
    if rc != 0:
        raise KernelError(f"{name}: {_error_text(rc)}")
    launch_count += 1
    if _recorder is not None:
        _recorder.launch(name, args)
    return True


def call(name: str, *args) -> None:
    """Launch ``name`` on torch's current stream."""
    global launch_count
    launch_count += 1
    fn = getattr(_lib if _lib is not None else library(), name)
    rc = fn(*args, _stream()) if _timing is None else _timed(name, fn, args)
    if rc != 0:
        raise KernelError(f"{name}: {_error_text(rc)}")
    if _recorder is not None:
        _recorder.launch(name, args)


_tape_indices: Dict[str, int] = {}


def tape_entries(calls) -> "ctypes.Array":
    """[(launcher name, argument tuple)] as the array of TapeEntry that :func:`tape_replay` runs."""
    arr = (TapeEntry * len(calls))()
    for e, (name, args) in zip(arr, calls):
        codes = _SIGNATURES[name]
        if len(args) != len(codes) or len(args) > TAPE_MAX_ARGS:
            raise KernelError(f"{name}: {len(args)} arguments recorded, {len(codes)} declared")
        idx = _tape_indices.get(name)
        if idx is None:
            idx = library().tb_tape_index(name.encode())
            if idx < 0:
                raise KernelError(f"{name} is not registered for replay")
            _tape_indices[name] = idx
        e.fn, e.n_args, mask = idx, len(args), 0
        for j, (c, v) in enumerate(zip(codes, args)):
            if c == "p":
                e.args[j].p = v or None
                mask |= 1 << j
            elif c == "i":
                e.args[j].i = int(v)
            elif c == "f":
                e.args[j].f = float(v)
            elif c == "l":
                e.args[j].l = int(v)
            else:
                e.args[j].u = int(v)
        e.ptr_mask = mask
    return arr


def tape_maps(moves) -> "ctypes.Array":
    """[(base, size, delta)] as an array of TapeMap."""
    arr = (TapeMap * max(1, len(moves)))()
    for m, (base, size, delta) in zip(arr, moves):
        m.base, m.size, m.delta = base, size, delta
    return arr


_failed_at = ctypes.c_int(0)


def tape_replay(entries, maps, n_maps: int) -> None:
    """Run recorded calls on torch's current stream with the pointers of ``maps`` moved."""
    global launch_count
    rc = library().tb_tape_replay(entries, len(entries), maps, n_maps, ctypes.byref(_failed_at), _stream())
    if rc != 0:
        raise KernelError(f"replayed call {_failed_at.value} of {len(entries)}: {_error_text(rc)}")
    launch_count += len(entries)


def ptr(t) -> int:
    return 0 if t is None else t.data_ptr()


def suffix(dtype: torch.dtype) -> str:
    if dtype == torch.float32:
        return "f32"
    if dtype == torch.bfloat16:
        return "bf16"
    raise KernelError(f"kernels exist for float32 and bfloat16, not {dtype}")


def random_fill(t: torch.Tensor, base: int, scale: float, first: int = 0) -> None:
    """Fill the contiguous tensor ``t`` (float32 or bfloat16) with elements first .. first + t.numel() - 1 of the
    counter-based stream that starts at ``base`` (see weights/counter_random.py)."""
    if not t.is_contiguous():
        raise KernelError("random_fill needs a contiguous tensor")
    call("tb_random_fill_" + suffix(t.dtype), t.data_ptr(), t.numel(), int(base), int(first), float(scale))


def attention_tile_tokens(nh: int, nkvh: int) -> int:
    return library().tb_attention_tile_tokens(nh, nkvh)


def gemm_tc_status() -> int:
    """0, or the code of a kernel with bounded waits (the tensor-core products, the tensor-core and the
    page-ring attention) that gave up on a wait since the last call; synchronises the device and clears it."""
    return library().tb_gemm_tc_status()


def kernel_status_async(host_int32: torch.Tensor) -> None:
    """Copy the same code into the first element of a pinned int32 host tensor, in stream order and without
    waiting: it lands together with the step's other results."""
    rc = library().tb_kernel_status_async(host_int32.data_ptr(), _stream())
    if rc != 0:
        raise KernelError(f"tb_kernel_status_async: {_error_text(rc)}")


def _gave_up(code: int) -> str:
    """Which kernel family a wait code belongs to (1..5 tensor-core products, 11..17 tensor-core prompt
    attention, 21..27 decode attention with the page ring, 31..32 the decaying memory's scan, 33..34 the split delta
    rule's)."""
    if 1 <= code <= 5:
        return "tensor-core matrix product"
    if 11 <= code <= 17:
        return "tensor-core prompt attention"
    if 21 <= code <= 22:
        return "decode attention"
    if 31 <= code <= 32:
        return "scan of the decaying memory"
    if 33 <= code <= 34:
        return "scan of the split delta rule"
    return "unknown kernel"


def raise_for_status(code: int, recover=None) -> None:
    """``code`` is the word the kernels with bounded waits share (0: all well).  Anything else means that a wait
    ran out and the kernel returned early: its result is not to be used.  ``recover()`` is called first (it puts
    back what such a kernel leaves behind), then :class:`KernelError` is raised."""
    if not code:
        return
    if recover is not None:
        recover()
    raise KernelError(f"a kernel gave up after its wait limit (code {code}: {_gave_up(int(code))}); the results of "
                      f"the steps since the last check are not valid")


def mlstm_state_size(dim: int, vdim: int) -> int:
    """Floats of state that the matrix-memory kernel keeps per (sequence, head)."""
    return library().tb_mlstm_state_size(dim, vdim)


def delta_state_size(kv_heads: int, heads: int, dim: int, vdim: int, taps: int) -> int:
    """Floats of state that the delta-rule kernels keep per sequence (the heads' memories, then the convolution's
    last inputs)."""
    return library().tb_delta_state_size(kv_heads, heads, dim, vdim, taps)


def delta_record_size(dim: int) -> int:
    """Floats of the record that the delta rule's first kernel leaves the scan per (token, head)."""
    return library().tb_delta_record_size(dim)


def delta_value_pitch(vdim: int) -> int:
    """Floats of a (token, head) row of values between the delta rule's two kernels."""
    return library().tb_delta_value_pitch(vdim)


def decay_state_size(heads: int, dim: int, width: int) -> int:
    """Floats of state that the decaying linear memory keeps per sequence (the heads' memories, then the last input)."""
    return library().tb_decay_state_size(heads, dim, width)


def decay_record_size(dim: int) -> int:
    """Floats of the record that the decaying memory's first kernel leaves the scan per (token, head)."""
    return library().tb_decay_record_size(dim)


def gated_linear_record_size(dim: int, vdim: int) -> int:
    """Floats of the record that the gated linear attention's first kernel leaves the scan per (token, head)."""
    return library().tb_decay_scan_rect_record_size(dim, vdim)


def split_delta_record_size(dim: int) -> int:
    """Floats of the record that the split delta rule's first kernel leaves the scan per (token, head)."""
    return library().tb_split_delta_record_size(dim)


def attention_window_mma_tile_tokens(nh: int, nkvh: int) -> int:
    """Query tokens per block of the tensor-core windowed attention (0: it does not take such head groups)."""
    return library().tb_attention_window_mma_tile_tokens(nh, nkvh)


def latent_attention_tile_tokens(heads: int) -> int:
    return library().tb_latent_attention_tile_tokens(heads)


def attention_prefill_tile_tokens() -> int:
    return library().tb_attention_prefill_tile_tokens()


def attention_tc_tile_tokens() -> int:
    return library().tb_attention_tc_tile_tokens()
