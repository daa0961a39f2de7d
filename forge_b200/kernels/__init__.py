"""Python face of the hand-written CUDA kernels (sm_100a).

Each function checks its tensors (device, dtype, contiguity, shapes), passes raw pointers and the
current CUDA stream to an ``extern "C"`` entry point through ctypes, and raises ``KernelError`` with the
library's message on a non-zero return.  There is no CPU or PyTorch fallback: if a library cannot be
compiled or loaded the first call that needs it raises.
"""
import ctypes
import os
from ctypes import c_float, c_int, c_void_p

import torch

from .build import BuildError, build_library

F32, BF16 = 0, 1


class KernelError(RuntimeError):
    pass


def dtype_code(dt):
    if dt == torch.float32:
        return F32
    if dt == torch.bfloat16:
        return BF16
    raise KernelError(f"kernels take float32 or bfloat16 tensors, not {dt}")


_P, _I, _F, _LL = c_void_p, c_int, c_float, ctypes.c_longlong

_SIGNATURES = {
    "core": {
        "forge_embedding": [_P, _P, _I, _P, _I, _I, _I, _F, _I, _P, _P],
        "forge_embedding_pair": [_P, _P, _P, _P, _P, _P, _LL, _P, _P, _I, _P, _I, _I, _I, _I, _LL, _LL, _P, _P],
        "forge_rmsnorm_add": [_P, _P, _P, _P, _P, _I, _I, _I, _F, _F, _P],
        "forge_streams_expand": [_P, _P, _I, _I, _I, _P],
        "forge_streams_mix": [_P] * 7 + [_I, _P, _I, _I, _I, _F, _P],
        "forge_layernorm": [_P, _P, _P, _P, _I, _P, _I, _I, _F, _P],
        "forge_act_rows": [_P, _I, _P, _I, _I, _I, _I, _F, _F, _P],
        "forge_depth_step": [_P, _LL, _I, _I, _I, _I] + [_P] * 4 + [_I, _I, _I, _P, _P, _I, _F, _P, _I, _P, _I, _I, _P],
        "forge_rmsnorm": [_P, _P, _P, _I, _P, _I, _I, _F, _P],
        "forge_join": [_P, _I] + [_P, _P, _F] * 4 + [_F, _P, _F, _P, _I, _I, _I, _P],
        "forge_rmsnorm_pair": [_P, _P, _P, _P, _P, _I, _I, _I, _F, _P],
        "forge_rope_kv_write": [_P, _P, _P, _P, _P, _I, _I, _I, _I, _I, _I, _F, _I, _P, _P],
        "forge_rope_table": [_P, _P, _I, _I, _F, _I, _P],
        "forge_silu_mul_interleaved": [_P, _P, _I, _I, _I, _I, _P],
        "forge_gemm_simt": [_P, _P, _P, _P, _I, _I, _I, _I, _I, _P],
        "forge_paged_attention_simt": [_P, _P, _P, _P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _I, _F, _P],
        "forge_argmax": [_P, _P, _I, _I, _P],
        "forge_repeat_penalty": [_P, _P, _P, _P, _P, _I, _I, _P],
        "forge_sample": [_P, _P, _P, _P, _P, _P, _I, _I, _P],
        "forge_history_penalty": [_P, _P, _P, _P, _I, _I, _P],
        "forge_history_add": [_P, _P, _P, _P, _I, _I, _P],
    },
    "gemm_sm100": {
        "forge_gemm_sm100": [_P, _P, _P, _P, _P, _I, _I, _I, _I, _I, _P, _F, _F, _P],
        "forge_gemm_sm100_set_workspace": [_P, ctypes.c_longlong],
        "forge_gemm_sm100_qkv_rope": [_P] * 8 + [_I] * 7 + [_P],
    },
    "attention_mma": {
        "forge_paged_attention_mma": [_P] * 10 + [_I] * 9 + [_F, _P],
        "forge_decode_attention_fused": [_P] * 6 + [_I] * 8 + [_F, _F, _I, _P],
        "forge_decode_attention_stream": [_P] * 7 + [_I] * 9 + [_F, _F, _I, _I, _P],
    },
    "attention_sm100": {
        "forge_paged_attention_sm100": [_P] * 10 + [_I] + [_P] * 3 + [_I] * 9 + [_F, _P],
    },
    "mixers": {
        "forge_headmix_prepare": [_P, _I] + [_P] * 9 + [_I] * 8 + [_LL, _I, _P],
        "forge_headmix_attention": [_P] * 10 + [_I] * 7 + [_LL, _I, _I, _I, _F, _I, _I, _P],
        "forge_headmix_mma_supports": [_I, _I, _I, _I, _I],
        "forge_headmix_attention_mma": [_P] * 11 + [_I, _P] + [_I] * 7 + [_LL, _I, _I, _I, _F, _P],
        "forge_state_scan": [_I, _P, _I, _P, _I, _P, _I, _P, _I, _P, _I, _P, _P, _P, _P, _P, _LL, _P, _P, _P, _P, _I, _I, _LL, _I, _I, _I, _I, _I, _P],
        "forge_scored_prepare": [_P, _I] + [_P] * 7 + [_I] * 8 + [_F, _F, _F, _I, _LL, _P],
        "forge_scored_prepare_heads": [_P, _I, _P, _P, _P, _F, _P, _P] + [_I] * 8 + [_F, _I, _LL, _P],
        "forge_scored_attention": [_P] * 10 + [_I] * 8 + [_LL, _I] + [_F] * 5 + [_I, _I, _LL, _I, _I, _F, _P, _P],
        "forge_scored_mma_supports": [_I] * 6,
        "forge_scored_attention_mma": [_P] * 11 + [_I, _P] + [_I] * 8 + [_LL, _I] + [_F] * 5 + [_LL, _I, _I, _F, _P, _P],
        "forge_token_shift": [_P, _P, _LL, _LL, _P, _P, _P, _P, _P, _I, _I, _I, _I, _P],
        "forge_head_finish": [_P, _P, _P, _I, _P, _I, _I, _I, _I, _F, _I, _F, _I, _LL, _P],
        "forge_tanh_rows": [_P, _I, _P, _I, _I, _I, _P],
        "forge_gla_scan": [_P, _I] * 4 + [_I, _P, _P, _F, _F, _P, _P, _LL, _P, _P, _P, _I, _I, _I, _I, _I, _P],
        "forge_gla_token": [_P, _I] * 5 + [_I, _P, _P, _F, _F, _P, _LL, _P, _P, _P, _F, _P, _I, _LL, _I, _I, _I, _I, _P],
        "forge_lightning_scan": [_P, _I, _P, _P, _P, _LL, _P, _P, _P] + [_I] * 5 + [_P],
        "forge_lightning_token": [_P, _I, _P, _P, _LL, _P, _P, _P] + [_I] * 4 + [_P],
        "forge_gated_delta_scan": [_P, _I] * 3 + [_P, _P, _P, _P, _LL, _P, _P, _P] + [_I] * 6 + [_P],
        "forge_delta_prepare": [_P, _I, _I, _I, _P, _I, _P, _LL, _LL] + [_P] * 9 + [_I] * 6 + [_P],
        "forge_gated_delta_token": [_P, _I, _I, _I, _I, _P, _I, _P, _LL, _LL] + [_P] * 6 + [_F, _P, _I, _LL] + [_I] * 5 + [_P],
        "forge_token_state_supports": [_I] * 3,
        "forge_gated_rows": [_P, _P, _P, _I, _P, _I, _LL, _I, _I, _F, _P],
        "forge_retention_scan": [_P, _I, _P, _I, _P, _I, _P, _P, _I, _F, _P, _P, _LL, _P, _P, _P, _I, _I, _I, _I, _I, _P],
    },
    "latent": {
        "forge_latent_prepare": [_P, _I, _P, _P, _P, _F, _P, _P, _P, _P, _I, _I, _I, _I, _I, _F, _I, _P],
        "forge_head_linear": [_P, _I, _LL, _I, _P, _P, _I, _LL, _I, _P, _P, _F, _I, _I, _I, _I, _I, _I, _P, _LL, _I, _I, _I, _P],
        "forge_latent_attention": [_P] * 8 + [_I] * 8 + [_F, _I, _I, _I, _P, _P],
        "forge_latent_mma_supports": [_I] * 4,
        "forge_latent_mma_heads": [_I],
        "forge_latent_attention_mma": [_P] * 9 + [_I, _P] + [_I] * 7 + [_F, _I, _P, _P],
    },
    "moe": {
        "forge_moe_route": [_P, _I, _P, _P, _P, _I, _I, _I, _I, _I, _I, _P, _I, _I, _I, _F, _P],
        "forge_moe_pair_gate_up": [_P, _P, _P, _P, _P, _I, _I, _I, _I, _I, _LL, _P],
        "forge_moe_pair_down": [_P, _P, _P, _P, _P, _I, _I, _I, _I, _I, _P],
        "forge_moe_expert_supports": [_I, _I, _I],
        "forge_moe_expert_rows": [_P, _P, _P, _LL, _P, _P, _P, _P, _I, _I, _I, _I, _I, _I, _P],
        "forge_moe_sort": [_P, _I, _P, _P, _P, _P, _P, _I, _I, _I, _I, _I, _P],
        "forge_moe_combine": [_P, _P, _P, _P, _I, _I, _I, _P],
    },
    "decode_layers": {
        "forge_decode_layers_desc_bytes": [],
        "forge_decode_layers_supports": [_I] * 6,
        "forge_decode_layers_describe": [_P, _I] + [_P] * 8 + [_I] * 5,
        "forge_decode_layers": [_P, _I] + [_P] * 12 + [_I] * 10 + [_F, _F, _F, _I, _P, _P],
        "forge_decode_layers_barrier_probe": [_P, _P, ctypes.c_ulonglong, _P],
    },
}

_libs = {}

# FORGE_CHECKS=1: every library is built with index checks (csrc/checks.cuh): page ids, slots and token indices are
# tested before use, a bad one raises bit 4 of the step's status word and is skipped.  The entries that tell a
# library the bounds, per library (one per source file that checks):
_CHECK_ENTRIES = {"core": ["forge_checks_configure_rope", "forge_checks_configure_attention_simt"],
                  "mixers": ["forge_checks_configure_attention_headmix", "forge_checks_configure_attention_headmix_mma",
                             "forge_checks_configure_attention_scored", "forge_checks_configure_attention_scored_mma"],
                  "latent": ["forge_checks_configure_attention_latent", "forge_checks_configure_attention_latent_mma"],
                  "gemm_sm100": ["forge_checks_configure_gemm_sm100"],
                  "attention_mma": ["forge_checks_configure_attention_mma", "forge_checks_configure_attention_decode_stream"],
                  "attention_sm100": ["forge_checks_configure_attention_sm100"]}
_check_bounds = [None]          # (num_pages, page_size, num_tokens, status tensor, first_bad tensor) of the current step


def checks_enabled():
    return os.environ.get("FORGE_CHECKS", "0") == "1"


def _configure_library_checks(name, lib):
    b = _check_bounds[0]
    if b is None:
        return
    for fn in _CHECK_ENTRIES.get(name, []):
        f = getattr(lib, fn)
        f.argtypes = [_I, _I, _I, _P, _P, _P]
        f.restype = c_int
        rc = f(b[0], b[1], b[2], b[3].data_ptr(), b[4].data_ptr(), _stream())
        if rc != 0:
            raise KernelError(f"{fn}: {lib.forge_last_error().decode(errors='replace')}")


def configure_checks(num_pages, page_size, num_tokens, status, first_bad):
    """(checks build) Gives every loaded library the bounds of the step that is about to run; libraries loaded later
    get them when they load.  ``status``: int32 [1]; ``first_bad``: int32 [3] (kind, value, limit of the first offender)."""
    if not checks_enabled():
        return
    _check_bounds[0] = (int(num_pages), int(page_size), int(num_tokens), status, first_bad)
    for (name, defines), lib in _libs.items():
        if ("FORGE_CHECKS", 1) in defines:
            _configure_library_checks(name, lib)


def library(name, defines=None):
    """Loads (building first if needed) kernel library ``name`` (variant ``defines``) and returns its
    ctypes handle."""
    if checks_enabled() and name in _CHECK_ENTRIES:
        defines = dict(defines or {}, FORGE_CHECKS=1)
    key = (name, tuple(sorted((defines or {}).items())))
    lib = _libs.get(key)
    if lib is not None:
        return lib
    if not torch.cuda.is_available():
        raise KernelError("forge_b200 runs on a CUDA device (B200, sm_100a) only; no device is visible")
    try:
        path = build_library(name, defines=defines)
    except BuildError as e:
        raise KernelError(f"kernel library '{name}' is not available: {e}") from e
    try:
        lib = ctypes.CDLL(path)
    except OSError as e:
        raise KernelError(f"cannot load {path}: {e}") from e
    for fn, argtypes in _SIGNATURES[name].items():
        f = getattr(lib, fn)
        f.argtypes = argtypes
        f.restype = c_int
        setattr(lib, fn, _Entry(lib, fn, f, argtypes))
    lib.forge_last_error.restype = ctypes.c_char_p
    _libs[key] = lib
    if defines and defines.get("FORGE_CHECKS") == 1:
        _configure_library_checks(name, lib)
    return lib


_launches = [0]

# ----------------------------------------------------------------------------- a layer's launches, noted and repeated
# The layers of a model mostly differ in nothing but the addresses of their weights and caches, while the host's share
# of a launch (choosing the kernel, checking the arguments, cutting outputs from the workspace, the foreign call) costs
# about 17 us against 3 to 10 us of device time at few tokens: a prompt of 128 tokens took 2.7 ms for 0.9 ms of device
# work.  So a model whose layers declare it (parts.base.replay_of) runs ONE layer through Python with the calls into
# the libraries noted, and repeats the noted calls for the other layers with the layer's own addresses in place.
# Launches that make what the whole step shares happen inside the layer that first needs it; they are marked
# (once_per_step) and left out of the notes.
_recording = [None]
_once = [0, 0]          # depth of open ``once_per_step`` blocks; launches counted inside them while a recording is open


class _OncePerStep:
    def __enter__(self):
        _once[0] += 1

    def __exit__(self, *exc):
        _once[0] -= 1
        return False


def once_per_step():
    """``with once_per_step():`` around launches that make something the whole step shares (a table of angles, a
    workspace handed to a library): a recording that is open leaves them out, and they are not repeated with the
    layer they happened to be made in."""
    return _OncePerStep()


class _Entry:
    """A library function that notes its calls while a recording is open."""
    __slots__ = ("lib", "name", "fn", "pointer_args")

    def __init__(self, lib, name, fn, argtypes):
        self.lib, self.name, self.fn = lib, name, fn
        self.pointer_args = tuple(i for i, t in enumerate(argtypes) if t is _P)

    def __call__(self, *args):
        rec = _recording[0]
        if rec is not None and not _once[0]:
            rec.append((self, args))
        return self.fn(*args)


class _Recording:
    def __enter__(self):
        self.calls, self.launches0 = [], _launches[0]
        _recording[0] = self.calls
        _once[1] = 0
        return self

    def __exit__(self, *exc):
        _recording[0] = None
        self.launches = _launches[0] - self.launches0 - _once[1]
        return False


def record_launches():
    """``with record_launches() as rec:`` notes every call into the kernel libraries made inside (``rec.calls``) and how
    many launches they counted for (``rec.launches``)."""
    return _Recording()


class LayerReplay:
    """The launches of one layer, to be repeated for layers of the same shape.  ``source``: the device tensors of the
    recorded layer (weights, cache), None where an optional one is absent; every pointer argument that points into one
    of them is exchanged for the same offset into the other layer's tensor."""

    def __init__(self, recording, source):
        spans = [(t.data_ptr(), t.data_ptr() + t.numel() * t.element_size(), i) for i, t in enumerate(source) if t is not None]
        self.calls = [(entry, list(args)) for entry, args in recording.calls]
        self.patches = []                       # (call, argument, tensor, byte offset)
        for ci, (entry, args) in enumerate(self.calls):
            for ai in entry.pointer_args:
                v = args[ai]
                if not v:
                    continue
                for lo, hi, ti in spans:
                    if lo <= v < hi:
                        self.patches.append((ci, ai, ti, v - lo))
                        break
        self.launches = recording.launches
        self.source_kinds = [t is None for t in source]

    def run(self, tensors):
        """Repeats the launches with ``tensors`` (same order and kinds as the source) in the recorded tensors' place."""
        if [t is None for t in tensors] != self.source_kinds:
            raise KernelError("a layer's launches cannot be repeated for a layer with other optional tensors")
        base = [0 if t is None else t.data_ptr() for t in tensors]
        calls = self.calls
        for ci, ai, ti, off in self.patches:
            calls[ci][1][ai] = base[ti] + off
        for entry, args in calls:
            rc = entry.fn(*args)
            if rc != 0:
                raise KernelError(f"{entry.name}: {entry.lib.forge_last_error().decode(errors='replace')} (code {rc})")
        _launches[0] += self.launches


def launch_count():
    """How many kernels of these libraries have been launched (graph replays add their kernels)."""
    return _launches[0]


def count_launches(n):
    _launches[0] += n


def _check(lib, rc, what):
    _launches[0] += 1
    if _once[0]:
        _once[1] += 1
    if rc != 0:
        raise KernelError(f"{what}: {lib.forge_last_error().decode(errors='replace')} (code {rc})")
    if _profile["on"]:
        _profile_mark(what)


# ------------------------------------------------------------------------------------------ timing
# A per-kernel-class timing table in the manner of the reference's PerfProfiler (include/forge/perf_profiler.h:28-218,
# src/bindings/profiler.cpp): while it is enabled an event is recorded after every launch, and a kernel's time is the
# time from the end of its predecessor on the stream to its own end (so it includes the hand-over between the two).
# Decode steps are launched kernel by kernel meanwhile (a CUDA graph replay has no launches to put events between).
_profile = {"on": False, "last": None, "pending": [], "records": {}}


def profiler_enable():
    _profile["on"] = True
    _profile["last"] = None


def profiler_disable():
    _profile["on"] = False


def profiler_enabled():
    return _profile["on"]


def profiler_reset():
    _profile["pending"].clear()
    _profile["records"].clear()
    _profile["last"] = None


def profiler_step_begin():
    """The time before a step's first kernel belongs to nobody."""
    if _profile["on"]:
        e = torch.cuda.Event(enable_timing=True)
        e.record()
        _profile["last"] = e


def _profile_mark(what):
    e = torch.cuda.Event(enable_timing=True)
    e.record()
    if _profile["last"] is not None:
        _profile["pending"].append((what, _profile["last"], e))
    _profile["last"] = e


def profiler_summary():
    """{kernel class: {count, total_ms, avg_ms, min_ms, max_ms, last_ms}} (the reference's field names)."""
    if _profile["pending"]:
        torch.cuda.synchronize()
        for what, e0, e1 in _profile["pending"]:
            ms = e0.elapsed_time(e1)
            r = _profile["records"].setdefault(what, {"count": 0, "total_ms": 0.0, "min_ms": float("inf"), "max_ms": 0.0, "last_ms": 0.0})
            r["count"] += 1
            r["total_ms"] += ms
            r["min_ms"], r["max_ms"], r["last_ms"] = min(r["min_ms"], ms), max(r["max_ms"], ms), ms
        _profile["pending"].clear()
    return {k: dict(v, avg_ms=v["total_ms"] / v["count"]) for k, v in _profile["records"].items()}


def profiler_print(file=None):
    import sys
    rows = sorted(profiler_summary().items(), key=lambda kv: -kv[1]["total_ms"])
    total = sum(r["total_ms"] for _, r in rows) or 1.0
    out = file or sys.stderr
    print(f"{'kernel':<28}{'count':>8}{'total ms':>12}{'avg us':>10}{'min us':>10}{'max us':>10}{'share':>8}", file=out)
    for name, r in rows:
        print(f"{name:<28}{r['count']:>8}{r['total_ms']:>12.3f}{1e3 * r['avg_ms']:>10.1f}{1e3 * r['min_ms']:>10.1f}"
              f"{1e3 * r['max_ms']:>10.1f}{100 * r['total_ms'] / total:>7.1f}%", file=out)


# The current stream's handle, asked for once per kernel launch: torch's two C entry points answer in a fraction of a
# microsecond, torch.cuda.current_stream() takes several (a prompt step of a 22-layer model launches 180 kernels and
# is as long on the host as on the device).
_raw_stream = getattr(torch._C, "_cuda_getCurrentRawStream", None)
_raw_device = getattr(torch._C, "_cuda_getDevice", None)


def _stream():
    if _raw_stream is not None and _raw_device is not None:
        return _raw_stream(_raw_device())
    return torch.cuda.current_stream().cuda_stream


def _need(t, name, dtype=None, ndim=None):
    if not t.is_cuda:
        raise KernelError(f"{name} must be a CUDA tensor")
    if not t.is_contiguous():
        raise KernelError(f"{name} must be contiguous")
    if dtype is not None and t.dtype != dtype:
        raise KernelError(f"{name} must be {dtype}, got {t.dtype}")
    if ndim is not None and t.dim() != ndim:
        raise KernelError(f"{name} must have {ndim} dims, got shape {tuple(t.shape)}")
    return t.data_ptr()


def _opt(t, name, dtype=None):
    return None if t is None else _need(t, name, dtype)


# ----------------------------------------------------------------------------------- step workspace

class StepWorkspace:
    """One device buffer that the outputs of a step's kernels are cut from, instead of one trip to the allocator per
    kernel output (the reference allocates device memory for every operator output, src/core/tensor.cpp:86-107).

    While a step is open (``with ws.step():``) every tensor that the functions of this module would allocate is a
    view into the buffer.  What lives for one layer is handed out front to back, and ``mark`` / ``release`` give a
    layer's intermediates back when the layer is done; what lives for the whole step (a step's tile lists, its table
    of rotary angles: made inside the first layer that needs them, used by all) is handed out from the back and
    stays until the step closes.  So the buffer holds one layer's worth plus the step's own.  The buffer is as large
    as the largest step so far needed: a step that outgrows it gets ordinary allocations for the overflow, and the
    buffer is enlarged after that step.  ``reserve(nbytes)`` sizes it ahead of time.  Tensors cut from it are dead
    when the next step opens; what a caller keeps (logits) must not come from here (``paused``)."""
    ALIGN = 256

    def __init__(self, device):
        self.device = torch.device(device)
        if self.device.type == "cuda" and self.device.index is None:
            self.device = torch.device("cuda", torch.cuda.current_device())
        self.buf = None
        self.typed = {}
        self.capacity = 0
        self.offset = 0          # next free byte at the front (may run past capacity: then it only measures)
        self.back = 0            # bytes handed out from the back
        self.high = 0
        self.open = False
        self.hold = 0            # > 0: paused
        self.allocations = 0     # outputs that had to come from the allocator while a step was open

    ITEMSIZE = {torch.float32: 4, torch.bfloat16: 2, torch.int32: 4, torch.float16: 2, torch.int64: 8, torch.uint8: 1}

    CANARY_BYTE = 0xA5

    def reserve(self, nbytes):
        nbytes = -(-int(nbytes) // self.ALIGN) * self.ALIGN
        if nbytes > self.capacity:
            whole = torch.empty(nbytes + self.ALIGN, dtype=torch.uint8, device=self.device)
            whole[nbytes:].fill_(self.CANARY_BYTE)              # canary words behind the buffer: nothing ever writes them
            self._whole, self.buf = whole, whole[:nbytes]
            self.capacity = nbytes
            self.typed = {dt: self.buf.view(dt) for dt in self.ITEMSIZE}     # one view per element type to slice from

    def canary_intact(self):
        """False if a kernel wrote past the end of the buffer (synchronises)."""
        return self.capacity == 0 or bool((self._whole[self.capacity:] == self.CANARY_BYTE).all())

    def step(self):
        return _OpenStep(self)

    def paused(self):
        return _Paused(self)

    def mark(self):
        return self.offset

    def release(self, mark):
        self.offset = mark

    def take(self, shape, dtype, whole_step=False):
        n = 1
        for d in shape:
            n *= d
        size = self.ITEMSIZE[dtype]
        nbytes = n * size
        padded = -(-nbytes // self.ALIGN) * self.ALIGN
        if whole_step:
            self.back += padded
            start = self.capacity - self.back
        else:
            start = self.offset
            self.offset += padded
        self.high = max(self.high, self.offset + self.back)
        if self.offset + self.back > self.capacity:
            self.allocations += 1
            return None
        first = start // size                        # start is a multiple of ALIGN, so of every element size
        return self.typed[dtype][first:first + n].view(shape)


class _OpenStep:
    def __init__(self, ws):
        self.ws = ws

    def __enter__(self):
        ws = self.ws
        ws.offset, ws.back, ws.high, ws.open = 0, 0, 0, True
        _active_workspace[0] = ws
        return ws

    def __exit__(self, *exc):
        ws = self.ws
        ws.open = False
        _active_workspace[0] = None
        if ws.high > ws.capacity:          # the next step of this size fits
            ws.reserve(ws.high + ws.high // 8)
        return False


class _Paused:
    def __init__(self, ws):
        self.ws = ws

    def __enter__(self):
        self.ws.hold += 1

    def __exit__(self, *exc):
        self.ws.hold -= 1
        return False


_active_workspace = [None]


def new_tensor(shape, dtype, device, whole_step=False):
    """An uninitialised tensor for a kernel's output: from the open step's workspace if there is one (and it is
    not paused, and lives on this device), else from the allocator.  ``whole_step``: the tensor is kept for the rest
    of the step (in the batch's plan, say), not only for the layer that makes it."""
    ws = _active_workspace[0]
    if ws is not None and ws.hold == 0 and device == ws.device:      # (a step is never open during a graph capture)
        t = ws.take(shape, dtype, whole_step)
        if t is not None:
            return t
    return torch.empty(tuple(shape), dtype=dtype, device=device)


def new_ints(values, device):
    """int32 device tensor of a host list (a step's tile lists and the like), kept for the whole step."""
    host = torch.tensor(values, dtype=torch.int32)
    out = new_tensor(host.shape, torch.int32, device, whole_step=True)
    out.copy_(host)
    return out


# ---------------------------------------------------------------------------------------------- core

def embedding(ids, table, out=None, status=None, scale=1.0, add=False):
    """out[t,:] = table[ids[t],:] * scale as float32 [T,H]; ids int32 [T]; table [V,H] float32 or bfloat16.  ``add``: the rows
    are added to ``out`` instead."""
    if add and out is None:
        raise KernelError("embedding: nothing to add to")
    lib = library("core")
    T, (V, H) = ids.numel(), table.shape
    if out is None:
        out = new_tensor((T, H), torch.float32, table.device)
    _check(lib, lib.forge_embedding(_need(ids, "ids", torch.int32), _need(table, "table", ndim=2),
                                    dtype_code(table.dtype), _need(out, "out", torch.float32), T, H, V, float(scale),
                                    1 if add else 0, _opt(status, "status", torch.int32), _stream()), "embedding")
    return out


def embedding_pair(batch, table, pair_table, last, buckets, mul_prev, mul_cur, status=None):
    """out[t,:] = table[id_t,:] + pair_table[row_t,:] as float32 [T,H], row_t = (id_{t-1} * mul_prev + id_t * mul_cur) mod buckets,
    or ``buckets`` (the table's last row) at position 0.  The token before a portion's first token is the one kept per request
    slot in ``last`` (int32 [slots, n]), which the kernel replaces with the last token the step brings for the request."""
    lib = library("core")
    ids = batch.token_ids
    T, (V, H) = ids.numel(), table.shape
    if tuple(pair_table.shape) != (buckets + 1, H) or pair_table.dtype != table.dtype:
        raise KernelError(f"embedding_pair: the second table is {tuple(pair_table.shape)} {pair_table.dtype}, expected {(buckets + 1, H)} {table.dtype}")
    out = new_tensor((T, H), torch.float32, table.device)
    _check(lib, lib.forge_embedding_pair(
        _need(ids, "ids", torch.int32), _need(batch.positions, "positions", torch.int32), _need(batch.tok_req, "tok_req", torch.int32),
        _need(batch.q_start, "q_start", torch.int32), _need(batch.slots, "slots", torch.int32), _need(last, "last", torch.int32, 2),
        last.shape[1], _need(table, "table", ndim=2), _need(pair_table, "pair_table", ndim=2), dtype_code(table.dtype),
        _need(out, "out", torch.float32), T, H, V, int(buckets), int(mul_prev), int(mul_cur), _opt(status, "status", torch.int32),
        _stream()), "embedding_pair")
    return out


def rmsnorm_add(y, w_y, residual, eps, mult=1.0, w_next=None, out_dtype=None):
    """residual += mult * y / rms(y) * w_y over the rows of float32 y, residual [T,H]; with ``w_next`` also returns
    residual / rms(residual) * w_next of the new rows in ``out_dtype`` (the next sublayer's input), else None."""
    lib = library("core")
    T, H = y.shape
    if tuple(residual.shape) != (T, H) or w_y.numel() != H or (w_next is not None and w_next.numel() != H):
        raise KernelError(f"rmsnorm_add: y {tuple(y.shape)}, residual {tuple(residual.shape)}, weights of {w_y.numel()}")
    out = new_tensor((T, H), out_dtype, y.device) if w_next is not None else None
    _check(lib, lib.forge_rmsnorm_add(_need(y, "y", torch.float32, 2), _need(w_y, "w_y", torch.float32), _need(residual, "residual", torch.float32, 2),
                                      _opt(w_next, "w_next", torch.float32), _opt(out, "out", out_dtype),
                                      dtype_code(out_dtype) if out is not None else F32, T, H, float(eps), float(mult), _stream()), "rmsnorm_add")
    return out


def streams_expand(x, S):
    """fp32 [T, W] -> fp32 [T, S*W]: S copies of every row side by side (a residual stream kept as S copies starts from the
    embedding output in all of them)."""
    lib = library("core")
    T, W = x.shape
    out = new_tensor((T, S * W), torch.float32, x.device)
    _check(lib, lib.forge_streams_expand(_need(x, "x", torch.float32, 2), _need(out, "out", torch.float32), T, int(S), W, _stream()), "streams_expand")
    return out


def streams_mix(xs, S, y=None, mix=None, out_w=None, in_next=None, w_next=None, eps=0.0, out_dtype=None, rows=None, out=None):
    """xs fp32 [T, S*W], the S copies of the stream.  With ``y`` fp32 [T, W] (a sublayer's output) every copy is rewritten at once
    from the old ones, copy t <- sum_s mix[s, t] copy_s + out_w[t] y (mix fp32 [S, S], out_w fp32 [S]).  With ``in_next`` fp32 [S]
    and ``w_next`` fp32 [W] returns rmsnorm(sum_s in_next[s] copy_s) * w_next of the (new) copies in ``out_dtype``, else None.
    ``rows`` int32 [R] (reading only): the tokens whose rows are wanted.  ``out``: the tensor that receives the normed rows instead
    of a new one."""
    lib = library("core")
    T, SW = xs.shape
    W = SW // S
    if S * W != SW or (y is not None and tuple(y.shape) != (T, W)):
        raise KernelError(f"streams_mix: {tuple(xs.shape)} is not {S} copies of rows like y's {None if y is None else tuple(y.shape)}")
    if (mix is not None and mix.numel() != S * S) or (out_w is not None and out_w.numel() != S) or (in_next is not None and in_next.numel() != S) \
            or (w_next is not None and w_next.numel() != W):
        raise KernelError("streams_mix: weights of the wrong size")
    R = T if rows is None else rows.numel()
    if in_next is None:
        out = None
    elif out is None:
        out = new_tensor((R, W), out_dtype, xs.device)
    elif tuple(out.shape) != (R, W) or out.dtype != out_dtype:
        raise KernelError(f"streams_mix: the output given is {tuple(out.shape)} {out.dtype}, the normed rows are {(R, W)} {out_dtype}")
    _check(lib, lib.forge_streams_mix(
        _need(xs, "xs", torch.float32, 2), _opt(y, "y", torch.float32), _opt(mix, "mix", torch.float32), _opt(out_w, "out_w", torch.float32),
        _opt(in_next, "in_next", torch.float32), _opt(w_next, "w_next", torch.float32), _opt(out, "out", out_dtype),
        dtype_code(out_dtype) if out is not None else F32, _opt(rows, "rows", torch.int32), R, int(S), W, float(eps), _stream()), "streams_mix")
    return out


def rmsnorm(x, weight, eps, out_dtype, rows=None, out=None):
    """y = x * rsqrt(mean(x^2)+eps) * w over the last dim of float32 x [T,H]; ``rows`` (int32) picks rows."""
    lib = library("core")
    H = x.shape[-1]
    R = x.shape[0] if rows is None else rows.numel()
    if weight.numel() != H:
        raise KernelError(f"rmsnorm: weight has {weight.numel()} elements, rows have {H}")
    if out is None:
        out = new_tensor((R, H), out_dtype, x.device)
    _check(lib, lib.forge_rmsnorm(_need(x, "x", torch.float32, 2), _need(weight, "weight", torch.float32),
                                  _need(out, "out", out_dtype), dtype_code(out_dtype),
                                  _opt(rows, "rows", torch.int32), R, H, float(eps), _stream()), "rmsnorm")
    return out


def layernorm(x, weight, bias, eps, out_dtype, rows=None):
    """y = (x - mean) / sqrt(mean((x - mean)^2) + eps) * w + b over the last dim of float32 x [T,H] (``bias`` None: no b); ``rows``
    (int32) picks rows."""
    lib = library("core")
    H = x.shape[-1]
    R = x.shape[0] if rows is None else rows.numel()
    if weight.numel() != H or (bias is not None and bias.numel() != H):
        raise KernelError(f"layernorm: weight and bias have {weight.numel()} and {None if bias is None else bias.numel()} elements, rows have {H}")
    out = new_tensor((R, H), out_dtype, x.device)
    _check(lib, lib.forge_layernorm(_need(x, "x", torch.float32, 2), _need(weight, "weight", torch.float32),
                                    _opt(bias, "bias", torch.float32), _need(out, "out", out_dtype), dtype_code(out_dtype),
                                    _opt(rows, "rows", torch.int32), R, H, float(eps), _stream()), "layernorm")
    return out


ACTIVATIONS = {"gelu": 0, "gelu_tanh": 1, "silu": 2, "xielu": 3}


def act_rows(x, out_dtype, activation, numbers=None):
    """activation(x) of float32 x [T,n] in ``out_dtype``: "gelu" (the exact one, with erf), "gelu_tanh", "silu", or "xielu" with
    ``numbers`` = (a, b): a x^2 + x/2 above zero, b (exp(x) - 1 - x) + x/2 below."""
    a, b = _act_numbers(activation, numbers)
    lib = library("core")
    T, n = x.shape
    out = new_tensor((T, n), out_dtype, x.device)
    _check(lib, lib.forge_act_rows(_need(x, "x", torch.float32, 2), n, _need(out, "out", out_dtype), dtype_code(out_dtype), T, n,
                                   ACTIVATIONS[activation], a, b, _stream()), "act_rows")
    return out


def _act_numbers(activation, numbers):
    if (activation == "xielu") != (numbers is not None):
        raise KernelError("the activation xielu takes two numbers, the others none")
    return (0.0, 0.0) if numbers is None else (float(numbers[0]), float(numbers[1]))


def depth_step(planes, n, x_plane, y1, y2=None, gates=None, weights=None, new_plane=-1, s_plane=-1, next_norm=None, out_dtype=None, rows=None,
               out=None):
    """What a layer does to a stream that is averaged over the depth.  ``planes`` fp32 [P, T, W]: plane j is what layer j - 1 left
    (0: the embedding output).  With x = planes[x_plane] and the gates sigmoid(z1), sigmoid(z2)
        X_new = x + (y1 * sigmoid(z1) + y2 * sigmoid(z2)),   s = sum_j weights[j] planes[j] + weights[n-1] X_new  (j < n - 1)
    X_new goes to planes[new_plane] and s to planes[s_plane] (-1: nowhere).  ``gates`` = (fp32 matrix, first column of z1, first
    column of z2), None: no gates; ``y2`` None: one sublayer; ``weights`` None (n = 0): s = X_new.  ``next_norm`` = ("layer" | "rms",
    weight, bias or None, eps): returns that norm of s in ``out_dtype`` ([T, W], or [R, W] with ``rows`` int32 [R], which then
    restricts everything to those tokens), written into ``out`` if given; None without it."""
    lib = library("core")
    P, T, W = planes.shape
    R = T if rows is None else rows.numel()
    if tuple(y1.shape) != (T, W) or (y2 is not None and tuple(y2.shape) != (T, W)) or max(x_plane, new_plane, s_plane, n - 2) >= P \
            or (0 if weights is None else weights.numel()) != n or (gates is not None and gates[0].shape[0] != T):
        raise KernelError(f"depth_step: planes {tuple(planes.shape)}, outputs {tuple(y1.shape)}, {n} weights do not fit")
    zp, z1, z2 = (None, 0, 0) if gates is None else gates
    kind, w, b, eps = next_norm if next_norm is not None else ("layer", None, None, 0.0)
    if w is None:
        out = None
    else:
        if w.numel() != W or (b is not None and b.numel() != W):
            raise KernelError(f"depth_step: the norm's weights do not fit rows of {W}")
        out = new_tensor((R, W), out_dtype, planes.device) if out is None else out
        if tuple(out.shape) != (R, W):
            raise KernelError(f"depth_step: the output given is {tuple(out.shape)}, the normed rows are {(R, W)}")
    _check(lib, lib.forge_depth_step(
        _need(planes, "planes", torch.float32, 3), T * W, n, x_plane, new_plane, s_plane, _opt(weights, "weights", torch.float32),
        _need(y1, "y1", torch.float32, 2), _opt(y2, "y2", torch.float32), _opt(zp, "gates", torch.float32), 0 if zp is None else zp.shape[1],
        int(z1), int(z2), _opt(w, "w", torch.float32), _opt(b, "b", torch.float32), {"rms": 0, "layer": 1}[kind], float(eps),
        _opt(out, "out", out_dtype), dtype_code(out_dtype) if out is not None else F32, _opt(rows, "rows", torch.int32), R, W, _stream()),
        "depth_step")
    return out


def join(residual, terms, eps, next_norm=None, out_dtype=None, out=None):
    """residual fp32 [T, W] += the sum of ``terms``, one to four of (y fp32 [T, W], weight fp32 [W] or None, scale): scale * y, or with a
    weight scale * y / rms(y) * weight (``eps`` inside the root).  ``next_norm`` = (weight fp32 [W], eps): also returns the new
    residual / rms * weight in ``out_dtype`` (written into ``out`` if given), else None."""
    lib = library("core")
    T, W = residual.shape
    if not 1 <= len(terms) <= 4 or any(tuple(y.shape) != (T, W) or (w is not None and w.numel() != W) for y, w, _ in terms):
        raise KernelError(f"join: {len(terms)} terms of {[tuple(y.shape) for y, _, _ in terms]} do not fit a stream of {(T, W)}")
    args = []
    for y, w, s in list(terms) + [(None, None, 0.0)] * (4 - len(terms)):
        args += [_opt(y, "y", torch.float32), _opt(w, "w", torch.float32), float(s)]
    w_next, eps_next = next_norm if next_norm is not None else (None, 0.0)
    if w_next is None:
        out = None
    else:
        out = new_tensor((T, W), out_dtype, residual.device) if out is None else out
        if tuple(out.shape) != (T, W) or w_next.numel() != W:
            raise KernelError(f"join: the next norm's output {tuple(out.shape)} and weight of {w_next.numel()} do not fit a stream of {(T, W)}")
    _check(lib, lib.forge_join(_need(residual, "residual", torch.float32, 2), len(terms), *args, float(eps), _opt(w_next, "next_w", torch.float32),
                               float(eps_next), _opt(out, "out", out_dtype), dtype_code(out_dtype) if out is not None else F32, T, W, _stream()), "join")
    return out


def rmsnorm_pair(x, w1, w2, eps, out_dtype):
    """(x * rsqrt(mean(x^2)+eps) * w1, the same * w2) over the rows of float32 x [T,H]: one read, one reduction."""
    lib = library("core")
    T, H = x.shape
    if w1.numel() != H or w2.numel() != H:
        raise KernelError(f"rmsnorm_pair: weights of {w1.numel()} and {w2.numel()} elements, rows have {H}")
    o1, o2 = new_tensor((T, H), out_dtype, x.device), new_tensor((T, H), out_dtype, x.device)
    _check(lib, lib.forge_rmsnorm_pair(_need(x, "x", torch.float32, 2), _need(w1, "w1", torch.float32), _need(w2, "w2", torch.float32),
                                       _need(o1, "out1", out_dtype), _need(o2, "out2", out_dtype), dtype_code(out_dtype), T, H,
                                       float(eps), _stream()), "rmsnorm_pair")
    return o1, o2


def rope_table(positions, head_dim, theta, by_pair=False):
    """float32 [T, head_dim/2, 2]: (cos, sin) of position / theta^(2d/head_dim) for the step's tokens; computed once
    per step and shared by every head of every layer with the same head size and base.  ``by_pair``: laid out
    [head_dim/2, T, 2] instead, which is what the projection whose epilogue rotates reads (a thread per token there,
    so neighbouring threads read neighbouring tokens of one pair)."""
    lib = library("core")
    T = positions.numel()
    shape = (head_dim // 2, T, 2) if by_pair else (T, head_dim // 2, 2)
    table = new_tensor(shape, torch.float32, positions.device, whole_step=True)
    with once_per_step():
        _check(lib, lib.forge_rope_table(_need(positions, "positions", torch.int32), _need(table, "table"), T, head_dim,
                                         float(theta), 1 if by_pair else 0, _stream()), "rope_table")
    return table


def rope_kv_write(qkv, positions, slot_mapping, kv_cache, n_heads, n_kv_heads, head_dim, page_size, theta,
                  act_dtype, rotary=True, q_out=None, table=None):
    """Rotates q and k of float32 qkv [T,(NH+2NKV)*HD], returns q [T,NH*HD] in ``act_dtype`` and writes
    k, v into ``kv_cache`` [pages,2,NKV,page,HD] at ``slot_mapping`` (int32 [T]; None or negative: no write)."""
    lib = library("core")
    T = qkv.shape[0]
    width = (n_heads + 2 * n_kv_heads) * head_dim
    if qkv.shape[1] != width:
        raise KernelError(f"rope_kv_write: qkv has width {qkv.shape[1]}, expected {width}")
    if q_out is None:
        q_out = new_tensor((T, n_heads * head_dim), act_dtype, qkv.device)
    if kv_cache is not None and kv_cache.dtype != act_dtype:
        raise KernelError("rope_kv_write: cache and activation dtypes differ")
    if kv_cache is None:
        slot_mapping = None
    _check(lib, lib.forge_rope_kv_write(_need(qkv, "qkv", torch.float32, 2), _need(positions, "positions", torch.int32),
                                        _opt(slot_mapping, "slot_mapping", torch.int32), _need(q_out, "q_out", act_dtype),
                                        _opt(kv_cache, "kv_cache"), dtype_code(act_dtype), T, n_heads, n_kv_heads,
                                        head_dim, page_size, float(theta), 1 if rotary else 0,
                                        _opt(table, "table", torch.float32), _stream()),
           "rope_kv_write")
    return q_out


GATE_ACTIVATIONS = {"silu": 0, "gelu_tanh": 1}


def silu_mul_interleaved(gu, out_dtype, out=None, activation="silu"):
    """out[t,j] = act(gu[t,2j]) * gu[t,2j+1]; gu float32 [T,2I]; act: silu, or the tanh form of gelu."""
    lib = library("core")
    T, two_i = gu.shape
    if out is None:
        out = new_tensor((T, two_i // 2), out_dtype, gu.device)
    _check(lib, lib.forge_silu_mul_interleaved(_need(gu, "gu", torch.float32, 2), _need(out, "out", out_dtype),
                                               dtype_code(out_dtype), T, two_i // 2, GATE_ACTIVATIONS[activation], _stream()),
           "silu_mul_interleaved")
    return out


def gemm_simt(a, w, bias=None, out=None, accumulate=False):
    """float32 C[M,N] = a[M,K] . w[N,K]^T (+bias) (+C when ``accumulate``), true fp32 FMA; a, w same dtype."""
    lib = library("core")
    (M, K), (N, K2) = a.shape, w.shape
    if K != K2 or a.dtype != w.dtype:
        raise KernelError(f"gemm_simt: a {tuple(a.shape)} {a.dtype} does not match w {tuple(w.shape)} {w.dtype}")
    if out is None:
        if accumulate:
            raise KernelError("gemm_simt: accumulate needs an output tensor")
        out = new_tensor((M, N), torch.float32, a.device)
    elif tuple(out.shape) != (M, N):
        raise KernelError(f"gemm_simt: out has shape {tuple(out.shape)}, expected {(M, N)}")
    _check(lib, lib.forge_gemm_simt(_need(a, "a", ndim=2), _need(w, "w", ndim=2), _opt(bias, "bias", torch.float32),
                                    _need(out, "out", torch.float32), dtype_code(a.dtype), M, N, K,
                                    1 if accumulate else 0, _stream()), "gemm_simt")
    return out


def paged_attention_simt(q, kv_cache, block_table, tok_req, positions, n_heads, n_kv_heads, head_dim, page_size,
                         window=0, scale=None, out=None):
    """Causal GQA over the paged cache, fp32 arithmetic; q [T,NH*HD]; block_table int32 [S,max_pages];
    tok_req / positions int32 [T] give each token's row of the table and its position."""
    lib = library("core")
    T = q.shape[0]
    if out is None:
        out = new_tensor(q.shape, q.dtype, q.device)
    if kv_cache.dtype != q.dtype:
        raise KernelError("paged_attention_simt: q and cache dtypes differ")
    scale = head_dim ** -0.5 if scale is None else scale
    _check(lib, lib.forge_paged_attention_simt(
        _need(q, "q", ndim=2), _need(kv_cache, "kv_cache"), _need(block_table, "block_table", torch.int32, 2),
        _need(tok_req, "tok_req", torch.int32), _need(positions, "positions", torch.int32), _need(out, "out", q.dtype),
        dtype_code(q.dtype), T, n_heads, n_kv_heads, head_dim, page_size, block_table.shape[1], int(window or 0),
        float(scale), _stream()), "paged_attention_simt")
    return out


def argmax(logits, out=None):
    """int32 [R]: index of the largest of each row of float32 logits [R,V]; lowest index wins a tie."""
    lib = library("core")
    R, V = logits.shape
    if out is None:
        out = new_tensor((R,), torch.int32, logits.device)
    _check(lib, lib.forge_argmax(_need(logits, "logits", torch.float32, 2), _need(out, "out", torch.int32), R, V,
                                 _stream()), "argmax")
    return out


def repeat_penalty(logits, tokens, counts, offsets, penalty):
    """In place: for row r and each (token, count) in [offsets[r], offsets[r+1]): logit>0 ? /pen : *pen, count times."""
    lib = library("core")
    R, V = logits.shape
    _check(lib, lib.forge_repeat_penalty(_need(logits, "logits", torch.float32, 2), _need(tokens, "tokens", torch.int32),
                                         _need(counts, "counts", torch.int32), _need(offsets, "offsets", torch.int32),
                                         _need(penalty, "penalty", torch.float32), R, V, _stream()), "repeat_penalty")
    return logits


def history_penalty(logits, counts, slot_of_row, penalty):
    """The repeat penalty with the history on the device: ``counts`` int32 [slots, V] (how often each token was
    generated, per request slot), ``slot_of_row`` int32 [R], ``penalty`` fp32 [R] (1 = none).  In place."""
    lib = library("core")
    R, V = logits.shape
    _check(lib, lib.forge_history_penalty(_need(logits, "logits", torch.float32, 2), _need(counts, "counts", torch.int32, 2),
                                          _need(slot_of_row, "slot_of_row", torch.int32), _need(penalty, "penalty", torch.float32),
                                          R, V, _stream()), "history_penalty")
    return logits


def history_add(counts, slot_of_row, tokens, penalty):
    """counts[slot_of_row[r], tokens[r]] += 1 for the rows with a penalty."""
    lib = library("core")
    R, V = tokens.numel(), counts.shape[1]
    _check(lib, lib.forge_history_add(_need(counts, "counts", torch.int32, 2), _need(slot_of_row, "slot_of_row", torch.int32),
                                      _need(tokens, "tokens", torch.int32), _need(penalty, "penalty", torch.float32), R, V,
                                      _stream()), "history_add")


def sample(logits, temperature, top_k, top_p, u, out=None):
    """int32 [R]: temperature / top-k / top-p sampling of each row with the caller's uniform numbers u [R]."""
    lib = library("core")
    R, V = logits.shape
    if out is None:
        out = new_tensor((R,), torch.int32, logits.device)
    _check(lib, lib.forge_sample(_need(logits, "logits", torch.float32, 2), _need(temperature, "temperature", torch.float32),
                                 _need(top_k, "top_k", torch.int32), _need(top_p, "top_p", torch.float32),
                                 _need(u, "u", torch.float32), _need(out, "out", torch.int32), R, V, _stream()), "sample")
    return out


# ------------------------------------------------------------------------------------------- mixers
# Attention whose heads exchange their weights (csrc/attention_headmix.cu) and mixers with a matrix of state per head
# (csrc/recurrent.cu).  Arithmetic is fp32 in both runtimes; the activation type is only what is stored.

HEADMIX_SMEM_LIMIT = 200 * 1024


def headmix_smem_bytes(H, G, D, E, TQ, KT):
    return 4 * (TQ * H * (D + E) + G * KT * (D + 1 + E) + 2 * TQ * H * KT + 2 * TQ * H + H * H)


def headmix_tile_shape(H, G, D, E, single_tokens=False):
    """(tokens per tile, keys per chunk) of the attention kernel for these head counts and sizes: of the shapes that fit
    the CTA's shared memory the one with the most (token, key) pairs, among equals the one with more tokens (a chunk's keys
    are loaded once per tile).  ``single_tokens``: a step of one token per request."""
    fits = [(TQ * KT, TQ, KT) for KT in (64, 32, 16, 8, 4, 2, 1) for TQ in ((1,) if single_tokens else (16, 8, 4, 2, 1))
            if headmix_smem_bytes(H, G, D, E, TQ, KT) <= HEADMIX_SMEM_LIMIT]
    if not fits:
        raise KernelError(f"headmix attention: {H} heads of {D}/{E} channels do not fit a CTA's shared memory")
    _, TQ, KT = max(fits)
    return TQ, KT


def headmix_plan(batch, TQ, device):
    """The step's tokens cut into tiles of up to TQ consecutive tokens of one request (first token, count), made once
    per step.  A step of single tokens that a CUDA graph replays has no list: tile i is token i."""
    if getattr(batch, "decode_only", False):
        return None, None, batch.num_tokens
    key = ("headmix", TQ)
    plan = batch.attention_plan.get(key)
    if plan is None:
        t0, n, qs = [], [], batch.host_q_start
        for s in range(batch.num_requests):
            for a in range(qs[s], qs[s + 1], TQ):
                t0.append(a)
                n.append(min(TQ, qs[s + 1] - a))
        with once_per_step():
            plan = batch.attention_plan[key] = (new_ints(t0, device), new_ints(n, device), len(t0))
    return plan


def _page_stride(cache):
    n = 1
    for d in cache.shape[1:]:
        n *= d
    return n


def headmix_prepare(proj, positions, slot_mapping, inv_freq, cache, H, G, D, E, page_size, act_dtype, has_gate=True,
                    v_first=None, lam=None, v_keep=None):
    """proj fp32 [T, >= (H+G)*D + G*E (+ H)]: rotates q and k heads on their first 2*len(inv_freq) channels (neighbouring
    pairs), blends v with ``v_first`` by ``lam`` (a one-element tensor), writes k and v at ``slot_mapping`` into ``cache``
    (None: no write) and returns (q [T, H*D] in ``act_dtype``, sigmoid gates fp32 [T, H] or None).  ``v_keep`` fp32
    [T, G*E] receives the values as projected."""
    lib = library("mixers")
    T, ld = proj.shape
    q = new_tensor((T, H * D), act_dtype, proj.device)
    gate = new_tensor((T, H), torch.float32, proj.device) if has_gate else None
    if cache is not None and cache.dtype != act_dtype:
        raise KernelError("headmix_prepare: cache and activation dtypes differ")
    if cache is None:
        slot_mapping = None
    stride = _page_stride(cache) if cache is not None else G * page_size * (D + E)
    _check(lib, lib.forge_headmix_prepare(
        _need(proj, "proj", torch.float32, 2), ld, _need(positions, "positions", torch.int32), _opt(slot_mapping, "slot_mapping", torch.int32),
        _need(inv_freq, "inv_freq", torch.float32), _opt(v_first, "v_first", torch.float32), _opt(lam, "lam", torch.float32),
        _opt(v_keep, "v_keep", torch.float32), _need(q, "q", act_dtype), _opt(cache, "cache"), _opt(gate, "gate", torch.float32),
        dtype_code(act_dtype), T, H, G, D, E, 2 * inv_freq.numel(), page_size, stride, 1 if has_gate else 0, _stream()), "headmix_prepare")
    return q, gate


def headmix_attention(q, cache, group_batch, batch, H, G, D, E, page_size, scale, window=0, keep_first=0, mix=None, gate=None):
    """Attention of every token of the step over its request's pages: ordinary softmax per head over the keys j <= i with
    (i - j < window or j < keep_first) (window 0: all), the heads' weights mixed by ``mix`` fp32 [H, H] (None: not mixed),
    applied to the values of each head's kv head, times ``gate`` fp32 [T, H] (None: no gate).  Returns [T, H*E] in q's type."""
    lib = library("mixers")
    T = q.shape[0]
    if q.dtype == torch.bfloat16 and _TENSOR_CORE_ATTENTION and lib.forge_headmix_mma_supports.fn(H, G, D, E, page_size):
        # tensor cores: one pass per head over all key/value heads' values, then the exchange between heads
        t0, tn, tiles = headmix_plan(batch, max(1, 64 // (H // G)), q.device)
        nsplit = 1
        if getattr(batch, "decode_only", False):
            # a step of single tokens brings T * G * (value chunks) CTAs: deal a request's key tiles out to several, up to
            # one CTA per SM, as far as the longest context (the graph's bucket) and the window have tiles
            ctas = T * G * -(-(G * E) // 256)
            reach = min(batch.max_context, (window + (keep_first or 0)) if window else batch.max_context)
            nsplit = max(1, min(8, -(-reach // 64), _sm_count(q.device) // max(1, ctas)))
        u = new_tensor((nsplit, T, H, G * E), torch.float32, q.device)
        part_ml = new_tensor((nsplit, T, H, 2), torch.float32, q.device) if nsplit > 1 else None
        out = new_tensor((T, H * E), q.dtype, q.device)
        _check(lib, lib.forge_headmix_attention_mma(
            _need(q, "q", torch.bfloat16, 2), _need(cache, "cache", torch.bfloat16), _need(group_batch.block_table, "block_table", torch.int32, 2),
            _need(batch.tok_req, "tok_req", torch.int32), _need(batch.positions, "positions", torch.int32), _opt(t0, "tile_t0", torch.int32),
            _opt(tn, "tile_n", torch.int32), _opt(mix, "mix", torch.float32), _opt(gate, "gate", torch.float32), _need(u, "u", torch.float32),
            _opt(part_ml, "part_ml", torch.float32), nsplit, _need(out, "out", torch.bfloat16), T, tiles, H, G, D, E, page_size, _page_stride(cache), group_batch.block_table.shape[1],
            int(window or 0), int(keep_first or 0), float(scale), _stream()), "headmix_attention_mma")
        count_launches(1)          # the kernel that takes the sum over heads
        return out
    single = getattr(batch, "decode_only", False) or batch.num_tokens == batch.num_requests
    TQ, KT = headmix_tile_shape(H, G, D, E, single_tokens=single)
    t0, tn, tiles = headmix_plan(batch, TQ, q.device)
    out = new_tensor((T, H * E), q.dtype, q.device)
    if cache.dtype != q.dtype:
        raise KernelError("headmix_attention: q and cache dtypes differ")
    _check(lib, lib.forge_headmix_attention(
        _need(q, "q", ndim=2), _need(cache, "cache"), _need(group_batch.block_table, "block_table", torch.int32, 2),
        _need(batch.tok_req, "tok_req", torch.int32), _need(batch.positions, "positions", torch.int32), _opt(t0, "tile_t0", torch.int32),
        _opt(tn, "tile_n", torch.int32), _opt(mix, "mix", torch.float32), _opt(gate, "gate", torch.float32), _need(out, "out", q.dtype),
        dtype_code(q.dtype), tiles, H, G, D, E, page_size, _page_stride(cache), group_batch.block_table.shape[1], int(window or 0),
        int(keep_first or 0), float(scale), TQ, KT, _stream()), "headmix_attention")
    return out


SCORED_KEYS_PER_CHUNK = 64          # fixed: a token's sums must not depend on the step's shape


def scored_tile_tokens(H, G, M, D, E, single_tokens=False):
    """Tokens per tile of the scored attention for these sizes: the most that fit a CTA's shared memory."""
    if single_tokens:
        return 1
    R, KT = H // G, SCORED_KEYS_PER_CHUNK
    for TQ in (16, 8, 4, 2, 1):
        if 4 * (TQ * R * M * (D + E + KT + 3) + KT * (M * D + 1 + E)) <= HEADMIX_SMEM_LIMIT:
            return TQ
    raise KernelError(f"scored attention: {H // G} heads of {M}x{D}/{E} channels do not fit a CTA's shared memory")


def _out_slice(out, n, T, dtype, device):
    """(tensor, pointer, row stride in elements) of a kernel's output of n columns: a new [T, n] tensor, or, given
    ``out`` = (matrix [T, >= col + n] of ``dtype``, first column), that slice of the matrix."""
    if out is None:
        t = new_tensor((T, n), dtype, device)
        return t, t.data_ptr(), n
    t, col = out
    if t.dtype != dtype or t.shape[0] != T or t.shape[1] < col + n:
        raise KernelError(f"output slice of {n} columns from {col} does not fit a {tuple(t.shape)} {t.dtype} matrix")
    return t, _need(t, "out", dtype, 2) + t.element_size() * int(col), t.shape[1]


def scored_prepare(proj, positions, slot_mapping, cache, H, G, M, D, E, page_size, act_dtype, inv_freq=None, q_norm=None,
                   k_norm=None, eps=0.0, temp_coef=0.0, temp_every=0.0, col=0):
    """proj fp32 [T, >= (H+G)*M*D + G*E] = [q | k | v] of a step's tokens: optionally an RMS norm over all of a token's query
    channels (weights ``q_norm`` fp32 [H*M*D]) and over all its key channels (``k_norm``), a rotation of the first
    2*len(inv_freq) channels of every map of D channels (channel i with i + half), a query temperature
    1 + temp_coef ln(floor((p+1)/temp_every) + 1); k and v go to ``slot_mapping`` in ``cache`` (None: no write); returns q
    [T, H*M*D] in ``act_dtype``.  ``col``: the first of the row's columns that are this mixer's."""
    lib = library("mixers")
    T, ld = proj.shape
    if ld - col < (H + G) * M * D + G * E:
        raise KernelError(f"scored_prepare: rows of {ld} from column {col} are too short")
    q = new_tensor((T, H * M * D), act_dtype, proj.device)
    if cache is not None and cache.dtype != act_dtype:
        raise KernelError("scored_prepare: cache and activation dtypes differ")
    if cache is None:
        slot_mapping = None
    stride = _page_stride(cache) if cache is not None else G * page_size * (M * D + E)
    rot = 0 if inv_freq is None else 2 * inv_freq.numel()
    _check(lib, lib.forge_scored_prepare(
        _need(proj, "proj", torch.float32, 2) + 4 * int(col), ld, _need(positions, "positions", torch.int32), _opt(slot_mapping, "slot_mapping", torch.int32),
        _opt(inv_freq, "inv_freq", torch.float32) if rot else None, _opt(q_norm, "q_norm", torch.float32), _opt(k_norm, "k_norm", torch.float32),
        _need(q, "q", act_dtype), _opt(cache, "cache"), dtype_code(act_dtype), T, H * M, G * M, G, D, E, rot, float(eps), float(temp_coef),
        float(temp_every), page_size, stride, _stream()), "scored_prepare")
    return q


def scored_prepare_heads(proj, positions, slot_mapping, cache, H, G, D, E, page_size, act_dtype, inv_freq=None, amp=1.0, norm=False, eps=0.0, col=0):
    """``scored_prepare`` head by head: every query and key head's first 2*len(inv_freq) channels turn by position * inv_freq (channel i
    with i + half; cos and sin times ``amp``), then with ``norm`` the head is divided by its root mean square (``eps`` inside the root)."""
    lib = library("mixers")
    T, ld = proj.shape
    if ld - col < (H + G) * D + G * E:
        raise KernelError(f"scored_prepare_heads: rows of {ld} from column {col} are too short")
    if cache is not None and cache.dtype != act_dtype:
        raise KernelError("scored_prepare_heads: cache and activation dtypes differ")
    q = new_tensor((T, H * D), act_dtype, proj.device)
    if cache is None:
        slot_mapping = None
    stride = _page_stride(cache) if cache is not None else G * page_size * (D + E)
    rot = 0 if inv_freq is None else 2 * inv_freq.numel()
    _check(lib, lib.forge_scored_prepare_heads(
        _need(proj, "proj", torch.float32, 2) + 4 * int(col), ld, _need(positions, "positions", torch.int32), _opt(slot_mapping, "slot_mapping", torch.int32),
        _opt(inv_freq, "inv_freq", torch.float32) if rot else None, float(amp), _need(q, "q", act_dtype), _opt(cache, "cache"), dtype_code(act_dtype),
        T, H, G, D, E, rot, 1 if norm else 0, float(eps), page_size, stride, _stream()), "scored_prepare_heads")
    return q


def scored_attention(q, cache, group_batch, batch, H, G, M, D, E, page_size, scale, r1=None, r2=None, lam=0.0, post=1.0, eps=0.0,
                     out_scale=1.0, out=None, window=0, chunk=0, softcap=0.0, sink=None):
    """Causal softmax attention of every token of the step over its request's pages, M maps per head (see
    csrc/attention_scored.cu): scores scale q.k - r1_h ln(1 + r2_h (i - j)); with M = 2 the maps' outputs are combined as
    a1 - lam a2, divided by their root mean square (``eps`` inside the root) and multiplied by ``post``.  Returns [T, H*E] in
    q's type, times ``out_scale``; ``out`` = (matrix, first column): written there instead (the matrix is returned).
    ``window``: key j counts for query i only if i - window < j; ``chunk``: only if i // chunk == j // chunk; ``softcap``: scores
    become softcap tanh(score / softcap); 0 switches each off.  ``sink`` fp32 [H] (M = 1): the softmax denominator of head h also counts
    exp(sink[h])."""
    lib = library("mixers")
    window, chunk, softcap = int(window or 0), int(chunk or 0), float(softcap or 0.0)
    if sink is not None and sink.numel() != H:
        raise KernelError(f"scored_attention: {sink.numel()} sinks for {H} heads")
    T = q.shape[0]
    out, out_ptr, out_ld = _out_slice(out, H * E, T, q.dtype, q.device)
    if q.dtype == torch.bfloat16 and _TENSOR_CORE_ATTENTION and lib.forge_scored_mma_supports.fn(H, G, M, D, E, page_size):
        # tensor cores: every (head, map) a one-pass attention of its own; two maps meet in a second small kernel
        t0, tn, tiles = headmix_plan(batch, max(1, 64 // (H // G)), q.device)
        nsplit = 1
        if getattr(batch, "decode_only", False):
            # a step of single tokens brings T * G * M * (value chunks) CTAs: deal a request's key tiles out to several, up to one
            # CTA per SM, as far as the longest context (the graph's bucket) has tiles
            ctas = T * G * M * -(-E // 256)
            reach = min([batch.max_context] + [n + 63 for n in (window, chunk) if n])      # a window may start inside a tile
            nsplit = max(1, min(8, -(-reach // 64), _sm_count(q.device) // max(1, ctas)))
        u = new_tensor((nsplit, T, H, M, E), torch.float32, q.device) if (M == 2 or nsplit > 1) else None
        part_ml = new_tensor((nsplit, T, H, M, 2), torch.float32, q.device) if nsplit > 1 else None
        _check(lib, lib.forge_scored_attention_mma(
            _need(q, "q", torch.bfloat16, 2), _need(cache, "cache", torch.bfloat16), _need(group_batch.block_table, "block_table", torch.int32, 2),
            _need(batch.tok_req, "tok_req", torch.int32), _need(batch.positions, "positions", torch.int32), _opt(t0, "tile_t0", torch.int32),
            _opt(tn, "tile_n", torch.int32), _opt(r1, "r1", torch.float32), _opt(r2, "r2", torch.float32), _opt(u, "u", torch.float32),
            _opt(part_ml, "part_ml", torch.float32), nsplit, out_ptr, T, tiles, H, G, M, D, E, page_size, _page_stride(cache), group_batch.block_table.shape[1],
            float(scale), float(lam), float(post), float(eps), float(out_scale), out_ld, window, chunk, softcap, _opt(sink, "sink", torch.float32), _stream()),
            "scored_attention_mma")
        if M == 2 or nsplit > 1:
            count_launches(1)      # the kernel that puts the runs of key tiles, and the two maps, together
        return out
    single = getattr(batch, "decode_only", False) or batch.num_tokens == batch.num_requests
    TQ = scored_tile_tokens(H, G, M, D, E, single_tokens=single)
    t0, tn, tiles = headmix_plan(batch, TQ, q.device)
    if cache.dtype != q.dtype:
        raise KernelError("scored_attention: q and cache dtypes differ")
    _check(lib, lib.forge_scored_attention(
        _need(q, "q", ndim=2), _need(cache, "cache"), _need(group_batch.block_table, "block_table", torch.int32, 2),
        _need(batch.tok_req, "tok_req", torch.int32), _need(batch.positions, "positions", torch.int32), _opt(t0, "tile_t0", torch.int32),
        _opt(tn, "tile_n", torch.int32), _opt(r1, "r1", torch.float32), _opt(r2, "r2", torch.float32), out_ptr,
        dtype_code(q.dtype), tiles, H, G, M, D, E, page_size, _page_stride(cache), group_batch.block_table.shape[1], float(scale),
        float(lam), float(post), float(eps), float(out_scale), TQ, SCORED_KEYS_PER_CHUNK, out_ld, window, chunk, softcap,
        _opt(sink, "sink", torch.float32), _stream()), "scored_attention")
    return out


def _cols(t, off=0):
    """(pointer, leading dimension) of the columns of fp32 matrix ``t`` from ``off`` on."""
    if t is None:
        return None, 0
    return _need(t, "matrix", torch.float32, 2) + 4 * int(off), t.shape[1]


STATE_SCANS = {"decay_bonus": 0, "delta": 1, "gated_write": 2}


def state_scan(kind, r, k, v, x, w0, state, batch, N, K, y=None, a0=None, bonus=None, last_in=None, prev_off=0, KV=None):
    """The recurrence of a mixer with a [K, K] state per head (``kind``: "decay_bonus" or "delta", see csrc/recurrent.cu)
    over the step's tokens, request by request, from and into ``state`` fp32 [slots, row].  r, k, v, x, y: (fp32 matrix,
    first column) pairs with N*K columns from there; x (and y) are overwritten with the decays (and removal rates) made from
    them; returns fp32 [T, N*K].  ``last_in`` ("decay_bonus"): the mixer's input
    [T, W], whose last row per request is kept in the state row at ``prev_off``.
    "gated_write": no k (None); x is the forget gate's input, w0 its bias, a0 its lower bound; r becomes silu(r) in place; v
    has N*KV columns and so has the result; a head's state is [K, KV]."""
    lib = library("mixers")
    T = r[0].shape[0]
    KV = K if KV is None else int(KV)
    out = new_tensor((T, N * KV), torch.float32, r[0].device)
    (rp, rl), (kp, kl), (vp, vl), (xp, xl) = _cols(*r), _cols(*k) if k is not None else (None, 0), _cols(*v), _cols(*x)
    yp, yl = _cols(*y) if y is not None else ((rp, rl) if kind == "gated_write" else (None, 0))
    W = last_in.shape[1] if last_in is not None else 0
    inv = new_tensor((T, N), torch.float32, r[0].device) if kind == "delta" else None       # the unit keys' divisors
    _check(lib, lib.forge_state_scan(
        STATE_SCANS[kind], rp, rl, kp, kl, vp, vl, xp, xl, yp, yl, _need(w0, "w0", torch.float32), _opt(a0, "a0", torch.float32),
        _opt(bonus, "bonus", torch.float32), _opt(inv, "inv", torch.float32), _need(state, "state", torch.float32, 2), state.shape[1],
        _need(batch.q_start, "q_start", torch.int32), _need(batch.slots, "slots", torch.int32), _need(out, "out", torch.float32),
        _opt(last_in, "last_in"), dtype_code(last_in.dtype) if last_in is not None else 0, W, int(prev_off), T, batch.num_requests, N, K, KV,
        _stream()), "state_scan")
    count_launches(1)              # the kernel that makes the decays (and removal rates) from x (and y), in place
    return out


def retention_scan(q, k, v, batch, freq, k_scale, decay, state, N, K, KV):
    """Retention over the step's tokens, request by request, from and into ``state`` fp32 [slots, N*K*KV]: q, k ((fp32 matrix,
    first column) pairs, N*K columns) are rotated IN PLACE on their first 2*len(freq) channels (channel i with i + half) by
    position * freq, k is multiplied by ``k_scale``; S <- decay[n] S + k v^T, out = S^T q per head.  v (N*KV columns); returns
    fp32 [T, N*KV]."""
    lib = library("mixers")
    T = q[0].shape[0]
    out = new_tensor((T, N * KV), torch.float32, q[0].device)
    (qp, ql), (kp, kl), (vp, vl) = _cols(*q), _cols(*k), _cols(*v)
    rot = 0 if freq is None else 2 * freq.numel()
    _check(lib, lib.forge_retention_scan(
        qp, ql, kp, kl, vp, vl, _need(batch.positions, "positions", torch.int32), _opt(freq, "freq", torch.float32) if rot else None, rot,
        float(k_scale), _need(decay, "decay", torch.float32), _need(state, "state", torch.float32, 2), state.shape[1],
        _need(batch.q_start, "q_start", torch.int32), _need(batch.slots, "slots", torch.int32), _need(out, "out", torch.float32), T,
        batch.num_requests, N, K, KV, _stream()), "retention_scan")
    count_launches(1)              # the kernel that rotates and scales q and k, in place
    return out


def gla_scan(q, k, v, hidden, rank, w2t, bias, tau, batch, state, N, K, KV):
    """Gated linear attention over the step's tokens, request by request, from and into ``state`` fp32 [slots, N*K*KV]: decays
    a = sigmoid(hidden . w2 + bias)^(1/tau) per key channel (``w2t`` fp32 [rank, N*K]), S <- diag(a) S + k v^T, out = K^-1/2 S^T q per
    head.  q, k, v, hidden: (fp32 matrix, first column) pairs; returns fp32 [T, N*KV]."""
    lib = library("mixers")
    T = q[0].shape[0]
    if tuple(w2t.shape) != (rank, N * K) or bias.numel() != N * K or not tau > 0.0:
        raise KernelError(f"gla_scan: w2 {tuple(w2t.shape)}, {bias.numel()} biases and tau {tau} do not fit {N} heads of {K}, rank {rank}")
    decay = new_tensor((T, N * K), torch.float32, q[0].device)
    out = new_tensor((T, N * KV), torch.float32, q[0].device)
    (qp, ql), (kp, kl), (vp, vl), (up, ul) = _cols(*q), _cols(*k), _cols(*v), _cols(*hidden)
    _check(lib, lib.forge_gla_scan(
        qp, ql, kp, kl, vp, vl, up, ul, int(rank), _need(w2t, "w2t", torch.float32, 2), _need(bias, "bias", torch.float32), 1.0 / float(tau),
        float(K) ** -0.5, _need(decay, "decay", torch.float32), _need(state, "state", torch.float32, 2), state.shape[1],
        _need(batch.q_start, "q_start", torch.int32), _need(batch.slots, "slots", torch.int32), _need(out, "out", torch.float32), T,
        batch.num_requests, N, K, KV, _stream()), "gla_scan")
    count_launches(1)              # the kernel that makes the decays
    return out


GLA_TOKEN_STATE = 1 << 15           # numbers of a head's state that one CTA walks at most


def gla_token_supports(batch, N, K, KV, rank):
    """A step in which every request brings one token, and heads small enough for one CTA each."""
    return batch.num_tokens == batch.num_requests and K * KV <= GLA_TOKEN_STATE and 4 * (3 * K + rank + max(KV, 1024)) <= 48 * 1024


def gla_token(q, k, v, gate, hidden, rank, w2t, bias, tau, batch, state, N, K, KV, weight, eps, out_dtype, out=None):
    """``gla_scan`` for a step in which every request brings one token, followed by the head's norm (``weight`` fp32 [KV], eps) and the
    silu of ``gate`` ((fp32 matrix, first column)): one kernel; returns [T, N*KV] in ``out_dtype`` (or writes them into ``out`` =
    (matrix, first column))."""
    lib = library("mixers")
    T = q[0].shape[0]
    if T != batch.num_requests or tuple(w2t.shape) != (rank, N * K) or bias.numel() != N * K or weight.numel() != KV or not tau > 0.0:
        raise KernelError(f"gla_token: {T} tokens of {batch.num_requests} requests, w2 {tuple(w2t.shape)}, {weight.numel()} weights do not fit")
    out, out_ptr, out_ld = _out_slice(out, N * KV, T, out_dtype, q[0].device)
    (qp, ql), (kp, kl), (vp, vl), (gp, gl), (up, ul) = _cols(*q), _cols(*k), _cols(*v), _cols(*gate), _cols(*hidden)
    _check(lib, lib.forge_gla_token(
        qp, ql, kp, kl, vp, vl, gp, gl, up, ul, int(rank), _need(w2t, "w2t", torch.float32, 2), _need(bias, "bias", torch.float32), 1.0 / float(tau),
        float(K) ** -0.5, _need(state, "state", torch.float32, 2), state.shape[1], _need(batch.q_start, "q_start", torch.int32),
        _need(batch.slots, "slots", torch.int32), _need(weight, "weight", torch.float32), float(eps), out_ptr, dtype_code(out_dtype), out_ld,
        batch.num_requests, N, K, KV, _stream()), "gla_token")
    return out


# recurrences whose inputs pass silu, or a short convolution and silu, first (csrc/recurrent_token.cu), eight tokens at a time
# (csrc/recurrent_block.cu)

def _gram(batch, T, heads, device):
    """Room for the products of a block's keys with its keys and queries, for every head of keys and every block of every request."""
    return new_tensor(((T // 8 + batch.num_requests) * heads * 64,), torch.float32, device)


def token_state_supports(batch, K, V, delta):
    """A step in which every request brings one token, and heads of K x V numbers that the kernel of single tokens takes."""
    return batch.num_tokens == batch.num_requests and bool(library("mixers").forge_token_state_supports.fn(int(K), int(V), 1 if delta else 0))


def lightning_scan(proj, col, decay, batch, state, N, K, V):
    """proj fp32 [T, >= col + N*(2K+V)]: [q | k | v] from column ``col``, which pass silu IN PLACE; S <- decay[n] S + k v^T, o = S^T q over the
    step's tokens, request by request, from and into ``state`` fp32 [slots, >= N*K*V].  Returns fp32 [T, N*V]."""
    lib = library("mixers")
    T = proj.shape[0]
    out = new_tensor((T, N * V), torch.float32, proj.device)
    p, ld = _cols(proj, col)
    _check(lib, lib.forge_lightning_scan(p, ld, _need(decay, "decay", torch.float32), _need(_gram(batch, T, N, proj.device), "gram"), _need(state, "state", torch.float32, 2), state.shape[1],
                                         _need(batch.q_start, "q_start", torch.int32), _need(batch.slots, "slots", torch.int32),
                                         _need(out, "out", torch.float32), T, batch.num_requests, N, K, V, _stream()), "lightning_scan")
    count_launches(2)              # the kernels that apply silu and take the blocks' products
    return out


def lightning_token(proj, col, decay, batch, state, N, K, V):
    """``lightning_scan`` for a step in which every request brings one token (proj is left as it is)."""
    lib = library("mixers")
    T = proj.shape[0]
    if T != batch.num_requests:
        raise KernelError(f"lightning_token: {T} tokens of {batch.num_requests} requests")
    out = new_tensor((T, N * V), torch.float32, proj.device)
    p, ld = _cols(proj, col)
    _check(lib, lib.forge_lightning_token(p, ld, _need(decay, "decay", torch.float32), _need(state, "state", torch.float32, 2), state.shape[1],
                                          _need(batch.q_start, "q_start", torch.int32), _need(batch.slots, "slots", torch.int32),
                                          _need(out, "out", torch.float32), T, N, K, V, _stream()), "lightning_token")
    return out


def gated_rows(o, weight, gate, eps, out_dtype, out=None):
    """o fp32 [T, n] / rms(o over the row) * ``weight`` fp32 [n] * sigmoid of ``gate`` ((fp32 matrix, first column)), [T, n] in ``out_dtype``
    (or written into ``out`` = (matrix, first column), the matrix returned)."""
    lib = library("mixers")
    T, n = o.shape
    if weight.numel() != n:
        raise KernelError(f"gated_rows: {weight.numel()} weights for rows of {n}")
    out, out_ptr, out_ld = _out_slice(out, n, T, out_dtype, o.device)
    gp, gl = _cols(*gate)
    _check(lib, lib.forge_gated_rows(_need(o, "o", torch.float32, 2), _need(weight, "weight", torch.float32), gp, gl, out_ptr, dtype_code(out_dtype),
                                     out_ld, T, n, float(eps), _stream()), "gated_rows")
    return out


def _delta_state(conv_w, state, N, M, K, V):
    """(taps, first number of the ring in a state row) of the gated delta rule's state; checks the sizes."""
    C, taps = 2 * M * K + N * V, conv_w.shape[0]
    ring_off = N * K * V
    if conv_w.shape[1] != C or state.shape[1] < ring_off + taps * C:
        raise KernelError(f"gated delta rule: convolutions {tuple(conv_w.shape)} and state rows of {state.shape[1]} do not fit {N}/{M} heads of {K} x {V}")
    return taps, ring_off


def gated_delta_prepare(proj, col, b_col, a_col, conv_w, decay_rate, dt, batch, state, N, M, K, V):
    """proj fp32 [T, ..]: [q: M*K | k: M*K | v: N*V] from column ``col``, and from ``b_col`` and ``a_col`` on the N inputs each of the write
    strengths and the decays.  Convolves q, k, v over time (``conv_w`` fp32 [taps, 2*M*K + N*V], row j the weights of the token
    j before; earlier inputs from the ring in the request's ``state`` row behind its N*K*V numbers, which is brought up to date), silu, q and k to unit vectors, q times K^-1/2.
    Returns (qkv fp32 [T, 2*M*K + N*V], decays fp32 [T, N], strengths fp32 [T, N])."""
    lib = library("mixers")
    T = proj.shape[0]
    taps, ring_off = _delta_state(conv_w, state, N, M, K, V)
    qkv = new_tensor((T, 2 * M * K + N * V), torch.float32, proj.device)
    g, beta = new_tensor((T, N), torch.float32, proj.device), new_tensor((T, N), torch.float32, proj.device)
    p, ld = _cols(proj, col)
    _check(lib, lib.forge_delta_prepare(
        p, ld, int(b_col - col), int(a_col - col), _need(conv_w, "conv_w", torch.float32, 2), taps, _need(state, "state", torch.float32, 2), state.shape[1],
        ring_off, _need(batch.tok_req, "tok_req", torch.int32), _need(batch.q_start, "q_start", torch.int32),
        _need(batch.positions, "positions", torch.int32), _need(batch.slots, "slots", torch.int32), _need(decay_rate, "decay_rate", torch.float32),
        _need(dt, "dt", torch.float32), _need(qkv, "qkv"), _need(g, "g"), _need(beta, "beta"), T, batch.num_requests, N, M, K, V, _stream()),
        "gated_delta_prepare")
    count_launches(1)              # the kernel that brings the rings up to date
    return qkv, g, beta


def gated_delta_scan(qkv, g, beta, batch, state, N, M, K, V):
    """The gated delta rule over the step's tokens, request by request, from and into ``state``: per head n with q and k of head n // (N/M),
    S <- g S;  S <- S + k (beta (v - S^T k))^T;  o = S^T q.  The inputs as ``gated_delta_prepare`` leaves them; returns fp32 [T, N*V]."""
    lib = library("mixers")
    T = qkv.shape[0]
    out = new_tensor((T, N * V), torch.float32, qkv.device)
    (qp, ld), (kp, _), (vp, _) = _cols(qkv, 0), _cols(qkv, M * K), _cols(qkv, 2 * M * K)
    _check(lib, lib.forge_gated_delta_scan(
        qp, ld, kp, ld, vp, ld, _need(g, "g", torch.float32, 2), _need(beta, "beta", torch.float32, 2), _need(_gram(batch, T, M, qkv.device), "gram"),
        _need(state, "state", torch.float32, 2), state.shape[1], _need(batch.q_start, "q_start", torch.int32), _need(batch.slots, "slots", torch.int32), _need(out, "out", torch.float32),
        T, batch.num_requests, N, M, K, V, _stream()), "gated_delta_scan")
    count_launches(1)              # the kernel that takes the blocks' products
    return out


def gated_delta_token(proj, col, g_col, b_col, a_col, conv_w, decay_rate, dt, batch, state, N, M, K, V, weight, eps, out_dtype, out=None):
    """Both of the above, the heads' norm (``weight`` fp32 [V], eps) and silu of the gate (N*V columns from ``g_col``) for a step in which every
    request brings one token: one kernel; returns [T, N*V] in ``out_dtype`` (or writes them into ``out`` = (matrix, first column))."""
    lib = library("mixers")
    T = proj.shape[0]
    if T != batch.num_requests or weight.numel() != V:
        raise KernelError(f"gated_delta_token: {T} tokens of {batch.num_requests} requests, {weight.numel()} norm weights for {V} channels")
    taps, ring_off = _delta_state(conv_w, state, N, M, K, V)
    out, out_ptr, out_ld = _out_slice(out, N * V, T, out_dtype, proj.device)
    p, ld = _cols(proj, col)
    _check(lib, lib.forge_gated_delta_token(
        p, ld, int(g_col - col), int(b_col - col), int(a_col - col), _need(conv_w, "conv_w", torch.float32, 2), taps, _need(state, "state", torch.float32, 2),
        state.shape[1], ring_off, _need(batch.q_start, "q_start", torch.int32), _need(batch.positions, "positions", torch.int32),
        _need(batch.slots, "slots", torch.int32), _need(decay_rate, "decay_rate", torch.float32), _need(dt, "dt", torch.float32),
        _need(weight, "weight", torch.float32), float(eps), out_ptr, dtype_code(out_dtype), out_ld, T, N, M, K, V, _stream()), "gated_delta_token")
    return out


# ---------------------------------------------------------------------------------------------- latent attention

LATENT_SPLITS = 16                  # runs that a request's rows are dealt out in, at most
LATENT_KEYS_PER_CHUNK = 32          # fixed: a token's sums must not depend on the step's shape


def latent_prepare(proj, batch, slot_mapping, cache, freq, amp, wq, wc, Cq, C, R, eps, act_dtype, halves=False):
    """proj fp32 [T, Cq (+ C + R)], or (matrix, first column): the query latent normed (weight ``wq``) -> [T, Cq] in ``act_dtype``
    (Cq = 0: none, returns None); with C > 0 the normed key/value latent (weight ``wc``) and the rotated shared key part go to
    ``slot_mapping`` in ``cache`` (rows of C + R).  ``halves``: the rotation pairs channel i with i + R/2 instead of 2i with 2i + 1."""
    lib = library("latent")
    proj, col = proj if isinstance(proj, tuple) else (proj, 0)
    T, ld = proj.shape
    store = C > 0 and cache is not None and slot_mapping is not None
    if Cq == 0 and not store:
        return None
    if ld < col + Cq + (C + R if store else 0):
        raise KernelError(f"latent_prepare: rows of {ld} numbers from column {col} do not hold {Cq} + {C} + {R}")
    cq = new_tensor((T, Cq), act_dtype, proj.device) if Cq else None
    if store and cache.dtype != act_dtype:
        raise KernelError("latent_prepare: cache and activation dtypes differ")
    _check(lib, lib.forge_latent_prepare(
        _cols(proj, col)[0], ld, _need(batch.positions, "positions", torch.int32),
        _need(slot_mapping, "slot_mapping", torch.int32) if store else None, _opt(freq, "freq", torch.float32), float(amp),
        _opt(wq, "wq", torch.float32), _opt(wc, "wc", torch.float32), _opt(cq, "cq", act_dtype), _need(cache, "cache") if store else None,
        dtype_code(act_dtype), T, Cq, C if store else 0, R, float(eps), 1 if halves else 0, _stream()), "latent_prepare")
    return cq


def head_linear(x, w, H, K, N, out_dtype, R=0, positions=None, freq=None, amp=1.0, simt=False, gate=None, halves=False, out=None):
    """out[t, h, :N] = sum_k x[t, h, k] w[h, k, :] for the H heads of x [T, H*(K+R)] (fp32 or the weights' type; or (matrix, first
    column), fp32); with R > 0 a head's last R channels are rotated by position * freq (channel 2i with 2i+1, with ``halves`` i with
    i + R/2; cos and sin times ``amp``) and follow the N outputs.  w [H, K, N] in ``out_dtype``; returns [T, H*(N+R)] in ``out_dtype``
    (or writes them into ``out`` = (matrix, first column)).  bfloat16 weights go to the tensor cores (an fp32 x rounded to bfloat16 on
    the way) unless ``simt`` asks for fp32 multiply-adds on the inputs as they are.  ``gate`` = (fp32 matrix, first column) or (fp32
    matrix, first column, "head"): the outputs are multiplied by the sigmoid of the H*N numbers from that column of the token's row,
    or of the H numbers there, one per head."""
    lib = library("latent")
    gate_ptr, gate_ld, gate_hs, gate_cs = None, 0, 0, 0
    if gate is not None:
        gate_hs, gate_cs = (1, 0) if gate[2:] == ("head",) else (N, 1)
        gate_ptr, gate_ld = _cols(gate[0], gate[1])
    T = (x[0] if isinstance(x, tuple) else x).shape[0]
    if gate is not None and (R or gate[0].shape[0] != T or gate[0].shape[1] < gate[1] + (H if gate_hs == 1 and gate_cs == 0 else H * N)):
        raise KernelError("head_linear: a gate wants rows of the step's tokens with H*N columns (or H), and no rotated channels")
    if isinstance(x, tuple):
        (x, col), fits = x, x[0].shape[1] >= x[1] + H * (K + R)
        x_ptr, x_ld = _cols(x, col)
    else:
        x_ptr, x_ld, fits = _need(x, "x", ndim=2), x.shape[1], x.shape[1] == H * (K + R)
    if not fits or tuple(w.shape) != (H, K, N) or w.dtype != out_dtype:
        raise KernelError(f"head_linear: x {tuple(x.shape)}, w {tuple(w.shape)} {w.dtype} do not fit {H} heads of {K}+{R} -> {N}")
    out, out_ptr, out_ld = _out_slice(out, H * (N + R), T, out_dtype, x.device)
    _check(lib, lib.forge_head_linear(
        x_ptr, dtype_code(x.dtype), x_ld, K + R, _need(w, "w"), out_ptr, dtype_code(out_dtype),
        out_ld, N + R, _opt(positions, "positions", torch.int32), _opt(freq, "freq", torch.float32), float(amp), T, H, K, N, R,
        1 if simt else 0, gate_ptr, gate_ld, gate_hs, gate_cs, 1 if halves else 0, _stream()), "head_linear")
    return out


def latent_tile_shape(H, C, R, single_tokens=False):
    """(tokens per tile, heads per CTA) of the latent attention for these sizes: of the shapes that fit a CTA's shared memory
    the one with the most rows, among equals the one with more heads (so that a chunk's rows are loaded for as many heads
    as possible)."""
    KT = LATENT_KEYS_PER_CHUNK
    best = None
    for TQ in ((1,) if single_tokens else (16, 8, 4, 2, 1)):
        for HG in sorted({H, -(-H // 2), -(-H // 4), -(-H // 8), -(-H // 16), 1}, reverse=True):
            if 4 * (TQ * HG * (2 * C + R + KT + 3) + KT * (C + R + 1)) <= HEADMIX_SMEM_LIMIT:
                if best is None or TQ * HG > best[0] * best[1]:
                    best = (TQ, HG)
                break
    if best is None:
        raise KernelError(f"latent attention: a latent of {C}+{R} channels does not fit a CTA's shared memory")
    return best


def latent_attention(q, cache, group_batch, batch, H, C, R, page_size, scale, window=0, sink=None):
    """Causal softmax attention of every token's H absorbed queries (q [T, H*(C+R)]) over its request's latent rows in
    ``cache`` (rows of C + R; the values are a row's first C channels); returns the weighted latents [T, H*C] in q's type.
    ``window``: position i reads the rows j with i - window < j <= i (0: every j <= i); ``sink`` fp32 [H]: exp(sink_h) is
    added to the softmax denominator of head h."""
    lib = library("latent")
    window = int(window or 0)
    if sink is not None and sink.numel() != H:
        raise KernelError(f"latent_attention: {sink.numel()} sinks for {H} heads")
    T = q.shape[0]
    if cache.dtype != q.dtype:
        raise KernelError("latent_attention: q and cache dtypes differ")
    if q.dtype == torch.bfloat16 and _TENSOR_CORE_ATTENTION and lib.forge_latent_mma_supports.fn(H, C, R, page_size):
        # tensor cores: rows of (token, head) over the same tiles of latent rows
        HG = lib.forge_latent_mma_heads.fn(H)
        t0, tn, tiles = headmix_plan(batch, max(1, 64 // HG), q.device)
        nsplit = 1
        if getattr(batch, "decode_only", False):
            # a step of single tokens brings T * (head groups) * (value chunks) CTAs: deal a request's tiles out to several, up to
            # one CTA per SM, as far as the longest context (the graph's bucket) has tiles
            ctas = T * -(-H // HG) * -(-C // 256)
            reach = min(batch.max_context, window + 63) if window else batch.max_context
            nsplit = max(1, min(LATENT_SPLITS, -(-reach // 64), _sm_count(q.device) // max(1, ctas)))
        u = new_tensor((nsplit, T, H, C), torch.float32, q.device) if nsplit > 1 else None
        part_ml = new_tensor((nsplit, T, H, 2), torch.float32, q.device) if nsplit > 1 else None
        out = new_tensor((T, H * C), q.dtype, q.device)
        _check(lib, lib.forge_latent_attention_mma(
            _need(q, "q", torch.bfloat16, 2), _need(cache, "cache", torch.bfloat16), _need(group_batch.block_table, "block_table", torch.int32, 2),
            _need(batch.tok_req, "tok_req", torch.int32), _need(batch.positions, "positions", torch.int32), _opt(t0, "tile_t0", torch.int32),
            _opt(tn, "tile_n", torch.int32), _opt(u, "u", torch.float32), _opt(part_ml, "part_ml", torch.float32), nsplit,
            _need(out, "out", torch.bfloat16), T, tiles, H, C, R, page_size, group_batch.block_table.shape[1], float(scale), window,
            _opt(sink, "sink", torch.float32), _stream()), "latent_attention_mma")
        if nsplit > 1:
            count_launches(1)      # the kernel that puts the runs of tiles together
        return out
    single = getattr(batch, "decode_only", False) or batch.num_tokens == batch.num_requests
    TQ, HG = latent_tile_shape(H, C, R, single_tokens=single)
    t0, tn, tiles = headmix_plan(batch, TQ, q.device)
    out = new_tensor((T, H * C), q.dtype, q.device)
    _check(lib, lib.forge_latent_attention(
        _need(q, "q", ndim=2), _need(cache, "cache"), _need(group_batch.block_table, "block_table", torch.int32, 2),
        _need(batch.tok_req, "tok_req", torch.int32), _need(batch.positions, "positions", torch.int32), _opt(t0, "tile_t0", torch.int32),
        _opt(tn, "tile_n", torch.int32), _need(out, "out", q.dtype), dtype_code(q.dtype), tiles, H, HG, C, R, page_size,
        group_batch.block_table.shape[1], float(scale), TQ, LATENT_KEYS_PER_CHUNK, window, _opt(sink, "sink", torch.float32), _stream()),
        "latent_attention")
    return out


# ---------------------------------------------------------------------------------------------- routed experts

def moe_route(x, router, top, softmax=False, renorm=False, correction=None, groups=0, keep=0, factor=1.0, group_top=1):
    """(int32 [T, top] experts, fp32 [T, top] weights): the ``top`` largest of sigmoid (or softmax) of router . x per token, the lower
    index winning a tie; the weights are those scores, divided by their sum with ``renorm``, times ``factor``.  router fp32 [E, W];
    fp32 arithmetic.  ``correction`` fp32 [E]: experts are ranked by score + correction (the weights stay the scores).  ``groups``
    > 1: the experts are cut into that many consecutive blocks of equal size, a block is ranked by the largest ranking number in it
    (``group_top`` 2: by the sum of its two largest), and only the ``keep`` best blocks' experts take part in the ranking."""
    lib = library("moe")
    T, W = x.shape
    E = router.shape[0]
    idx = new_tensor((T, top), torch.int32, x.device)
    wts = new_tensor((T, top), torch.float32, x.device)
    _check(lib, lib.forge_moe_route(_need(x, "x", ndim=2), dtype_code(x.dtype), _need(router, "router", torch.float32, 2), _need(idx, "idx"),
                                    _need(wts, "wts"), T, W, E, int(top), 1 if softmax else 0, 1 if renorm else 0,
                                    _opt(correction, "correction", torch.float32), int(groups or 0), int(keep or 0), int(group_top), float(factor),
                                    _stream()), "moe_route")
    return idx, wts


def moe_pairs(x, idx, wts, w_gate_up, w_down):
    """y fp32 [T, W] = sum_k wts[t,k] * W_down[e] (silu(W_gate[e] x_t) * (W_up[e] x_t)), e = idx[t,k], every (token, expert) pair
    on its own; w_gate_up [E, 2F, W] (row 2j the gate's, 2j+1 the up's), w_down [E, W, F] in x's type.  Reads everything from
    device memory."""
    lib = library("moe")
    T, W = x.shape
    E, F2, _ = w_gate_up.shape
    F = F2 // 2
    top = idx.shape[1]
    act = new_tensor((T * top, F), x.dtype, x.device)
    gp = _need(w_gate_up, "w_gate_up", x.dtype)
    _check(lib, lib.forge_moe_pair_gate_up(_need(x, "x", ndim=2), gp, gp + W * x.element_size(), _need(idx, "idx", torch.int32),
                                           _need(act, "act"), dtype_code(x.dtype), T, W, F, top, 2 * W, _stream()), "moe_pair_gate_up")
    y = new_tensor((T, W), torch.float32, x.device)
    _check(lib, lib.forge_moe_pair_down(_need(act, "act"), _need(w_down, "w_down", x.dtype), _need(idx, "idx", torch.int32),
                                        _need(wts, "wts", torch.float32), _need(y, "y"), dtype_code(x.dtype), T, W, F, top, _stream()),
           "moe_pair_down")
    return y


def moe_experts_supported(P, W, F):
    return bool(library("moe").forge_moe_expert_supports.fn(int(P), int(W), int(F)))


def moe_experts(x, idx, wts, w_gate_up, w_down):
    """The same as ``moe_pairs`` to the last bit, expert by expert: an expert's weight rows are read once for up to eight of the
    pairs that chose it instead of once per pair.  Reads everything from device memory; three launches."""
    lib = library("moe")
    T, W = x.shape
    E, F2, _ = w_gate_up.shape
    F = F2 // 2
    top = idx.shape[1]
    act = new_tensor((T * top, F), x.dtype, x.device)
    ys = new_tensor((T * top, W), torch.float32, x.device)
    gp = _need(w_gate_up, "w_gate_up", x.dtype)
    _check(lib, lib.forge_moe_expert_rows(_need(x, "x", ndim=2), gp, gp + W * x.element_size(), 2 * W, _need(w_down, "w_down", x.dtype),
                                          _need(idx, "idx", torch.int32), _need(act, "act"), _need(ys, "ys"), dtype_code(x.dtype), T, W, F, E, top,
                                          _stream()), "moe_expert_rows")
    count_launches(1)
    return moe_combine(ys, _pair_numbers(T, top, x.device), wts)


_PAIR_NUMBERS = {}


def _pair_numbers(T, top, device):
    """int32 [T, top] = the pairs' own numbers (kept: a CUDA graph must not allocate it anew at every capture)."""
    key = (T, top, str(device))
    t = _PAIR_NUMBERS.get(key)
    if t is None:
        if len(_PAIR_NUMBERS) > 256:
            _PAIR_NUMBERS.clear()
        t = _PAIR_NUMBERS[key] = torch.arange(T * top, dtype=torch.int32, device=device).view(T, top)
    return t


def moe_sort(x, idx, E, cap=0):
    """The (token, expert) pairs ranked by (expert, token): returns (xg [T*top, W]: each pair's input row at its rank, counts int32 [E],
    dest int32 [T, top]: the rank of every pair).  With ``cap`` (at least T) every expert has room for ``cap`` rows: xg [E*cap, W], expert
    e's rows from e*cap on, the rows beyond its count left as they were; nothing then depends on the counts' values on the host."""
    lib = library("moe")
    T, W = x.shape
    top = idx.shape[1]
    rank = new_tensor((T * top,), torch.int32, x.device)
    dest = new_tensor((T, top), torch.int32, x.device)
    counts = new_tensor((E,), torch.int32, x.device)
    if cap and cap < T:
        raise KernelError(f"moe_sort: room for {cap} rows per expert, a step of {T} tokens")
    xg = new_tensor((E * cap if cap else T * top, W), x.dtype, x.device)
    _check(lib, lib.forge_moe_sort(_need(x, "x", ndim=2), dtype_code(x.dtype), _need(idx, "idx", torch.int32), _need(rank, "rank"),
                                   _need(counts, "counts"), _need(dest, "dest"), _need(xg, "xg"), T, W, E, top, int(cap), _stream()), "moe_sort")
    count_launches(1)
    return xg, counts, dest


def moe_combine(ys, dest, wts):
    """y fp32 [T, W] = sum_k wts[t,k] * ys[dest[t,k], :], k in order."""
    lib = library("moe")
    T, top = dest.shape
    W = ys.shape[1]
    y = new_tensor((T, W), torch.float32, ys.device)
    _check(lib, lib.forge_moe_combine(_need(ys, "ys", torch.float32, 2), _need(dest, "dest", torch.int32), _need(wts, "wts", torch.float32),
                                      _need(y, "y"), T, W, top, _stream()), "moe_combine")
    return y


def token_shift(h, state, prev_off, batch, mu):
    """[n, T, W] in h's type: h + (previous token's h - h) * mu[m]; the previous token of a request's first token of the
    step is the row kept in its state (fp32 [slots, row], at ``prev_off``)."""
    lib = library("mixers")
    T, W = h.shape
    n = mu.shape[0]
    out = new_tensor((n, T, W), h.dtype, h.device)
    _check(lib, lib.forge_token_shift(_need(h, "h", ndim=2), _need(state, "state", torch.float32, 2), state.shape[1], int(prev_off),
                                      _need(batch.tok_req, "tok_req", torch.int32), _need(batch.q_start, "q_start", torch.int32),
                                      _need(batch.slots, "slots", torch.int32), _need(mu, "mu", torch.float32, 2), _need(out, "out", h.dtype),
                                      dtype_code(h.dtype), T, W, n, _stream()), "token_shift")
    return out


HEAD_GATES = {"sigmoid": 0, "silu": 1, "none": 2}


def head_finish(o, weight, gate, N, K, eps, gate_activation, out_dtype, scale=1.0, out=None):
    """o fp32 [T, N*K]: every head divided by its root mean square (eps inside the root), times ``weight`` fp32 [N*K] (or [K],
    shared by the heads), times the activation of ``gate`` ((fp32 matrix, first column); None with "none"), times ``scale``;
    [T, N*K] in ``out_dtype``; ``out`` = (matrix, first column): written there instead (the matrix is returned)."""
    lib = library("mixers")
    T = o.shape[0]
    out, out_ptr, out_ld = _out_slice(out, N * K, T, out_dtype, o.device)
    gp, gl = _cols(*gate) if gate is not None else (None, 0)
    if weight.numel() not in (K, N * K):
        raise KernelError(f"head_finish: {weight.numel()} weights for {N} heads of {K}")
    share = 1 if (weight.numel() == K and N > 1) else 0
    _check(lib, lib.forge_head_finish(_need(o, "o", torch.float32, 2), _need(weight, "weight", torch.float32), gp, gl,
                                      out_ptr, dtype_code(out_dtype), T, N, K, float(eps),
                                      HEAD_GATES[gate_activation], float(scale), share, out_ld, _stream()), "head_finish")
    return out


def tanh_rows(x, out_dtype, n=None):
    """tanh of the first ``n`` columns of (fp32 matrix, first column) ``x``, [T, n] in ``out_dtype``."""
    lib = library("mixers")
    t, off = x
    n = t.shape[1] - off if n is None else n
    out = new_tensor((t.shape[0], n), out_dtype, t.device)
    xp, xl = _cols(t, off)
    _check(lib, lib.forge_tanh_rows(xp, xl, _need(out, "out", out_dtype), dtype_code(out_dtype), t.shape[0], n, _stream()), "tanh_rows")
    return out


# ------------------------------------------------------------------------------- tensor-core kernels

def gemm_sm100_supports(n, k):
    """The tcgen05 kernel reads rows by TMA: a row of K bfloat16 must be a multiple of 16 bytes."""
    return _TENSOR_CORE_GEMM and k % 8 == 0 and n >= 1


def attention_mma_supports(head_dim, group, page_size):
    """Head sizes in steps of 16 up to 256, any group size, any page size; other shapes use the fp32 kernel."""
    return _TENSOR_CORE_ATTENTION and head_dim % 16 == 0 and 16 <= head_dim <= 256


BQ_ROWS = 64        # query rows (token, head-of-group pairs) per attention tile
KV_TILE = 64        # keys per inner iteration
_NUM_SMS = {}


def _sm_count(device):
    key = str(device)
    if key not in _NUM_SMS:
        _NUM_SMS[key] = torch.cuda.get_device_properties(device).multi_processor_count
    return _NUM_SMS[key]


TC_ROWS = 128       # query rows per tile of the tcgen05 attention kernel
TC_MIN_ROWS = 64    # requests with at least this many rows in the step go to it


def attention_plan(batch, group, device, only_below=None):
    """How the step's query rows are cut into tiles for the tensor-core attention kernel, and into how
    many slices each tile's keys are cut.  Computed once per step and group size (all layers share it).
    A request with q_len tokens has q_len * group rows; tiles never span requests.  ``only_below``: plan
    only the requests with fewer rows than that (the others are served by the tcgen05 kernel)."""
    key = ("mma", group, only_below)
    plan = batch.attention_plan.get(key)
    if plan is not None:
        return plan
    tile_req, tile_row0, max_rows = [], [], 1
    qs = batch.host_q_start
    for s in range(batch.num_requests):
        rows = (qs[s + 1] - qs[s]) * group
        if only_below is not None and rows >= only_below:
            continue
        for r0 in range(0, rows, BQ_ROWS):
            tile_req.append(s)
            tile_row0.append(r0)
            max_rows = max(max_rows, min(BQ_ROWS, rows - r0))
    max_ctx = getattr(batch, "max_context", None)
    if max_ctx is None:
        max_ctx = max(c + qs[s + 1] - qs[s] for s, c in enumerate(batch.host_context_before))
    plan = {"tile_req": new_ints(tile_req, device), "tile_row0": new_ints(tile_row0, device),
            "num_tiles": len(tile_req), "max_rows": max_rows, "max_kv_tiles": -(-max_ctx // KV_TILE), "scratch": {}}
    batch.attention_plan[key] = plan
    return plan


TC_MIN_SHARE = 8     # key tiles (of 64 keys) that a share of a tile's keys holds at least
TC_MAX_SHARES = 32


def attention_plan_tc(batch, group, device, n_kv_heads=1, head_dim=64, window=0, shares=None):
    """Tiles of (128 // group) whole tokens, that is up to 128 rows, for the requests that bring at least TC_MIN_ROWS
    rows, heaviest (most keys) first.  When the step has at most half as many (tile, kv head) pairs as the GPU has
    places for the kernel's CTAs, the keys of the long tiles are cut into shares, in proportion to their length, so that the places
    are taken (a short portion on a long context); ``shares`` forces a number for every tile (tests)."""
    key = ("tc", group, n_kv_heads, head_dim, window, shares)
    plan = batch.attention_plan.get(key)
    if plan is not None:
        return plan
    tiles, qs = [], batch.host_q_start
    tile_rows = (TC_ROWS // group) * group
    for s in range(batch.num_requests):
        rows = (qs[s + 1] - qs[s]) * group
        if rows < TC_MIN_ROWS:
            continue
        ctx = batch.host_context_before[s]
        for r0 in range(0, rows, tile_rows):
            kv_hi = ctx + (min(rows, r0 + tile_rows) - 1) // group + 1
            kv_lo = max(0, ctx + r0 // group - window + 1) if window else 0
            tiles.append((-(-kv_hi // KV_TILE) - kv_lo // KV_TILE, s, r0))
    places = _sm_count(device) * (2 if head_dim <= 64 else 1)
    total = max(1, sum(t[0] for t in tiles) * n_kv_heads)

    def worth(n, scale):        # n / (total / places): how many places this tile's keys are worth
        return max(1, min(n // TC_MIN_SHARE, n * places * scale // (10 * total), TC_MAX_SHARES))
    if shares is not None:
        cut = [max(1, min(int(shares), t[0], TC_MAX_SHARES)) for t in tiles]
    else:
        cut = [1] * len(tiles)
        # (with more than half of the places taken already there is nothing to gain that pays for the second kernel)
        for scale in range(10, 4, -1) if 2 * len(tiles) * n_kv_heads <= places else ():
            # short tiles count as one whole place each: shrink the others' worth until all fit
            trial = [worth(t[0], scale) for t in tiles]
            if sum(trial) * n_kv_heads <= places:
                cut = trial
                break
    entries, merges, slots = [], [], 0
    for (n, s, r0), z in zip(tiles, cut):
        if z > 1:
            merges.append((s, r0, slots, z))
        entries += [(n / z, s, r0, i, z, slots if z > 1 else 0) for i in range(z)]
        slots += z if z > 1 else 0
    entries.sort(key=lambda e: (-e[0], e[1], e[2], e[3]))
    plan = {"tile_req": new_ints([e[1] for e in entries], device), "tile_row0": new_ints([e[2] for e in entries], device),
            "num_tiles": len(entries), "num_merge": len(merges), "tile_cut": None, "merge_list": None, "part_o": None, "part_ml": None}
    if merges:
        plan["tile_cut"] = new_ints([v for e in entries for v in e[3:6]], device)
        plan["merge_list"] = new_ints([v for m in merges for v in m], device)
        plan["part_o"] = new_tensor((slots * n_kv_heads * TC_ROWS * head_dim,), torch.float32, device, whole_step=True)
        plan["part_ml"] = new_tensor((slots * n_kv_heads * TC_ROWS * 2,), torch.float32, device, whole_step=True)
    batch.attention_plan[key] = plan
    return plan


def attention_sm100_supports(head_dim, group, page_size):
    """Head sizes 64 and 128, any group of up to 128 query heads per kv head, pages of 8 to 64 tokens."""
    return _TENSOR_CORE_ATTENTION and head_dim in (64, 128) and 1 <= group <= TC_ROWS and page_size in (8, 16, 32, 64)


def paged_attention_sm100(q, kv_cache, group_batch, batch, n_heads, n_kv_heads, head_dim, page_size, window=0,
                          scale=None, out=None, shares=None):
    """tcgen05/TMEM attention for the requests of the step that bring many rows (prompt portions).  Writes
    only those requests' rows of ``out``.  Returns (out, number of tiles run: a tile whose keys are cut into
    shares counts once per share)."""
    lib = library("attention_sm100", {"FORGE_ATT_HD": head_dim})
    plan = attention_plan_tc(batch, n_heads // n_kv_heads, q.device, n_kv_heads, head_dim, int(window or 0), shares)
    if out is None:
        out = new_tensor(q.shape, q.dtype, q.device)
    if plan["num_tiles"] == 0:
        return out, 0
    scale = head_dim ** -0.5 if scale is None else scale
    _check(lib, lib.forge_paged_attention_sm100(
        _need(q, "q", torch.bfloat16, 2), _need(kv_cache, "kv_cache", torch.bfloat16), _need(out, "out", torch.bfloat16),
        _need(group_batch.block_table, "block_table", torch.int32, 2), _need(plan["tile_req"], "tile_req"),
        _need(plan["tile_row0"], "tile_row0"), _opt(plan["tile_cut"], "tile_cut"), _opt(plan["part_o"], "part_o"),
        _opt(plan["part_ml"], "part_ml"), _opt(plan["merge_list"], "merge_list"), plan["num_merge"],
        _need(batch.q_start, "q_start", torch.int32),
        _need(batch.context_before, "context_before", torch.int32), _need(_gemm_status(q.device), "status", torch.int32),
        plan["num_tiles"], q.shape[0], kv_cache.shape[0], n_heads, n_kv_heads, head_dim, page_size,
        group_batch.block_table.shape[1], int(window or 0), float(scale), _stream()), "paged_attention_sm100")
    if plan["num_merge"]:
        count_launches(1)      # the kernel that adds the shares up
    return out, plan["num_tiles"]


def paged_attention_mma(q, kv_cache, group_batch, batch, n_heads, n_kv_heads, head_dim, page_size, window=0,
                        scale=None, out=None, num_splits=None, only_below=None):
    """bf16 tensor-core attention over the paged cache for every token of the step (or, with ``only_below``,
    for the requests that bring fewer rows than that)."""
    lib = library("attention_mma", {"FORGE_ATT_HD": head_dim})
    plan = attention_plan(batch, n_heads // n_kv_heads, q.device, only_below)
    if out is None:
        out = new_tensor(q.shape, q.dtype, q.device)
    if plan["num_tiles"] == 0:
        return out
    if num_splits is None:
        # decode-like steps (every tile is one warp with small buffers, ten of which fit an SM): slice the
        # keys until about eight CTAs per SM exist, so that enough loads are in flight to hide their latency
        base = plan["num_tiles"] * n_kv_heads
        num_splits = 1
        if plan["max_rows"] <= 16:
            num_splits = max(1, min(plan["max_kv_tiles"], -(-8 * _sm_count(q.device) // base)))
    part_o = part_ml = None
    if num_splits > 1:
        pr = 16 if plan["max_rows"] <= 16 else BQ_ROWS
        sk = (num_splits, head_dim, pr)
        if sk not in plan["scratch"]:
            n = plan["num_tiles"] * n_kv_heads * num_splits * pr
            plan["scratch"][sk] = (new_tensor((n * head_dim,), torch.float32, q.device, whole_step=True),
                                   new_tensor((n * 2,), torch.float32, q.device, whole_step=True))
        part_o, part_ml = plan["scratch"][sk]
    if out is None:
        out = new_tensor(q.shape, q.dtype, q.device)
    scale = head_dim ** -0.5 if scale is None else scale
    _check(lib, lib.forge_paged_attention_mma(
        _need(q, "q", torch.bfloat16, 2), _need(kv_cache, "kv_cache", torch.bfloat16), _need(out, "out", torch.bfloat16),
        _opt(part_o, "part_o"), _opt(part_ml, "part_ml"), _need(group_batch.block_table, "block_table", torch.int32, 2),
        _need(plan["tile_req"], "tile_req"), _need(plan["tile_row0"], "tile_row0"),
        _need(batch.q_start, "q_start", torch.int32), _need(batch.context_before, "context_before", torch.int32),
        plan["num_tiles"], plan["max_rows"], n_heads, n_kv_heads, head_dim, page_size, group_batch.block_table.shape[1],
        int(window or 0), int(num_splits), float(scale), _stream()), "paged_attention_mma")
    if num_splits > 1:
        count_launches(1)      # the merge kernel
    return out


def decode_attention_fused_supports(dtype, head_dim, group, num_requests, n_kv_heads, max_context, page_size=None):
    """One launch for rotary encoding + cache write + attention of a decode step: bfloat16, head sizes in steps
    of 16 up to 128, at most 16 query heads per kv head.  With few requests and long contexts the
    sliced kernel (keys spread over many CTAs) is the better choice."""
    if not (_TENSOR_CORE_ATTENTION and dtype == torch.bfloat16 and head_dim % 16 == 0 and 16 <= head_dim <= 128 and group <= 16):
        return False
    # with few requests the kernel spreads a request's keys over a cluster of up to 4 CTAs; measured (22 layers, 4 kv
    # heads, 8 requests x 6,000 cached tokens) 1.10 ms per step against 1.26 for the sliced kernel + merge.  Beyond
    # 16k cached tokens with a handful of CTAs the sliced kernel's many CTAs are the better choice again.
    if page_size is not None and decode_attention_stream_supports(head_dim, page_size, group):
        # the kernel that streams the cache spreads a request over up to 8 CTAs and keeps a ring of tiles in flight:
        # the sliced kernel only wins with at most 16 (request, kv head) pairs beyond 16k tokens (measured: 4 pairs x
        # 32k tokens 25 against 18 us, 16 pairs 46 against 38; 32 pairs 50 against 63)
        return not (num_requests * n_kv_heads <= 16 and max_context > 16384)
    return not (num_requests * n_kv_heads < 64 and max_context > 16384)


# The decode attention that streams the cache through a TMA ring pays where a request has many tiles of 64 keys, or
# where there are more (request, kv head) pairs than SMs; with few pairs and fewer than this many cached tokens (an
# upper bound known on the host) the kernel with one buffer pair per warp, which asks for a short context's tiles
# before its dependency wait, is the faster one inside a step (measured, 8 requests x 540 tokens: 0.826 against
# 0.846 ms per step; 64 requests: 48.6 against 49.9 thousand tokens a second the other way round).
STREAM_ATTENTION_MIN_CONTEXT = int(os.environ.get("FORGE_STREAM_ATTENTION_MIN_CONTEXT", "2048"))
STREAM_ATTENTION_MANY_PAIRS = 148


def decode_attention_stream_supports(head_dim, page_size, group):
    return _TENSOR_CORE_ATTENTION and head_dim in (64, 128) and page_size in (16, 32, 64) and group <= 16


def decode_attention_stream(qkv, kv_cache, block_table, positions, slot_mapping, n_heads, n_kv_heads, head_dim, page_size,
                            theta, rotary=True, window=0, scale=None, out=None, max_context=0, ksplit=0):
    """The same step as ``decode_attention_fused`` with the keys and values brought by TMA into a ring of tiles
    (csrc/attention_decode_stream.cu): head sizes 64 and 128, pages of 16, 32 or 64 tokens.  ``ksplit``: CTAs that
    share a request's keys (0: chosen from ``max_context``)."""
    lib = library("attention_mma", {"FORGE_ATT_HD": head_dim})
    S = qkv.shape[0]
    if out is None:
        out = new_tensor((S, n_heads * head_dim), torch.bfloat16, qkv.device)
    scale = head_dim ** -0.5 if scale is None else scale
    _check(lib, lib.forge_decode_attention_stream(
        _need(qkv, "qkv", torch.float32, 2), _need(kv_cache, "kv_cache", torch.bfloat16), _need(out, "out", torch.bfloat16),
        _need(block_table, "block_table", torch.int32, 2), _need(positions, "positions", torch.int32),
        _need(slot_mapping, "slot_mapping", torch.int32), _need(_gemm_status(qkv.device), "status", torch.int32), S, n_heads,
        n_kv_heads, head_dim, page_size, block_table.shape[1], kv_cache.shape[0], int(window or 0), 1 if rotary else 0,
        float(theta), float(scale), int(max_context or 0), int(ksplit), _stream()), "decode_attention_stream")
    return out


def decode_attention_fused(qkv, kv_cache, block_table, positions, slot_mapping, n_heads, n_kv_heads, head_dim, page_size,
                           theta, rotary=True, window=0, scale=None, out=None, max_context=0):
    """qkv fp32 [S,(NH+2NKV)*HD], one new token per request: rotates q and k (``rotary``), writes k and v into
    the cache at ``slot_mapping`` and returns the attention output bf16 [S, NH*HD], all in one kernel.
    ``max_context``: an upper bound of any request's cached tokens + 1, if known: with few requests and many keys
    the kernel then spreads a request's keys over 2 or 4 CTAs."""
    pairs = qkv.shape[0] * n_kv_heads
    # (beyond some 768 pairs with short contexts the per-warp kernel is ahead again: 256 requests x 1,024 tokens 60 against 67 us)
    if ((max_context or 0) >= STREAM_ATTENTION_MIN_CONTEXT or STREAM_ATTENTION_MANY_PAIRS < pairs <= 768) and \
            decode_attention_stream_supports(head_dim, page_size, n_heads // n_kv_heads):
        return decode_attention_stream(qkv, kv_cache, block_table, positions, slot_mapping, n_heads, n_kv_heads, head_dim,
                                       page_size, theta, rotary=rotary, window=window, scale=scale, out=out, max_context=max_context)
    lib = library("attention_mma", {"FORGE_ATT_HD": head_dim})
    S = qkv.shape[0]
    if out is None:
        out = new_tensor((S, n_heads * head_dim), torch.bfloat16, qkv.device)
    scale = head_dim ** -0.5 if scale is None else scale
    _check(lib, lib.forge_decode_attention_fused(
        _need(qkv, "qkv", torch.float32, 2), _need(kv_cache, "kv_cache", torch.bfloat16), _need(out, "out", torch.bfloat16),
        _need(block_table, "block_table", torch.int32, 2), _need(positions, "positions", torch.int32),
        _need(slot_mapping, "slot_mapping", torch.int32), S, n_heads, n_kv_heads, head_dim, page_size, block_table.shape[1],
        int(window or 0), 1 if rotary else 0, float(theta), float(scale), int(max_context or 0), _stream()),
        "decode_attention_fused")
    return out


class DecodeLayers:
    """All layers of a decode step as one persistent kernel (csrc/decode_layers.cu).

    Made once per model from the layers' device tensors; ``run`` then takes the residual stream of a step of
    at most ``max_tokens`` single tokens through every layer, in place.  The object owns the kernel's scratch
    (fp32 results of the projections, attention output, barrier words), so calls must not overlap on the GPU.
    """
    MAX_TOKENS = 16

    @staticmethod
    def supports(hidden, intermediate, n_heads, n_kv_heads, head_dim, tokens=1):
        if not (_TENSOR_CORE_GEMM and _TENSOR_CORE_ATTENTION) or head_dim % 16 != 0 or not 16 <= head_dim <= 128:
            return False
        lib = library("decode_layers", {"FORGE_ATT_HD": head_dim})
        return bool(lib.forge_decode_layers_supports(int(tokens), hidden, intermediate, n_heads, n_kv_heads, head_dim))

    def __init__(self, layers, hidden, intermediate, n_heads, n_kv_heads, head_dim, page_size, theta, rotary, eps,
                 window=0, scale=None, max_tokens=MAX_TOKENS):
        """layers: per layer a dict of device tensors: wqkv bf16 [(NH+2NKV)*HD, H], wo [H, NH*HD], wgu [2I, H] (gate and
        up rows interleaved), wdown [H, I], norm1 / norm2 fp32 [H], bias fp32 [(NH+2NKV)*HD] or None, kv (the layer's
        cache [pages, 2, NKV, page_size, HD] bf16)."""
        self.lib = lib = library("decode_layers", {"FORGE_ATT_HD": head_dim})
        self.dims = (hidden, intermediate, n_heads, n_kv_heads, head_dim)
        self.page_size, self.theta, self.rotary, self.eps, self.window = int(page_size), float(theta), bool(rotary), float(eps), int(window or 0)
        self.scale = head_dim ** -0.5 if scale is None else float(scale)
        self.max_tokens = min(int(max_tokens), self.MAX_TOKENS)
        # weights are asked into L2 two or three products ahead of their use (0: off); a layer's matrices must fit
        # the L2 beside what is in use for that to pay
        self.prefetch_units = int(os.environ.get("FORGE_DECODE_PREFETCH_UNITS", "1"))
        dev = layers[0]["wqkv"].device
        self.num_layers = len(layers)
        nbytes = lib.forge_decode_layers_desc_bytes()
        self.descs = torch.zeros(self.num_layers * nbytes, dtype=torch.uint8, device=dev)
        self._keep = layers                                    # the maps hold raw pointers into these tensors
        with torch.cuda.device(dev):
            for i, t in enumerate(layers):
                rc = lib.forge_decode_layers_describe(
                    self.descs.data_ptr(), i, _need(t["wqkv"], "wqkv", torch.bfloat16, 2), _need(t["wo"], "wo", torch.bfloat16, 2),
                    _need(t["wgu"], "wgu", torch.bfloat16, 2), _need(t["wdown"], "wdown", torch.bfloat16, 2),
                    _need(t["norm1"], "norm1", torch.float32), _need(t["norm2"], "norm2", torch.float32),
                    _opt(t.get("bias"), "bias", torch.float32), _need(t["kv"], "kv", torch.bfloat16), hidden, intermediate,
                    n_heads, n_kv_heads, head_dim)
                if rc != 0:
                    raise KernelError(f"decode_layers: {lib.forge_last_error().decode(errors='replace')} (code {rc})")
        B, qkv = self.max_tokens, (n_heads + 2 * n_kv_heads) * head_dim
        self.qkv_acc = torch.zeros(B * qkv, dtype=torch.float32, device=dev)
        self.gu_acc = torch.zeros(B * 2 * intermediate, dtype=torch.float32, device=dev)
        self.ssq = torch.zeros(128, dtype=torch.float32, device=dev)
        self.rope_tab = torch.zeros(B * head_dim, dtype=torch.float32, device=dev)
        self.part_o = torch.zeros(B * n_kv_heads * 4 * 16 * head_dim, dtype=torch.float32, device=dev)
        self.part_ml = torch.zeros(B * n_kv_heads * 4 * 16 * 2, dtype=torch.float32, device=dev)
        self.barrier = torch.zeros(4, dtype=torch.int32, device=dev)

    def run(self, residual, block_table, positions, slot_mapping, timeline=None):
        """residual fp32 [B, H], updated in place; block_table int32 [B, max_pages]; positions, slot_mapping int32 [B].
        ``timeline``: an int64 tensor [SMs, 1 + 5 * layers, 2] that receives when each CTA reached and left each of
        the kernel's barriers (ns of the device's clock), for a look at where a step's time goes."""
        H, I, NH, NKV, HD = self.dims
        B = residual.shape[0]
        if B > self.max_tokens or residual.shape[1] != H:
            raise KernelError(f"decode_layers: residual {tuple(residual.shape)} does not fit ({self.max_tokens} tokens of {H})")
        lib = self.lib
        _check(lib, lib.forge_decode_layers(
            self.descs.data_ptr(), self.num_layers, _need(residual, "residual", torch.float32, 2), self.qkv_acc.data_ptr(),
            self.gu_acc.data_ptr(), self.ssq.data_ptr(), self.rope_tab.data_ptr(), self.part_o.data_ptr(),
            self.part_ml.data_ptr(), _need(block_table, "block_table", torch.int32, 2),
            _need(positions, "positions", torch.int32), _need(slot_mapping, "slot_mapping", torch.int32), self.barrier.data_ptr(),
            _need(_gemm_status(residual.device), "status", torch.int32), B, H, I, NH, NKV, HD, self.page_size,
            block_table.shape[1], self.window, 1 if self.rotary else 0, self.theta, self.scale, self.eps, self.prefetch_units,
            _opt(timeline, "timeline", torch.int64), _stream()), "decode_layers")
        return residual

    def reset_after_error(self):
        """After a wait ran out the barrier words are left as they were; clear them before the next step."""
        self.barrier.zero_()


def paged_attention(q, kv_cache, group_batch, batch, n_heads, n_kv_heads, head_dim, page_size, window=None,
                    scale=None):
    """Attention of every token of the step over its request's pages; picks the kernel by dtype and shape."""
    if q.dtype == torch.bfloat16 and attention_mma_supports(head_dim, n_heads // n_kv_heads, page_size):
        group = n_heads // n_kv_heads
        if attention_sm100_supports(head_dim, group, page_size) and not getattr(batch, "decode_only", False):
            out, n = paged_attention_sm100(q, kv_cache, group_batch, batch, n_heads, n_kv_heads, head_dim, page_size,
                                           window=window or 0, scale=scale)
            if n:       # the requests with few rows (decode tokens, short portions) use the mma.sync kernel
                return paged_attention_mma(q, kv_cache, group_batch, batch, n_heads, n_kv_heads, head_dim, page_size,
                                           window=window or 0, scale=scale, out=out, only_below=TC_MIN_ROWS)
        return paged_attention_mma(q, kv_cache, group_batch, batch, n_heads, n_kv_heads, head_dim, page_size,
                                   window=window or 0, scale=scale)
    return paged_attention_simt(q, kv_cache, group_batch.block_table, batch.tok_req, batch.positions, n_heads,
                                n_kv_heads, head_dim, page_size, window=window or 0, scale=scale)


EPILOGUES = {"none": 0, "accumulate": 1, "cast": 2, "swiglu": 3, "geglu": 5}
GELU_GATE_VARIANT = {"FORGE_GATE_GELU": 1}
# libraries whose bfloat16 store applies an activation first: the exact gelu, xIELU with the call's two numbers
CAST_VARIANTS = {"gelu": {"FORGE_CAST_ACT": 1}, "xielu": {"FORGE_CAST_ACT": 2}}


def gemm_sm100(x, w, bias=None, accumulate_into=None, epilogue="none", tile_n=0, status=None, out=None, live=None, numbers=None):
    """bf16 x [M,K] . w [N,K]^T on the tcgen05 tensor cores, fp32 accumulation.
    epilogue "none": fp32 [M,N] (added into ``accumulate_into`` when given); "cast": bf16 [M,N];
    "swiglu": bf16 [M,N/2] = silu(y[:,2j]) * y[:,2j+1]; "geglu": the same with the tanh form of gelu; "gelu": bf16 [M,N] =
    y/2 (1 + erf(y / sqrt 2)); "xielu": bf16 [M,N], see ``act_rows`` (``numbers`` its two numbers).
    ``live``: an int32 device word (a one-element tensor) written by an earlier kernel; where it holds 0 the product is skipped on the
    device, nothing read and nothing written."""
    # the gelu gate lives in a variant of the library of its own, so that the silu epilogues stay as short as they were
    lib = library("gemm_sm100", GELU_GATE_VARIANT if epilogue == "geglu" else CAST_VARIANTS.get(epilogue))
    (M, K), (N, K2) = x.shape, w.shape
    if K != K2:
        raise KernelError(f"gemm_sm100: x {tuple(x.shape)} does not match w {tuple(w.shape)}")
    if epilogue == "none":
        if accumulate_into is not None:
            out, code = accumulate_into, EPILOGUES["accumulate"]
        else:
            out = new_tensor((M, N), torch.float32, x.device) if out is None else out
            code = EPILOGUES["none"]
        want_shape, want_dtype = (M, N), torch.float32
    elif epilogue in ("cast", "gelu", "xielu"):
        out = new_tensor((M, N), torch.bfloat16, x.device) if out is None else out
        code, want_shape, want_dtype = EPILOGUES["cast"], (M, N), torch.bfloat16
    elif epilogue in ("swiglu", "geglu"):
        out = new_tensor((M, N // 2), torch.bfloat16, x.device) if out is None else out
        code, want_shape, want_dtype = EPILOGUES[epilogue], (M, N // 2), torch.bfloat16
    else:
        raise KernelError(f"gemm_sm100: unknown epilogue {epilogue!r}")
    if tuple(out.shape) != want_shape:
        raise KernelError(f"gemm_sm100: output has shape {tuple(out.shape)}, expected {want_shape}")
    if status is None:
        status = _gemm_status(x.device)
    _gemm_workspace(lib, x.device)
    _check(lib, lib.forge_gemm_sm100(_need(x, "x", torch.bfloat16, 2), _need(w, "w", torch.bfloat16, 2),
                                     _opt(bias, "bias", torch.float32), _need(out, "out", want_dtype),
                                     _need(status, "status", torch.int32), M, N, K, code, int(tile_n), _opt(live, "live", torch.int32),
                                     *_act_numbers(epilogue, numbers), _stream()),
           "gemm_sm100")
    return out


def gemm_sm100_qkv_rope_supports(rows, head_dim, k):
    """The projection whose epilogue rotates and stores: prompt portions (more than 128 rows), head sizes 64 and 128."""
    return _TENSOR_CORE_GEMM and rows > 128 and head_dim in (64, 128) and k % 8 == 0


def gemm_sm100_qkv_rope(x, w, bias, rope_table, slot_mapping, kv_cache, n_heads, n_kv_heads, head_dim, page_size, q_out=None,
                        tile=0):
    """bf16 x [M,K] . w [(NH+2NKV)*HD, K]^T (+ bias) on the tensor cores; the epilogue rotates q and k by ``rope_table``
    (fp32 [HD/2, M, 2] of (cos, sin), ``rope_table(..., by_pair=True)``; None: no rotation), returns q bf16 [M, NH*HD] and writes k and v into ``kv_cache``
    at ``slot_mapping`` (None: not written).  The fp32 product never reaches global memory.  ``tile``: 0 lets the
    library choose; 128 / 256 one CTA per tile of that width, 1128 / 1192 / 1256 a pair of CTAs on 256 rows of it."""
    lib = library("gemm_sm100")
    (M, K), (N, K2) = x.shape, w.shape
    if K != K2 or N != (n_heads + 2 * n_kv_heads) * head_dim:
        raise KernelError(f"gemm_sm100_qkv_rope: x {tuple(x.shape)}, w {tuple(w.shape)} do not fit {n_heads}+2*{n_kv_heads} heads of {head_dim}")
    if q_out is None:
        q_out = new_tensor((M, n_heads * head_dim), torch.bfloat16, x.device)
    if kv_cache is None:
        slot_mapping = None
    _check(lib, lib.forge_gemm_sm100_qkv_rope(
        _need(x, "x", torch.bfloat16, 2), _need(w, "w", torch.bfloat16, 2), _opt(bias, "bias", torch.float32),
        _need(q_out, "q_out", torch.bfloat16, 2), _opt(kv_cache, "kv_cache", torch.bfloat16), _opt(rope_table, "rope_table", torch.float32),
        _opt(slot_mapping, "slot_mapping", torch.int32), _need(_gemm_status(x.device), "status", torch.int32), M, K, n_heads,
        n_kv_heads, head_dim, page_size, tile, _stream()), "gemm_sm100_qkv_rope")
    return q_out


_status_words = {}
_workspaces = {}
GEMM_WORKSPACE_BYTES = 48 * 1024 * 1024


def _gemm_workspace(lib, device):
    """One zeroed buffer per device for the few-rows GEMM's partial sums and flags, given to the library once."""
    key = (id(lib), str(device))           # a variant of the library is a library of its own, with a workspace of its own
    if key not in _workspaces:
        ws = torch.zeros(GEMM_WORKSPACE_BYTES, dtype=torch.uint8, device=device)
        with torch.cuda.device(device), once_per_step():
            rc = lib.forge_gemm_sm100_set_workspace(ws.data_ptr(), GEMM_WORKSPACE_BYTES)
        if rc != 0:
            raise KernelError(f"gemm_sm100: {lib.forge_last_error().decode(errors='replace')}")
        _workspaces[key] = ws
    return _workspaces[key]



def _gemm_status(device):
    """One int32 per device on which tensor-core kernels raise bit 1 when a bounded wait runs out."""
    dev = torch.device(device)
    if dev.type == "cuda" and dev.index is None:
        dev = torch.device("cuda", torch.cuda.current_device())
    key = str(dev)
    if key not in _status_words:
        _status_words[key] = torch.zeros(1, dtype=torch.int32, device=dev)
    return _status_words[key]


def check_kernel_status(device="cuda:0"):
    """Synchronises and raises if a tensor-core kernel gave up on a wait since the last check."""
    dev = torch.device(device)
    if dev.type == "cuda" and dev.index is None:
        dev = torch.device("cuda", torch.cuda.current_device())
    w = _status_words.get(str(dev))
    if w is not None:
        v = int(w.item())
        if v:
            w.zero_()
            raise KernelError(f"a tensor-core kernel reported status {v:#x} (a bounded wait ran out)")


_TENSOR_CORE_GEMM = True
_TENSOR_CORE_ATTENTION = True
