"""Loads the kernel library (building it at first use) and declares its C entry points."""

from __future__ import annotations

import ctypes
import threading
from ctypes import c_float, c_int, c_longlong, c_void_p

_lock = threading.Lock()
_lib: ctypes.CDLL | None = None

P, I, F, LL = c_void_p, c_int, c_float, c_longlong

# name -> argument types (the stream is the last c_void_p of each)
_SIGNATURES: dict[str, list] = {
    "cw_embed": [P, P, P, I, I, I, I, F, P, P],
    "cw_add_rmsnorm": [P, P, P, P, P, I, I, I, F, I, I, P, P, P, P],
    "cw_silu_mul": [P, P, I, I, I, P],
    "cw_add_to_residual": [P, P, I, I, I, P],
    "cw_add_parts_rmsnorm": [P, P, I, I, P, P, I, I, F, I, I, P, P, P],
    "cw_gemm_ref": [P, P, P, P, I, I, I, I, I, I, I, P],
    "cw_gemm_ref_swiglu": [P, P, P, P, I, I, I, I, P],
    "cw_rope_store": [P, P, P, P, P, P, I, I, I, I, I, I, I, I, P, P],
    "cw_copy_pages": [P, P, I, I, I, LL, P, P],
    "cw_attention_ref": [P, I, P, P, P, P, P, P, I, I, I, I, I, I, I, F, I, I, P, P],
    "cw_argmax": [P, P, I, I, LL, P],
    "cw_sample": [P, P, P, P, P, P, I, I, LL, P],
    "cw_argmax_state": [P, P, I, I, LL, P, P, I, P],
    "cw_sample_state": [P, P, P, P, P, P, I, I, LL, P, P, I, P],
    "cw_sample_rows": [P, P, P, P, P, P, I, I, LL, P, P, I, P, P],
    "cw_sample_workspace_words": [I],
    "cw_step_from_state": [P, P, P, P, I, I, I, I, I, I, P, P, P, P, P, P, P, P, P, P, P, P, P, P],
    # layers with a state of fixed size (csrc/recurrence.cu)
    "cw_shift_mix": [P, P, P, LL, LL, P, P, P, P, I, I, I, I, P],
    "cw_causal_conv": [P, I, P, P, P, LL, LL, P, P, P, P, I, I, I, P],
    "cw_carry_rows": [P, I, P, LL, LL, P, P, P, I, I, I, I, P],
    "cw_recurrence_scan": [I, P, I, P, I, P, I, P, I, P, P, P, P, LL, LL, P, P, P, I, I, I, I, I, P, I, F, I, P],
    "cw_sigmoid_power_decay": [P, I, I, I, F, P],
    "cw_activation_cols": [P, I, I, I, I, I, P],
    "cw_recurrence_coefficients": [I, P, I, P, P, P, I, I, P],
    "cw_gated_group_norm": [P, P, I, P, P, I, I, I, F, I, I, P],
    "cw_activation": [P, LL, I, I, P],
    "cw_rotate_heads": [P, I, P, P, I, I, F, I, I, I, P],
    # attention over a window of rows [key | value] (csrc/window_attention.cu); absolute positions and the sum of two normed
    # contributions (csrc/embed_norm.cu)
    "cw_store_rows": [P, I, I, I, P, P, I, LL, I, P, P],
    "cw_window_attention": [P, I, P, P, I, I, I, P, P, I, I, I, I, I, I, F, P, P, P, I, I, P, P, I, P, P, I, I, P,
                            F, P, F, I, P, I, I, P, P, I, I, I, I, I, P],
    "cw_pool_rows": [P, P, I, I, I, P, P, P, P, LL, I, I, I, I, P, P],
    "cw_pair_embed_add": [P, P, P, P, P, P, P, LL, P, I, LL, LL, I, I, I, I, I, P, P],
    "cw_axpy_rmsnorm": [P, P, P, F, F, P, P, P, F, I, I, I, P],
    "cw_depth_average": [P, P, P, F, F, P, LL, I, P, P, P, P, F, I, I, I, P],
    "cw_bounded_forget": [P, I, P, P, P, I, I, P],
    "cw_rotate_store": [P, I, P, P, P, P, I, I, F, P, P, F, I, I, I, I, I, I, P, P, LL, I, P, P],
    "cw_window_attention_set_mma": [I],
    "cw_scale_add_sinusoid": [P, P, P, F, I, I, P],
    "cw_pair_rmsnorm_add": [P, P, P, P, P, F, F, I, I, P],
    "cw_sum_rmsnorm_add": [P, P, P, F, F, P, F, I, I, P],
    "cw_softcap": [P, LL, F, F, P],
    # products in groups and the mixture of experts (csrc/grouped_gemm.cu)
    "cw_grouped_gemm": [P, I, I, P, P, LL, P, I, I, P, P, I, P, P, I, I, I, I, I, I, F, I, P],
    "cw_grouped_gemm_set_mma": [I],
    "cw_latent_attention_set_mma": [I],
    "cw_moe_choose": [P, P, P, P, P, I, I, I, I, I, I, P, F, I, I, P],
    "cw_moe_group": [P, P, P, P, I, I, P],
    "cw_moe_combine": [P, P, P, P, P, I, I, I, I, I, I, P],
    # the delta rule, the gates and the read-out of a matrix memory (csrc/recurrence_gated.cu)
    "cw_unit_heads": [P, I, I, I, I, F, I, F, F, P],
    "cw_delta_coefficients": [P, I, P, P, P, I, I, I, I, P],
    "cw_delta_prepare": [P, I, P, I, P, LL, LL, P, P, P, I, I, I, I, F, F, P, I, P, I, P, P, I, P, P, P],
    "cw_delta_scan": [P, I, P, I, P, I, P, I, I, P, I, P, LL, LL, P, P, P, I, I, I, I, I, P, I, P, I, I, I, LL, I, P],
    "cw_gate_scan": [P, I, P, I, P, P, F, P, LL, LL, P, P, P, I, I, I, P, P],
    "cw_memory_norm": [P, P, I, P, I, P, P, I, I, I, F, I, P],
    # attention over a cached latent (csrc/latent_attention.cu)
    "cw_latent_prepare": [P, I, P, I, I, P, P, P, P, P, I, F, P, P, I, I, I, I, I, I, F, I, I, P, P],
    "cw_latent_attention": [P, P, P, P, P, P, P, I, P, I, I, I, I, I, I, I, F, I, I, P, I, P, P],
    "cw_latent_attention_on_tensor_cores": [I, I],
}
_OPTIONAL: dict[str, list] = {}


class KernelLibraryError(RuntimeError):
    pass


def register_optional(name: str, argtypes: list) -> None:
    _OPTIONAL[name] = argtypes


def library() -> ctypes.CDLL:
    """The loaded library.  Raises ``KernelLibraryError`` when it cannot be built or loaded:
    there is no fallback path."""
    global _lib
    if _lib is not None:
        return _lib
    with _lock:
        if _lib is not None:
            return _lib
        from ..csrc.build import ensure_built

        try:
            path = ensure_built()
            lib = ctypes.CDLL(str(path))
        except Exception as exc:  # noqa: BLE001
            raise KernelLibraryError(
                f"the clockwork_b200 CUDA kernels are unavailable ({exc}); "
                "they are required: there is no CPU or library fallback"
            ) from exc
        for name, argtypes in {**_SIGNATURES, **_OPTIONAL}.items():
            try:
                fn = getattr(lib, name)
            except AttributeError:
                if name in _OPTIONAL:
                    continue
                raise KernelLibraryError(f"{path} does not export {name}") from None
            fn.argtypes = argtypes
            fn.restype = c_int
        _lib = lib
        return lib


ERROR_NAMES = {-1: "refused size", -2: "unknown dtype code", -3: "unsupported combination", -4: "set-up failed",
               -5: "needs more scratch than the built-in maximum"}


_launches = 0
_pdl_on = True


def set_pdl(on: bool) -> None:
    """Whether kernels are launched so that each may begin while its predecessor drains (programmatic
    dependent launch; the default) or strictly one after the other."""
    global _pdl_on
    library().cw_set_pdl(1 if on else 0)
    _pdl_on = bool(on)


class serial_launch:
    """Launches inside this block start only after everything before them on the stream has finished."""

    def __enter__(self):
        self.was = _pdl_on
        if self.was:
            set_pdl(False)

    def __exit__(self, *exc):
        if self.was:
            set_pdl(True)



def launch_count() -> int:
    """Kernel launches made through this library so far (each entry point launches one kernel)."""
    return _launches


def check(code: int, what: str) -> None:
    global _launches
    _launches += 1
    if code == 0:
        return
    if code < 0:
        raise ValueError(f"{what}: kernel refused the call ({ERROR_NAMES.get(code, code)})")
    raise RuntimeError(f"{what}: CUDA error {code} at launch")
