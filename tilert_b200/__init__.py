"""tilert_b200 -- B200-native batch-1 decoding behind the TileRT operator interface.

Mirrors the reference package entry points (tilert/__init__.py:51-80, tilert/tilert_init.py):
``load_backend(model_type)`` loads the in-tree CUDA library of a model type once per process and
``tilert_init()`` creates its per-device context.  There is no CPU fallback: without the
compiled library, or without a CUDA device, these raise.
"""

from __future__ import annotations

import ctypes
import logging
from dataclasses import dataclass
from pathlib import Path

__version__ = "0.1.0"
logger = logging.getLogger(__name__)

@dataclass(frozen=True)
class Backend:
    """A native library: its file, the header that declares it and the prefix of its runtime calls."""

    library: str
    header: str
    prefix: str
    exported_globally: bool = False  # another library links to its symbols


_BACKENDS = {
    "deepseek_v3_2": Backend("libtilert_b200.so", "tilert_b200.h", "tilert_b200", exported_globally=True),
    "ralasun": Backend("libtilert_gqa.so", "tilert_gqa.h", "tilert_gqa"),
}
_DEFAULT = "deepseek_v3_2"
_libs: dict[str, ctypes.CDLL] = {}
_contexts: dict[tuple[str, int], int] = {}


class TilertError(RuntimeError):
    """An error reported by the native library (mirrors the RuntimeError of a failed torch op)."""


def library_path(model_type: str = _DEFAULT) -> Path:
    """The in-tree library; ``TILERT_B200_LIB`` names another build of the default one's sources (tuning)."""
    import os

    override = os.environ.get("TILERT_B200_LIB") if model_type == _DEFAULT else None
    return Path(override) if override else Path(__file__).resolve().parent / _BACKENDS[model_type].library


def load_backend(model_type: str = _DEFAULT) -> ctypes.CDLL:
    """Load the native library for ``model_type`` (tilert/__init__.py:51-80)."""
    if model_type not in _BACKENDS:
        raise ValueError(f"Unknown model_type {model_type!r}. Supported: {sorted(_BACKENDS)}")
    if model_type in _libs:
        return _libs[model_type]
    path = library_path(model_type)
    if not path.exists():
        raise RuntimeError(
            f"Backend library not found: {path}. Build it with `python -m tilert_b200.build` "
            "(needs nvcc; compiles for sm_100a).")
    from ._cabi import bind, header_path

    be = _BACKENDS[model_type]
    _libs[model_type] = bind(path, header_path(be.header), be.exported_globally)
    logger.info("Loaded tilert_b200 backend %s", path.name)
    return _libs[model_type]


def lib(model_type: str = _DEFAULT) -> ctypes.CDLL:
    return load_backend(model_type)


def _call(model_type: str, name: str):
    return getattr(lib(model_type), f"{_BACKENDS[model_type].prefix}_{name}")


def check(rc: int, model_type: str = _DEFAULT) -> None:
    """Raise ``TilertError`` for a negative return code of a C-ABI call."""
    if rc != 0:
        msg = _call(model_type, "last_error")()
        raise TilertError(f"tilert_b200 call failed ({rc}): {msg.decode() if msg else ''}")


def tilert_init(device: int | None = None, model_type: str = _DEFAULT) -> int:
    """Create (once) the context of ``device`` and return its handle (tilert/tilert_init.py:11-13)."""
    import torch

    if not torch.cuda.is_available():
        raise RuntimeError("tilert_b200 needs a CUDA device (sm_100a); there is no CPU path")
    dev = torch.cuda.current_device() if device is None else device
    if (model_type, dev) not in _contexts:
        ctx = ctypes.c_void_p()
        check(_call(model_type, "default_context")(dev, ctypes.byref(ctx)), model_type)
        _contexts[(model_type, dev)] = ctx.value
    return _contexts[(model_type, dev)]


def device_status(device: int | None = None, model_type: str = _DEFAULT) -> int:
    """Synchronise and return the device status word (0 = every kernel ran to completion)."""
    st = ctypes.c_int(0)
    check(_call(model_type, "status")(tilert_init(device, model_type), ctypes.byref(st)), model_type)
    return st.value


def launch_count(model_type: str = _DEFAULT) -> int:
    """Kernels the library has launched (or recorded into graphs) in this process."""
    return int(_call(model_type, "launch_count")())


def set_wait_budget(cycles: int, device: int | None = None, model_type: str = _DEFAULT) -> None:
    """Upper bound (SM clock cycles) of every bounded wait in the library's kernels; ``cycles <= 0`` restores
    the default of about half a second."""
    check(_call(model_type, "set_wait_budget")(ctypes.c_void_p(tilert_init(device, model_type)), int(cycles)), model_type)


__all__ = ["set_wait_budget", "load_backend", "tilert_init", "device_status", "launch_count", "lib", "check", "TilertError", "__version__"]
