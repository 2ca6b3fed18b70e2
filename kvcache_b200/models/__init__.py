"""Architectures known to the registry; importing this package registers them."""
from . import kakipel, kaposun, karorax, kunulorn, libulorn, lipelix, qwen2  # noqa: F401
from .kakipel import build_kakipel
from .kaposun import build_kaposun
from .karorax import build_karorax
from .kunulorn import build_kunulorn
from .libulorn import build_libulorn
from .lipelix import build_lipelix
from .qwen2 import build_qwen2

__all__ = ["build_kakipel", "build_kaposun", "build_karorax", "build_kunulorn", "build_libulorn", "build_lipelix", "build_qwen2"]
