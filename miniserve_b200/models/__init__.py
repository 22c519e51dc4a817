"""Architectures this package ships. Importing the package registers them."""
from . import fekulix, kovusun, mugipel, qwen3, rofozen, tunadra, vumedra  # noqa: F401
