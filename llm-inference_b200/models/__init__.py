"""Architectures this engine knows; importing the package registers them."""

from . import dugalix, gunedra, lerorax, qwen2, tosipel, tunadra, zetizen  # noqa: F401
