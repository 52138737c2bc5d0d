"""Architectures: importing this package registers each one under its config.json name."""
from . import bogupel, fovirax, fuvipel, goridra, llama, mavinex, pusunex  # noqa: F401
