"""Architectures: importing this package registers them."""
from . import bapavik, gebilorn, lilunex, llama, rogisun, vivepel  # noqa: F401
from .decoder import DecoderModel  # noqa: F401
