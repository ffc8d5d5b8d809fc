"""Architectures: importing this package registers them."""
from . import bapavik, filezen, gebilorn, lilunex, llama, rogisun, vivepel  # noqa: F401
from .decoder import DecoderModel  # noqa: F401
