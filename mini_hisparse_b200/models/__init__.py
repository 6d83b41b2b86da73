from . import dotivik, koronex, qwen2, rizovik, rudutar, tudasun, zetenex  # noqa: F401  (each registers its architecture)
from .decoder import DecoderModel
