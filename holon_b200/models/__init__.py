"""Built-in architectures; importing this package registers them."""
from . import bukuvik, gegunex, kasovik, qwen3, rulorax, tilarax, vobosun  # noqa: F401
