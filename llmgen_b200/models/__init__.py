"""Built-in architectures; importing this package registers them."""
from . import derupel, fonuvik, kugisun, nasozen, qwen3, sarulix, zuvasun  # noqa: F401
