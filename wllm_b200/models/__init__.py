"""Built-in architectures: importing this package registers them."""
from . import fusanex, gemma, gudarax, pesanex, taritar, vifirax, zafilix  # noqa: F401
