"""Built-in architectures; importing this package registers them."""

from . import kapitar, lakatar, llama, pufevik, venezen, vizotar, vogolix  # noqa: F401
