"""Built-in architectures.  Importing this package registers them."""
from . import famalorn, kerepel, llama, neruzen, sogidra, zezilix, zuvepel  # noqa: F401
