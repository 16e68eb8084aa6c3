"""Architectures: each module registers one name of config.json `architectures` (or `architecture`)."""
from . import kasarax, llama, selinex, sogutar, vapelix, zudatar, zulopel  # noqa: F401
