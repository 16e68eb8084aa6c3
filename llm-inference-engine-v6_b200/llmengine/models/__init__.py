"""Architectures: each module registers one name of config.json `architectures` (or `architecture`)."""
from . import llama, selinex, sogutar, vapelix, zudatar, zulopel  # noqa: F401
