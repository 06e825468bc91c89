"""Architectures: each module registers itself in ``hfee_b200.config.registry``."""
from . import bamipel, dobelix, fokalorn, llama, muvetar, pupinex  # noqa: F401
