"""Architectures: each module registers itself in ``hfee_b200.config.registry``."""
from . import bamipel, bumisun, dobelix, fokalorn, llama, muvetar, pupinex  # noqa: F401
