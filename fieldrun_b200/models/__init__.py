"""Built-in architectures; importing this package registers them."""
from . import bakasun, bamasun, depelix, duzinex, fotanex, kifunex, minimax_m2  # noqa: F401
