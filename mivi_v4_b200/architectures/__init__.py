"""One file per architecture; importing this package registers them all."""
from . import lfm2, mevulix, puzorax, redisun, ropelix, tevirax, votavik  # noqa: F401
