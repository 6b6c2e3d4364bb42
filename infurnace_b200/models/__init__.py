"""Architectures known to the engine.  Importing this package registers them; it needs
neither torch nor CUDA."""
from .registry import (  # noqa: F401
    Architecture, register_architecture, get_architecture, known_architectures,
    config_from_dict, read_config, plan_for,
)
from . import qwen3  # noqa: F401  (registers "Qwen3ForCausalLM")
from . import kafunex  # noqa: F401  (registers "Kafunex")
from . import lunelorn  # noqa: F401  (registers "Lunelorn")
from . import filorax  # noqa: F401  (registers "Filorax")
from . import golonex  # noqa: F401  (registers "Golonex")
from . import mubutar  # noqa: F401  (registers "Mubutar")
from . import tigelorn  # noqa: F401  (registers "Tigelorn")
