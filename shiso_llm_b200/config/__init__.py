"""Typed configurations and the architecture registry."""

from .errors import ConfigError, ConfigMissing, InvalidValue, UnknownArchitecture, UnsupportedShape
from .registry import (
    Architecture,
    architecture_of,
    load_config,
    plan_from_document,
    read_config_document,
    register_architecture,
    registered_architectures,
    unregister_architecture,
)
from . import lfm2  # registers Lfm2ForCausalLM
from . import filulix  # registers Filulix
from . import zetavik  # registers Zetavik
from . import volalorn  # registers Volalorn
from . import povilorn  # registers Povilorn
from . import nodepel  # registers Nodepel
from . import raketar  # registers Raketar
from .filulix import FilulixConfig
from .zetavik import ZetavikConfig
from .volalorn import VolalornConfig
from .povilorn import PovilornConfig
from .nodepel import NodepelConfig
from .raketar import RaketarConfig
from .lfm2 import Lfm2Config, feed_forward_width

__all__ = [
    "Architecture",
    "ConfigError",
    "ConfigMissing",
    "FilulixConfig",
    "InvalidValue",
    "Lfm2Config",
    "NodepelConfig",
    "PovilornConfig",
    "RaketarConfig",
    "UnknownArchitecture",
    "UnsupportedShape",
    "VolalornConfig",
    "ZetavikConfig",
    "architecture_of",
    "feed_forward_width",
    "load_config",
    "plan_from_document",
    "read_config_document",
    "register_architecture",
    "registered_architectures",
    "unregister_architecture",
]
