"""A B200-native inference engine for Qwen2-MoE, built from parts.

Importing the package registers the built-in parts and architectures.  The public
entry points are :class:`cajeta_llm_b200.engine.llm_engine.LlmEngine` (load, submit,
generate), ``python -m cajeta_llm_b200`` (command line) and ``bin/trace_run``.
"""
from . import parts  # noqa: F401  (registers the built-in parts)
from .models import balalorn, dimuvik, govuvik, qwen2_moe, rugezen, saropel, zoporax  # noqa: F401  (register the architectures)

__version__ = "0.1.0"
