"""Importing this package registers the architectures that ship with the engine."""
from . import bevuvik, kefetar, lufizen, mukenex, qwen3, sigudra, torinex  # noqa: F401
