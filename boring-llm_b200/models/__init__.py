"""Architectures of this engine. Importing the package registers them."""
from . import qwen2, fezopel, kavotar, miforax, dapuzen, gipinex
from .loading import build_model, load_model, load_random_model, write_random_model

__all__ = ["qwen2", "fezopel", "kavotar", "miforax", "dapuzen", "gipinex", "build_model", "load_model", "load_random_model", "write_random_model"]
