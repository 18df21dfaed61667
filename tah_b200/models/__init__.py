"""Model families: the Qwen3 backbone of TaH (0.6B / 1.7B / 4B shapes and the tiny test model), Gunuvik, Ditilix,
Niralix and Pidenex."""
from tah_b200.models.ditilix import DitilixConfig, DitilixForCausalLM, ditilix_preset
from tah_b200.models.gunuvik import GunuvikConfig, GunuvikForCausalLM, gunuvik_preset
from tah_b200.models.niralix import NiralixConfig, NiralixForCausalLM, niralix_preset
from tah_b200.models.pidenex import PidenexConfig, PidenexForCausalLM, pidenex_preset
from tah_b200.models.qwen3 import (PRESETS, LoRASpec, Qwen3Config, Qwen3ForCausalLM, attach_lora,
                                   export_hf_state_dict, from_hf_model, import_hf_state_dict, preset)
from tah_b200.models.registry import load_model, make_engine, register_family

__all__ = ["PRESETS", "LoRASpec", "Qwen3Config", "Qwen3ForCausalLM", "attach_lora",
           "export_hf_state_dict", "from_hf_model", "import_hf_state_dict", "preset",
           "DitilixConfig", "DitilixForCausalLM", "ditilix_preset",
           "GunuvikConfig", "GunuvikForCausalLM", "gunuvik_preset", "NiralixConfig", "NiralixForCausalLM", "niralix_preset",
           "PidenexConfig", "PidenexForCausalLM", "pidenex_preset", "load_model", "make_engine", "register_family"]
