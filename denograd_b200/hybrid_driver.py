"""The drivers of layer-list checkpoints (hybrid.py): one class per architecture, the same calls as the package's other models."""
from __future__ import annotations

from . import synth
from .device import Device
from .driver import Driver, Llama3Usage
from .hybrid import HybridTransformer


class HybridDriver(Driver):
    """``Name(config).load_weights(path)``, then prefill / generate / chat as with the package's other models.  Defaults as for
    Llama3; greedy decoding is ``temperature=0``."""
    architecture = ""

    def __init__(self, config: dict, dtype: str = "bfloat16", max_context: int = 8192, max_batch: int = 1, device: str | None = None,
                 temperature: float = 0.95, top_k: int = 0, top_p: float = 0.0, alpha_f: float = 0.0, alpha_p: float = 0.0,
                 jit: bool = True, page_size: int = 64, max_rows: int = 2048, tokenizer=None):
        config = dict(config, architecture=self.architecture)
        self.config, self.dtype, self.max_context, self.tokenizer = config, dtype, max_context, tokenizer
        self.temperature, self.top_k, self.top_p, self.alpha_f, self.alpha_p = temperature, top_k, top_p, alpha_f, alpha_p
        self.model = HybridTransformer(config, dtype, max_context, max_batch, jit, Device[device], page_size, max_rows)
        self.usage = Llama3Usage()
        self.start_pos, self.last_seen_toks = 0, []

    def load_state_dict(self, weights: dict) -> "HybridDriver":
        self.model.load_state_dict(weights)
        return self

    def load_weights(self, path: str) -> "HybridDriver":
        """A .safetensors file (or the shards of a *.index.json) in the checkpoint's own names; bf16 values are kept exactly."""
        from .state import load_checkpoint
        return self.load_state_dict(load_checkpoint(path, widen_bf16=True))

    def load_synthetic(self, seed: int = synth.BASE_SEED) -> "HybridDriver":
        synth.fill_hybrid(self.model, seed)
        return self
