"""Model registry: the `architecture` of a config.json -> its configuration class and runlist builder, and the named
shapes of the synthetic benchmark models."""
import os

from . import ripidra, supevik
from .checkpoint import Tensors, read_config
from .runlists import QWEN3_0P6B, QWEN3_4B

# architecture -> (configuration from config.json, builder(config, tensors, dtype, max_tokens, max_rows, max_sel))
ARCHITECTURES = {
    "Ripidra": (ripidra.RipidraConfig.from_json, ripidra.build_runlist),
    "Supevik": (supevik.SupevikConfig.from_json, supevik.build_runlist),
}
# synthetic decoder shapes (seeded weights, runlists.py)
SHAPES = {c.name: c for c in (QWEN3_0P6B, QWEN3_4B)}


class Model:
    """A configuration, its tensors and its runlist builder."""

    def __init__(self, config, tensors):
        arch = config.get("architecture")
        if arch not in ARCHITECTURES:
            raise ValueError("architecture %r; known: %s" % (arch, ", ".join(sorted(ARCHITECTURES))))
        read, self._build = ARCHITECTURES[arch]
        self.architecture, self.config, self.tensors = arch, read(config), tensors

    def runlist(self, dtype="bfloat16", max_tokens=2048, max_rows=2048, max_sel=64):
        return self._build(self.config, self.tensors, dtype, max_tokens, max_rows, max_sel)


def load_model(folder):
    """Model of a folder with config.json and model.safetensors."""
    return Model(read_config(folder), Tensors(os.path.join(folder, "model.safetensors")))
