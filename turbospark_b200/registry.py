"""Model registry: a folder with config.json and model.safetensors -> a loaded model of the class its config names."""
import json
import os

from . import gimozen, nigenex, plain, ronelorn, tarivik
from .safetensors import SafeTensors

COMPUTE = {"bfloat16": plain.BF16, "float32": plain.F32}
# config.json "architecture" -> build(ctx, config, get_tensor, max_context, compute)
ARCHITECTURES = {m.ARCHITECTURE: m.build for m in (gimozen, nigenex, ronelorn, tarivik)}


def read_config(folder):
    with open(os.path.join(folder, "config.json"), encoding="utf-8") as f:
        return json.load(f)


def load(ctx, folder, max_context, compute="bfloat16"):
    """The model in `folder`, weights on the GPU.  max_context bounds a request's positions."""
    config = read_config(folder)
    name = config.get("architecture")
    if name not in ARCHITECTURES:
        raise ValueError("architecture %r is not one of %s" % (name, sorted(ARCHITECTURES)))
    if compute not in COMPUTE:
        raise ValueError("compute type %r is not one of %s" % (compute, sorted(COMPUTE)))
    tensors = SafeTensors(os.path.join(folder, "model.safetensors"))
    return ARCHITECTURES[name](ctx, config, tensors.get, max_context, COMPUTE[compute])
