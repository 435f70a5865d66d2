"""Model folder -> runner: the class is chosen by config.json ("architecture", or the first of "architectures")."""
import json
import os

import torch


def _plain_weights(module, entry):
    def load(path, dtype, device, weight_dtype):
        if weight_dtype not in (None, "bf16", "bfloat16"):
            raise ValueError("this model family runs on its bfloat16 (or float32) weights: no quantized weight_dtype")
        import importlib
        return getattr(importlib.import_module("." + module, __package__), entry)(path, dtype, device)
    load.quantizes = False
    return load


def _hugging_face(module, entry):
    def load(path, dtype, device, weight_dtype):
        if dtype != torch.bfloat16:
            raise ValueError("this model family computes in bfloat16")
        import importlib
        from transformers import AutoModelForCausalLM
        optimize = getattr(importlib.import_module("." + module, __package__), entry)
        model = AutoModelForCausalLM.from_pretrained(path, dtype=torch.bfloat16, local_files_only=True)
        return optimize(model, dtype, device, weight_dtype or "mxfp4")
    return load


# architecture -> (loader, activation types it runs in)
ARCHITECTURES = {
    "Dofivik": (_plain_weights("fused_dofivik_infer", "load_dofivik"), (torch.bfloat16, torch.float32)),
    "Vedizen": (_plain_weights("fused_vedizen_infer", "load_vedizen"), (torch.bfloat16, torch.float32)),
    "LlamaForCausalLM": (_hugging_face("fused_llama_infer", "OptimizeModelForLlama"), (torch.bfloat16,)),
    "Qwen2ForCausalLM": (_hugging_face("fused_llama_infer", "OptimizeModelForQwen2"), (torch.bfloat16,)),
    "OPTForCausalLM": (_hugging_face("fused_opt_infer", "OptimizeModelForOPT"), (torch.bfloat16,)),
    "GPTJForCausalLM": (_hugging_face("fused_gptj_infer", "OptimizeModelForGPTJ"), (torch.bfloat16,)),
}


def architecture_of(path):
    with open(os.path.join(path, "config.json")) as f:
        cfg = json.load(f)
    name = cfg.get("architecture") or (cfg.get("architectures") or [None])[0]
    if name not in ARCHITECTURES:
        raise ValueError(f"{path}: unknown architecture {name!r} (known: {', '.join(sorted(ARCHITECTURES))})")
    return name


def dtypes_of(name):
    return ARCHITECTURES[name][1]


def quantizes(name):
    """Whether the family takes a quantized weight_dtype."""
    return getattr(ARCHITECTURES[name][0], "quantizes", True)


def load_model(path, dtype=torch.bfloat16, device="cuda", weight_dtype=None):
    return ARCHITECTURES[architecture_of(path)][0](path, dtype, device, weight_dtype)
