"""Load HF safetensors checkpoints into the in-framework decoder (tunix/models/safetensors_loader.py:73-541).

Weights keep the HF `[out, in]` layout, so loading is: memory-map each file, map the HF key to the module
path with a per-family regex table, optionally stack per-expert tensors (Qwen3-MoE), cast, and copy straight
into the (possibly sharded) destination parameter. One tensor is resident on the host at a time.
"""
from __future__ import annotations

import glob
import json
import os
import re
from typing import Callable, Optional

import torch

# (HF key regex, our parameter name template). Applied in order; first match wins.
_COMMON = [
    (r"model\.embed_tokens\.weight", "embed_tokens"),
    (r"model\.norm\.weight", "norm.weight"),
    (r"lm_head\.weight", "lm_head"),
    (r"model\.layers\.(\d+)\.self_attn\.(q|k|v|o)_proj\.(weight|bias)", r"layers.\1.self_attn.\2_proj.\3"),
    (r"model\.layers\.(\d+)\.self_attn\.(q|k)_norm\.weight", r"layers.\1.self_attn.\2_norm.weight"),
    (r"model\.layers\.(\d+)\.mlp\.(gate|up|down)_proj\.weight", r"layers.\1.mlp.\2_proj.weight"),
    (r"model\.layers\.(\d+)\.input_layernorm\.weight", r"layers.\1.input_layernorm.weight"),
]
_KEY_MAPS = {
    "default": _COMMON + [
        (r"model\.layers\.(\d+)\.post_attention_layernorm\.weight", r"layers.\1.post_attention_layernorm.weight"),
        (r"model\.layers\.(\d+)\.mlp\.gate\.weight", r"layers.\1.mlp.router.weight"),
        (r"model\.layers\.(\d+)\.mlp\.experts\.(\d+)\.(gate|up|down)_proj\.weight", r"layers.\1.mlp.\3_proj#\2"),
    ],
    # Gemma-2/3 use four norms per layer; HF's `post_attention_layernorm` is the norm applied to the
    # attention OUTPUT, and `pre_feedforward_layernorm` is the MLP input norm.
    "gemma_post_norms": _COMMON + [
        (r"model\.layers\.(\d+)\.post_attention_layernorm\.weight", r"layers.\1.post_attn_norm.weight"),
        (r"model\.layers\.(\d+)\.pre_feedforward_layernorm\.weight", r"layers.\1.post_attention_layernorm.weight"),
        (r"model\.layers\.(\d+)\.post_feedforward_layernorm\.weight", r"layers.\1.post_ffw_norm.weight"),
    ],
    # Gemma-4 keeps the HF norm names; "a|b" = the tensor is split in equal parts along its second-to-last axis
    "gemma4": _COMMON + [
        (r"model\.embed_tokens_per_layer\.weight", "embed_tokens_per_layer"),
        (r"model\.per_layer_(model_projection|projection_norm)\.weight", r"per_layer_\1.weight"),
        (r"model\.layers\.(\d+)\.(post_attention|pre_feedforward|post_feedforward)_layernorm\.weight", r"layers.\1.\2_layernorm.weight"),
        (r"model\.layers\.(\d+)\.(post_feedforward_layernorm_1|post_feedforward_layernorm_2|pre_feedforward_layernorm_2)\.weight",
         r"layers.\1.\2.weight"),
        (r"model\.layers\.(\d+)\.(per_layer_input_gate|per_layer_projection|post_per_layer_input_norm)\.weight", r"layers.\1.\2.weight"),
        (r"model\.layers\.(\d+)\.layer_scalar", r"layers.\1.layer_scalar"),
        (r"model\.layers\.(\d+)\.router\.proj\.weight", r"layers.\1.moe.router.weight"),
        (r"model\.layers\.(\d+)\.router\.scale", r"layers.\1.moe.router_scale"),
        (r"model\.layers\.(\d+)\.router\.per_expert_scale", r"layers.\1.moe.per_expert_scale"),
        (r"model\.layers\.(\d+)\.experts\.gate_up_proj", r"layers.\1.moe.gate_proj|layers.\1.moe.up_proj"),
        (r"model\.layers\.(\d+)\.experts\.down_proj", r"layers.\1.moe.down_proj"),
    ],
    # Layer-stack checkpoints (models/stack.py) number their layers l0, l1, ...
    "roluzen": [
        (r"embed", "embed_tokens"),
        (r"head", "lm_head"),
        (r"final\.norm", "norm.weight"),
        (r"l(\d+)\.norm1", r"layers.\1.input_layernorm.weight"),
        (r"l(\d+)\.norm2", r"layers.\1.post_attention_layernorm.weight"),
        (r"l(\d+)\.hc(1|2)\.(in|out)", r"layers.\1.hc\2.weight_\3"),
        (r"l(\d+)\.hc(1|2)\.mix", r"layers.\1.hc\2.mix"),
        (r"l(\d+)\.mlp\.(gate|up|down)", r"layers.\1.mlp.\2_proj.weight"),
        (r"l(\d+)\.mix\.(left|right)\.out", r"layers.\1.mixer.\2_norm.weight"),
        (r"l(\d+)\.mix\.left\.(q|k)\.norm", r"layers.\1.mixer.left.\2_norm.weight"),
        (r"l(\d+)\.mix\.left\.rel", r"layers.\1.mixer.left.rel"),
        (r"l(\d+)\.mix\.right\.norm", r"layers.\1.mixer.right.norm.weight"),
        (r"l(\d+)\.mix\.right\.(i|f)\.b", r"layers.\1.mixer.right.\2_proj.bias"),
        (r"l(\d+)\.mix\.(left|right)\.(q|k|v|g|o|i|f)", r"layers.\1.mixer.\2.\3_proj.weight"),
        (r"l(\d+)\.mix\.(y|x)\.b", r"layers.\1.mixer.\2_proj.bias"),
        (r"l(\d+)\.mix\.(y|x|o)", r"layers.\1.mixer.\2_proj.weight"),
        (r"l(\d+)\.mix\.(conv|ra|ri)\.b", r"layers.\1.mixer.\2_bias"),
        (r"l(\d+)\.mix\.(conv|ra|ri)", r"layers.\1.mixer.\2_weight"),
        (r"l(\d+)\.mix\.lam", r"layers.\1.mixer.lam"),
    ],
    "tovalix": [
        (r"embed", "embed_tokens"),
        (r"embed\.norm", "embed_norm.weight"),
        (r"side\.embed", "side_embed"),
        (r"head", "lm_head"),
        (r"final\.norm", "norm.weight"),
        (r"l(\d+)\.norm1", r"layers.\1.input_layernorm.weight"),
        (r"l(\d+)\.norm2", r"layers.\1.post_attention_layernorm.weight"),
        (r"l(\d+)\.mlp\.(up|down)", r"layers.\1.mlp.\2_proj.weight"),
        (r"l(\d+)\.mlp\.act", r"layers.\1.mlp.act"),
        (r"l(\d+)\.side\.gate", r"layers.\1.side.gate_proj.weight"),
        (r"l(\d+)\.side\.(proj|norm)", r"layers.\1.side.\2.weight"),
        (r"l(\d+)\.mix\.mu\.(r|k|v|g|w)", r"layers.\1.mixer.mu_\2"),
        (r"l(\d+)\.mix\.(w0|u|lower)", r"layers.\1.mixer.\2"),
        (r"l(\d+)\.mix\.norm", r"layers.\1.mixer.norm.weight"),
        (r"l(\d+)\.mix\.(q|k|v|o|f)\.b", r"layers.\1.mixer.\2_proj.bias"),
        (r"l(\d+)\.mix\.(r|k|v|g|q|f|o|w1|w2)", r"layers.\1.mixer.\2_proj.weight"),
    ],
    "zikezen": [
        (r"embed", "embed_tokens"),
        (r"pos", "pos_embed"),
        (r"side\.embed", "side_embed"),
        (r"head", "lm_head"),
        (r"final\.norm", "norm.weight"),
        (r"l(\d+)\.norm1", r"layers.\1.input_layernorm.weight"),
        (r"l(\d+)\.norm2", r"layers.\1.post_attention_layernorm.weight"),
        (r"l(\d+)\.norm1b", r"layers.\1.post_attn_norm.weight"),
        (r"l(\d+)\.norm2b", r"layers.\1.post_ffw_norm.weight"),
        (r"l(\d+)\.mlp\.(gate|up|down)", r"layers.\1.mlp.\2_proj.weight"),
        (r"l(\d+)\.mlp\.e(\d+)\.(gate|up|down)", r"layers.\1.mlp.\3_proj#\2"),
        (r"l(\d+)\.mlp\.router", r"layers.\1.mlp.router.weight"),
        (r"l(\d+)\.mlp\.correction", r"layers.\1.mlp.correction"),
        (r"l(\d+)\.side\.gate", r"layers.\1.side.gate_proj.weight"),
        (r"l(\d+)\.side\.(proj|norm)", r"layers.\1.side.\2.weight"),
        (r"l(\d+)\.mix\.left\.(q|k)\.norm", r"layers.\1.mixer.left.\2_norm.weight"),
        (r"l(\d+)\.mix\.right\.norm", r"layers.\1.mixer.right.norm.weight"),
        (r"l(\d+)\.mix\.(left|right)\.(q|k|v|a2)\.b", r"layers.\1.mixer.\2.\3_proj.bias"),
        (r"l(\d+)\.mix\.(left|right)\.(q|k|v|g|o|a1|a2)", r"layers.\1.mixer.\2.\3_proj.weight"),
    ],
    "zigipel": [
        (r"embed", "embed_tokens"),
        (r"bigram", "bigram_embed"),
        (r"loop\.in", "loop_in.weight"),
        (r"loop\.step", "loop_step"),
        (r"head", "lm_head"),
        (r"final\.norm", "norm.weight"),
        (r"l(\d+)\.norm1", r"layers.\1.input_layernorm.weight"),
        (r"l(\d+)\.shift", r"layers.\1.shift"),
        (r"l(\d+)\.mlp\.(gate|up|down)\.b", r"layers.\1.mlp.\2_proj.bias"),
        (r"l(\d+)\.mlp\.(gate|up|down)", r"layers.\1.mlp.\2_proj.weight"),
        (r"l(\d+)\.mix\.dkv\.norm", r"layers.\1.mixer.kv_norm.weight"),
        (r"l(\d+)\.mix\.(r1|r2|sink)", r"layers.\1.mixer.\2"),
        (r"l(\d+)\.mix\.(q|k|v|g|o|dkv|uk|uv)", r"layers.\1.mixer.\2_proj.weight"),
    ],
}


def key_map_for(cfg) -> list:
    if cfg.family == "gemma4" or cfg.family in _STACK_INVERSE:
        return _KEY_MAPS[cfg.family]
    return _KEY_MAPS["gemma_post_norms" if cfg.post_norms else "default"]


def map_key(hf_key: str, table: list) -> Optional[str]:
    hf_key = re.sub(r"^language_model\.", "", hf_key)                 # language_model.model.layers... (Gemma 3)
    hf_key = re.sub(r"^model\.language_model\.", "model.", hf_key)    # model.language_model.layers... (Gemma 4)
    for pat, repl in table:
        m = re.fullmatch(pat, hf_key)
        if m:
            return m.expand(repl)
    return None


def inverse_map_key(our_key: str, cfg) -> str:
    """Our parameter name -> HF key (used by the saver)."""
    if cfg.family in _STACK_INVERSE:
        return _inverse_stack_key(our_key, cfg.family)
    if our_key == "embed_tokens":
        return "model.embed_tokens.weight"
    if our_key == "lm_head":
        return "lm_head.weight"
    if our_key == "norm.weight":
        return "model.norm.weight"
    k = "model." + our_key
    if cfg.post_norms:
        k = k.replace(".post_attention_layernorm.", ".pre_feedforward_layernorm.")
        k = k.replace(".post_attn_norm.", ".post_attention_layernorm.")
        k = k.replace(".post_ffw_norm.", ".post_feedforward_layernorm.")
    k = k.replace(".mlp.router.weight", ".mlp.gate.weight")
    return k


# parameter name -> checkpoint name of layer-stack models, the inverse of their tables in _KEY_MAPS
_STACK_ENDS = [
    (r"embed_tokens", "embed"), (r"lm_head", "head"), (r"norm\.weight", "final.norm"),
    (r"layers\.(\d+)\.input_layernorm\.weight", r"l\1.norm1"),
    (r"layers\.(\d+)\.post_attention_layernorm\.weight", r"l\1.norm2"),
]
_STACK_INVERSE = {"roluzen": _STACK_ENDS + [
    (r"layers\.(\d+)\.(hc\d)\.weight_(in|out)", r"l\1.\2.\3"),
    (r"layers\.(\d+)\.(hc\d)\.mix", r"l\1.\2.mix"),
    (r"layers\.(\d+)\.mlp\.(gate|up|down)_proj\.weight", r"l\1.mlp.\2"),
    (r"layers\.(\d+)\.mixer\.(left|right)_norm\.weight", r"l\1.mix.\2.out"),
    (r"layers\.(\d+)\.mixer\.left\.(q|k)_norm\.weight", r"l\1.mix.left.\2.norm"),
    (r"layers\.(\d+)\.mixer\.left\.rel", r"l\1.mix.left.rel"),
    (r"layers\.(\d+)\.mixer\.right\.norm\.weight", r"l\1.mix.right.norm"),
    (r"layers\.(\d+)\.mixer\.right\.(i|f)_proj\.bias", r"l\1.mix.right.\2.b"),
    (r"layers\.(\d+)\.mixer\.(left|right)\.(\w)_proj\.weight", r"l\1.mix.\2.\3"),
    (r"layers\.(\d+)\.mixer\.(y|x)_proj\.bias", r"l\1.mix.\2.b"),
    (r"layers\.(\d+)\.mixer\.(y|x|o)_proj\.weight", r"l\1.mix.\2"),
    (r"layers\.(\d+)\.mixer\.(conv|ra|ri)_bias", r"l\1.mix.\2.b"),
    (r"layers\.(\d+)\.mixer\.(conv|ra|ri)_weight", r"l\1.mix.\2"),
    (r"layers\.(\d+)\.mixer\.lam", r"l\1.mix.lam"),
], "tovalix": _STACK_ENDS + [
    (r"embed_norm\.weight", "embed.norm"), (r"side_embed", "side.embed"),
    (r"layers\.(\d+)\.mlp\.(up|down)_proj\.weight", r"l\1.mlp.\2"),
    (r"layers\.(\d+)\.mlp\.act", r"l\1.mlp.act"),
    (r"layers\.(\d+)\.side\.gate_proj\.weight", r"l\1.side.gate"),
    (r"layers\.(\d+)\.side\.(proj|norm)\.weight", r"l\1.side.\2"),
    (r"layers\.(\d+)\.mixer\.mu_(\w)", r"l\1.mix.mu.\2"),
    (r"layers\.(\d+)\.mixer\.(w0|u|lower)", r"l\1.mix.\2"),
    (r"layers\.(\d+)\.mixer\.norm\.weight", r"l\1.mix.norm"),
    (r"layers\.(\d+)\.mixer\.(\w+)_proj\.bias", r"l\1.mix.\2.b"),
    (r"layers\.(\d+)\.mixer\.(\w+)_proj\.weight", r"l\1.mix.\2"),
], "zikezen": _STACK_ENDS + [
    (r"pos_embed", "pos"), (r"side_embed", "side.embed"),
    (r"layers\.(\d+)\.post_attn_norm\.weight", r"l\1.norm1b"),
    (r"layers\.(\d+)\.post_ffw_norm\.weight", r"l\1.norm2b"),
    (r"layers\.(\d+)\.mlp\.(gate|up|down)_proj\.weight", r"l\1.mlp.\2"),
    (r"layers\.(\d+)\.mlp\.(gate|up|down)_proj#(\d+)", r"l\1.mlp.e\3.\2"),
    (r"layers\.(\d+)\.mlp\.router\.weight", r"l\1.mlp.router"),
    (r"layers\.(\d+)\.mlp\.correction", r"l\1.mlp.correction"),
    (r"layers\.(\d+)\.side\.gate_proj\.weight", r"l\1.side.gate"),
    (r"layers\.(\d+)\.side\.(proj|norm)\.weight", r"l\1.side.\2"),
    (r"layers\.(\d+)\.mixer\.left\.(q|k)_norm\.weight", r"l\1.mix.left.\2.norm"),
    (r"layers\.(\d+)\.mixer\.right\.norm\.weight", r"l\1.mix.right.norm"),
    (r"layers\.(\d+)\.mixer\.(left|right)\.(\w+)_proj\.bias", r"l\1.mix.\2.\3.b"),
    (r"layers\.(\d+)\.mixer\.(left|right)\.(\w+)_proj\.weight", r"l\1.mix.\2.\3"),
], "zigipel": _STACK_ENDS + [
    (r"bigram_embed", "bigram"), (r"loop_in\.weight", "loop.in"), (r"loop_step", "loop.step"),
    (r"layers\.(\d+)\.shift", r"l\1.shift"),
    (r"layers\.(\d+)\.mlp\.(gate|up|down)_proj\.bias", r"l\1.mlp.\2.b"),
    (r"layers\.(\d+)\.mlp\.(gate|up|down)_proj\.weight", r"l\1.mlp.\2"),
    (r"layers\.(\d+)\.mixer\.kv_norm\.weight", r"l\1.mix.dkv.norm"),
    (r"layers\.(\d+)\.mixer\.(r1|r2|sink)", r"l\1.mix.\2"),
    (r"layers\.(\d+)\.mixer\.(\w+)_proj\.weight", r"l\1.mix.\2"),
]}


def _inverse_stack_key(our_key: str, family: str) -> str:
    for pat, repl in _STACK_INVERSE[family]:
        m = re.fullmatch(pat, our_key)
        if m:
            return m.expand(repl)
    raise KeyError(f"no checkpoint name for parameter {our_key!r}")


def tensor_shapes(path: str) -> dict:
    """name -> shape of every tensor in the safetensors files under `path` (headers only, no data is read)."""
    out = {}
    for f in ([path] if os.path.isfile(path) else sorted(glob.glob(os.path.join(path, "*.safetensors")))):
        with open(f, "rb") as fh:
            header = json.loads(fh.read(int.from_bytes(fh.read(8), "little")))
        out.update({k: tuple(v["shape"]) for k, v in header.items() if k != "__metadata__"})
    return out


def load_safetensors_into(model, path: str, dtype: Optional[torch.dtype] = None, strict: bool = True,
                          preprocess_fn: Optional[Callable] = None) -> list:
    """Load every `*.safetensors` under `path` (a file or a directory) into `model`. Returns unused HF keys."""
    from safetensors import safe_open
    files = [path] if os.path.isfile(path) else sorted(glob.glob(os.path.join(path, "*.safetensors")))
    if not files:
        raise FileNotFoundError(f"no safetensors files under {path}")
    table = key_map_for(model.config)
    params = dict(model.named_parameters())
    params.update({n: b for n, b in model.named_buffers() if n.endswith("layer_scalar")})
    seen, unused = set(), []
    with torch.no_grad():
        for f in files:
            with safe_open(f, framework="pt", device="cpu") as sf:
                for key in sf.keys():
                    name = map_key(key, table)
                    if name is None:
                        unused.append(key)
                        continue
                    t = sf.get_tensor(key)
                    if preprocess_fn is not None:
                        t = preprocess_fn(name, t)
                    if "|" in name:
                        names = name.split("|")
                        for nm, part in zip(names, t.chunk(len(names), dim=-2)):
                            params[nm].copy_(part.to(params[nm].device, dtype or params[nm].dtype))
                            seen.add((nm, None))
                        continue
                    expert = None
                    if "#" in name:
                        name, e = name.split("#")
                        expert = int(e)
                    if name not in params:
                        if name == "lm_head" and model.config.weight_tying:
                            continue
                        unused.append(key)
                        continue
                    dst = params[name]
                    dst = dst[expert] if expert is not None else dst
                    if dst.shape != t.shape:
                        raise ValueError(f"shape mismatch for {key} -> {name}: checkpoint {tuple(t.shape)} vs model {tuple(dst.shape)}")
                    dst.copy_(t.to(dst.device, dtype or dst.dtype))
                    seen.add((name, expert))
    if strict:
        missing = []
        for n, p in params.items():
            if "lora_" in n or (n, None) in seen:
                continue
            if p.dim() == 3 and n.endswith(("gate_proj", "up_proj", "down_proj")) and \
                    (model.config.is_moe or model.config.family in _STACK_INVERSE):
                missing += [f"{n}#{e}" for e in range(p.shape[0]) if (n, e) not in seen]
            elif (n, None) not in seen:
                missing.append(n)
        if missing:
            raise KeyError(f"parameters missing from checkpoint: {missing[:8]}{'...' if len(missing) > 8 else ''}")
    return unused


def create_model_from_safe_tensors(path: str, config, device=None, dtype: Optional[torch.dtype] = None):
    """Build the model of `config` and fill it from the checkpoint at `path`."""
    from .transformer import create_model
    if dtype is not None:
        config = config.replace(dtype=dtype)
    model = create_model(config, device=device, init=False)
    load_safetensors_into(model, path)
    return model
