"""Govopel checkpoints: tensors by name -> :class:`HybridWeights` of the hybrid executor's stream layout.

Names: ``embed`` (also the head), ``embed.norm``, ``final.norm`` and per layer ``l<i>.`` with ``norm1 / norm2`` (behind the
sub-layers), ``mix.*`` and ``mlp.{gate, up, down}``. Projections that read the same input are stacked into one matrix."""
from __future__ import annotations

import json
import math
from pathlib import Path

import torch

from ..config import ModelConfig
from ..ops.reference import rope_inv_freq
from .attention_mixer import AttentionMixerWeights, stack_rows
from .hybrid import HybridBlock, HybridWeights
from .latent_mixer import LatentMixerWeights

def rotation_table(rot: dict, device) -> tuple[torch.Tensor, float]:
    """(fp32 frequencies of the pairs, factor on cosine and sine) of a mixer's ``rot`` record."""
    sc = rot.get("scaling")
    if sc:
        sc = dict(rope_type="yarn", factor=sc["factor"], original_max_position_embeddings=sc["original"], beta_fast=sc["fast"],
                  beta_slow=sc["slow"], attention_factor=0.1 * math.log(sc["factor"]) + 1.0)
    inv, mscale = rope_inv_freq(rot["dims"], rot["base"], sc)
    return inv.to(device), mscale


def build_govopel_weights(get, cfg: ModelConfig, dtype=torch.bfloat16, device="cpu") -> HybridWeights:
    """``get(name)`` returns a stored tensor."""
    mat = lambda n: get(n).to(device=device, dtype=dtype).contiguous()                 # noqa: E731
    vec = lambda n: get(n).to(device=device, dtype=torch.float32).contiguous()         # noqa: E731
    layers = []
    for i, spec in enumerate(cfg.extra["layer_specs"]):
        p, m = f"l{i}.", spec["mixer"]
        x = p + "mix."
        inv, mscale = rotation_table(m["rot"], device)
        if spec["type"] == "attention":
            attn = AttentionMixerWeights(
                w_in=stack_rows([mat(x + "q"), mat(x + "k")]), out_proj=mat(x + "o"), heads=m["heads"], kv_heads=m["kv_heads"],
                dim=m["dim"], vdim=m["vdim"], scale=m["scale"], softcap=m["softcap"], chunk=m["mask"]["size"] if m["mask"] else 0,
                inv_freq=inv, mscale=mscale, unit=True, values_are_keys=True)
            blk = HybridBlock("attention_mixer", None, attn=attn)
        else:
            w_uk = mat(x + "uk")
            attn = LatentMixerWeights(
                w_in=stack_rows([mat(x + "dq"), mat(x + "dkv")]), q_norm=vec(x + "dq.norm"), c_norm=vec(x + "dkv.norm"), w_uq=mat(x + "uq"),
                w_uk=w_uk, w_uk_t=w_uk.view(m["heads"], m["dim"], m["kv_rank"]).transpose(1, 2).contiguous(), w_uv=mat(x + "uv"),
                out_proj=mat(x + "o"), heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"], q_rank=m["q_rank"],
                kv_rank=m["kv_rank"], scale=m["scale"], inv_freq=inv, mscale=mscale)
            blk = HybridBlock("latent_mixer", None, attn=attn)
        blk.post_norm = vec(p + "norm1")
        blocks = [blk]
        if spec["mlp"]:
            blocks.append(HybridBlock("mlp", None, up=torch.cat([mat(p + "mlp.gate"), mat(p + "mlp.up")], 0).contiguous(),
                                      down=mat(p + "mlp.down"), gated=True, act="clipped_swiglu", act_alpha=1.702, act_limit=spec["mlp"]["limit"],
                                      post_norm=vec(p + "norm2")))
        layers.append(blocks)
    embed = mat("embed")
    return HybridWeights(embed=embed, blocks=[b for bs in layers for b in bs], final_norm=vec("final.norm"), lm_head=embed,
                         runs=[layers[i] for i in cfg.extra["layer_runs"]], embed_norm=vec("embed.norm"))


def load_govopel_weights(path, cfg: ModelConfig, dtype=torch.bfloat16, device="cpu") -> HybridWeights:
    from ..loading.checkpoint import TensorSource

    src = TensorSource(path)

    def get(name):
        if not src.has(name):
            raise KeyError(f"{path}: missing tensor {name}")
        return src.get(name)

    return build_govopel_weights(get, cfg, dtype, device)


def govopel_shapes(cfg: ModelConfig) -> dict[str, tuple]:
    """Tensor names and shapes of a checkpoint of this configuration."""
    H, V = cfg.hidden_size, cfg.vocab_size
    out = {"embed": (V, H), "embed.norm": (H,), "final.norm": (H,)}
    for i, spec in enumerate(cfg.extra["layer_specs"]):
        p, m = f"l{i}.", spec["mixer"]
        x, h = p + "mix.", m["heads"]
        out[p + "norm1"] = (H,)
        if spec["type"] == "attention":
            out.update({x + "q": (h * m["dim"], H), x + "k": (m["kv_heads"] * m["dim"], H), x + "o": (H, h * m["vdim"])})
        else:
            q, c, d, r, v = m["q_rank"], m["kv_rank"], m["dim"], m["rot_dim"], m["vdim"]
            out.update({x + "dq": (q, H), x + "dq.norm": (q,), x + "uq": (h * (d + r), q), x + "dkv": (c + r, H), x + "dkv.norm": (c,),
                        x + "uk": (h * d, c), x + "uv": (h * v, c), x + "o": (H, h * v)})
        if spec["mlp"]:
            ff = spec["mlp"]["ff"]
            out.update({p + "norm2": (H,), p + "mlp.gate": (ff, H), p + "mlp.up": (ff, H), p + "mlp.down": (H, ff)})
    return out


def random_govopel_tensors(cfg: ModelConfig, seed: int = 0, dtype=torch.bfloat16, device="cpu") -> dict:
    """Random tensors under the checkpoint's names: projections of unit gain, norm weights around one."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in govopel_shapes(cfg).items():
        t = torch.randn(*shape, generator=g, device=device)
        out[name] = (t * shape[1] ** -0.5 if len(shape) == 2 else 1 + 0.2 * t).to(dtype)
    return out


def random_govopel_weights(cfg: ModelConfig, seed: int = 0, dtype=torch.bfloat16, device="cpu") -> HybridWeights:
    t = random_govopel_tensors(cfg, seed, torch.bfloat16 if dtype == torch.bfloat16 else torch.float32, device)
    return build_govopel_weights(t.__getitem__, cfg, dtype, device)


def govopel_config_dict(cfg: ModelConfig) -> dict:
    return dict(architecture="Govopel", vocab=cfg.vocab_size, width=cfg.hidden_size, layers=cfg.extra["layer_specs"],
                norm=dict(eps=cfg.rms_norm_eps), logit_softcap=cfg.final_logit_softcap)


def save_govopel_checkpoint(path, cfg: ModelConfig, tensors: dict) -> None:
    from safetensors.torch import save_file

    path = Path(path)
    path.mkdir(parents=True, exist_ok=True)
    save_file({k: v.detach().cpu().contiguous() for k, v in tensors.items()}, str(path / "model.safetensors"))
    (path / "config.json").write_text(json.dumps(govopel_config_dict(cfg)))
