"""Vavadra checkpoints: tensors by name -> :class:`HybridWeights` of the hybrid executor's stream layout.

Names: ``embed`` (also the head), ``final.norm``, ``loop.step`` and per layer ``l<i>.`` with ``norm1 / norm2`` (in front of
the sub-layers), ``mix.*`` and ``mlp.{router, correction, e<n>.*, shared.*}``. Layers that run several times appear once; the
run order is the configuration's (``extra["layer_runs"]``). Projections that read the same input are stacked into one
matrix, the experts' into one tensor per layer, and the logits' factor is part of the final norm's weight."""
from __future__ import annotations

import json
import math
from pathlib import Path

import torch

from ..config import ModelConfig
from ..ops.reference import rope_inv_freq
from .attention_mixer import AttentionMixerWeights, stack_rows
from .gated_delta import GatedDeltaWeights
from .hybrid import HybridBlock, HybridWeights
from .latent_mixer import LatentMixerWeights
from .moe import MoeBlockWeights

GLU_SLOPE = 1.702                 # slope of the gate's sigmoid in the experts


def second_map_factor(get, p: str, diff: float) -> float:
    """``exp(lq1 . lk1) - exp(lq2 . lk2) + diff`` of a differential attention layer."""
    dot = lambda a, b: float((get(p + a).double() * get(p + b).double()).sum())        # noqa: E731
    return math.exp(dot("lq1", "lk1")) - math.exp(dot("lq2", "lk2")) + diff


def build_vavadra_weights(get, cfg: ModelConfig, dtype=torch.bfloat16, device="cpu") -> HybridWeights:
    """``get(name)`` returns a stored tensor."""
    mat = lambda n: get(n).to(device=device, dtype=dtype).contiguous()                 # noqa: E731
    vec = lambda n: get(n).to(device=device, dtype=torch.float32).contiguous()         # noqa: E731
    layers = []
    for i, spec in enumerate(cfg.extra["layer_specs"]):
        p, m = f"l{i}.", spec["mixer"]
        x, norm = p + "mix.", vec(p + "norm1")
        if spec["type"] == "attention":
            blk = HybridBlock("attention_mixer", norm, attn=AttentionMixerWeights(
                w_in=stack_rows([mat(x + n) for n in "qkv"]), b_in=stack_rows([mat(x + n + ".b")[:, None] for n in "qkv"])[:, 0].contiguous(),
                out_proj=mat(x + "o"), heads=m["heads"], kv_heads=m["kv_heads"], dim=2 * m["dim"], vdim=m["vdim"], scale=m["scale"],
                chunk=m["mask"]["size"], diff=(second_map_factor(get, x, m["diff"]), 1.0 - m["diff"])))
        elif spec["type"] == "latent_attention":
            w_uk = mat(x + "uk")
            inv, mscale = rope_inv_freq(m["rot"]["dims"], m["rot"]["base"], None)
            blk = HybridBlock("latent_mixer", norm, attn=LatentMixerWeights(
                w_in=stack_rows([mat(x + "q"), mat(x + "dkv")]), q_norm=None, c_norm=vec(x + "dkv.norm"), w_uq=None, w_uk=w_uk,
                w_uk_t=w_uk.view(m["heads"], m["dim"], m["kv_rank"]).transpose(1, 2).contiguous(), w_uv=mat(x + "uv"), out_proj=mat(x + "o"),
                heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"], q_rank=0, kv_rank=m["kv_rank"], scale=m["scale"],
                inv_freq=inv.to(device), mscale=mscale, adjacent=True, window=m["mask"]["size"], sinks=vec(x + "sink")))
        else:
            blk = HybridBlock("gated_delta", norm, mamba=GatedDeltaWeights(
                w_in=stack_rows([mat(x + n) for n in "qkvg"]), w_rates=torch.cat([mat(x + "b"), mat(x + "a")], 0).contiguous(),
                conv_w=torch.cat([vec(x + n + ".conv") for n in "qkv"], 0).contiguous(), A_log=vec(x + "A_log"), dt_bias=vec(x + "dt_bias"),
                norm_w=vec(x + "norm"), out_proj=mat(x + "o"), heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"]))
        blocks = [blk]
        if spec["mlp"]:
            r, e, sh, y = spec["mlp"]["router"], spec["mlp"]["expert"], spec["mlp"]["shared"], p + "mlp."
            pair = lambda n: torch.cat([mat(f"{y}{n}.gate"), mat(f"{y}{n}.up")], 0)      # noqa: E731
            blocks.append(HybridBlock("moe_stream", vec(p + "norm2"), moe=MoeBlockWeights(
                router=mat(y + "router"), correction=vec(y + "correction"), gate_up=torch.stack([pair(f"e{n}") for n in range(r["experts"])]),
                down=torch.stack([mat(f"{y}e{n}.down") for n in range(r["experts"])]), top=r["top"], scale=r["scale"], limit=e["limit"],
                alpha=GLU_SLOPE, shared_gate_up=pair("shared") if sh else None, shared_down=mat(y + "shared.down") if sh else None,
                shared_limit=sh["limit"] if sh else 0.0)))
        layers.append(blocks)
    embed, runs = mat("embed"), cfg.extra["layer_runs"]
    loop, entries = cfg.extra.get("loop"), {}
    if loop and loop["stop"] > loop["start"]:
        step = vec("loop.step")
        entries = {loop["start"] + t * (loop["stop"] - loop["start"]): (t > 0, step[t].contiguous()) for t in range(loop["times"])}
    return HybridWeights(embed=embed, blocks=[b for bs in layers for b in bs], final_norm=vec("final.norm") * cfg.extra["logit_scale"],
                         lm_head=embed, runs=[layers[i] for i in runs], run_entries=entries)


def load_vavadra_weights(path, cfg: ModelConfig, dtype=torch.bfloat16, device="cpu") -> HybridWeights:
    from ..loading.checkpoint import TensorSource

    src = TensorSource(path)

    def get(name):
        if not src.has(name):
            raise KeyError(f"{path}: missing tensor {name}")
        return src.get(name)

    return build_vavadra_weights(get, cfg, dtype, device)


def vavadra_shapes(cfg: ModelConfig) -> dict[str, tuple]:
    """Tensor names and shapes of a checkpoint of this configuration."""
    H, V, loop = cfg.hidden_size, cfg.vocab_size, cfg.extra.get("loop")
    out = {"embed": (V, H), "final.norm": (H,)}
    if loop:
        out["loop.step"] = (loop["times"], H)
    for i, spec in enumerate(cfg.extra["layer_specs"]):
        p, m = f"l{i}.", spec["mixer"]
        x, h, d, v = p + "mix.", m["heads"], m["dim"], m["vdim"]
        out[p + "norm1"] = (H,)
        if spec["type"] == "attention":
            rows = dict(q=2 * h * d, k=2 * m["kv_heads"] * d, v=m["kv_heads"] * v)
            out.update({x + n: (r, H) for n, r in rows.items()})
            out.update({x + n + ".b": (r,) for n, r in rows.items()})
            out.update({x + n: (d,) for n in ("lq1", "lk1", "lq2", "lk2")})
        elif spec["type"] == "latent_attention":
            c, r = m["kv_rank"], m["rot_dim"]
            out.update({x + "q": (h * (d + r), H), x + "dkv": (c + r, H), x + "dkv.norm": (c,), x + "uk": (h * d, c), x + "uv": (h * v, c),
                        x + "sink": (h,)})
        else:
            for n, r in dict(q=m["kv_heads"] * d, k=m["kv_heads"] * d, v=h * v).items():
                out.update({x + n: (r, H), f"{x}{n}.conv": (r, m["conv"])})
            out.update({x + "a": (h, H), x + "b": (h, H), x + "A_log": (h,), x + "dt_bias": (h,), x + "norm": (v,), x + "g": (h * v, H)})
        out[x + "o"] = (H, h * v)
        if spec["mlp"]:
            r, e, sh, y = spec["mlp"]["router"], spec["mlp"]["expert"], spec["mlp"]["shared"], p + "mlp."
            n = r["experts"] + r["identity"]
            out.update({p + "norm2": (H,), y + "router": (n, H), y + "correction": (n,)})
            for name, ff in [(f"e{j}", e["ff"]) for j in range(r["experts"])] + ([("shared", sh["ff"])] if sh else []):
                out.update({f"{y}{name}.gate": (ff, H), f"{y}{name}.up": (ff, H), f"{y}{name}.down": (H, ff)})
    return out


def random_vavadra_tensors(cfg: ModelConfig, seed: int = 0, dtype=torch.bfloat16, device="cpu") -> dict:
    """Random tensors under the checkpoint's names: projections of unit gain, norm weights around one, decays of a few to
    some hundred tokens."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in vavadra_shapes(cfg).items():
        t, leaf = torch.randn(*shape, generator=g, device=device), name.rsplit(".", 1)[-1]
        if len(shape) == 2:
            t = t if name == "loop.step" else t * shape[1] ** -0.5
        elif leaf.startswith("norm"):
            t = 1 + 0.2 * t
        elif leaf == "dt_bias":
            t = t - 3
        elif leaf in ("lq1", "lk1", "lq2", "lk2"):
            t = 0.5 * t * shape[0] ** -0.25
        elif leaf in ("b", "correction"):
            t = 0.1 * t
        out[name] = t.to(dtype)
    return out


def random_vavadra_weights(cfg: ModelConfig, seed: int = 0, dtype=torch.bfloat16, device="cpu") -> HybridWeights:
    t = random_vavadra_tensors(cfg, seed, torch.bfloat16 if dtype == torch.bfloat16 else torch.float32, device)
    return build_vavadra_weights(t.__getitem__, cfg, dtype, device)


def vavadra_config_dict(cfg: ModelConfig) -> dict:
    return dict(architecture="Vavadra", vocab=cfg.vocab_size, width=cfg.hidden_size, layers=cfg.extra["layer_specs"],
                loop=cfg.extra.get("loop"), embedding=dict(scale=cfg.embed_scale), norm=dict(eps=cfg.rms_norm_eps),
                logit_scale=cfg.extra["logit_scale"])


def save_vavadra_checkpoint(path, cfg: ModelConfig, tensors: dict) -> None:
    from safetensors.torch import save_file

    path = Path(path)
    path.mkdir(parents=True, exist_ok=True)
    save_file({k: v.detach().cpu().contiguous() for k, v in tensors.items()}, str(path / "model.safetensors"))
    (path / "config.json").write_text(json.dumps(vavadra_config_dict(cfg)))
