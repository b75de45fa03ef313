"""Pamasun checkpoints: tensors by name -> :class:`HybridWeights` of the hybrid executor's stream layout.

Names: ``embed``, ``head``, ``final.norm`` and per layer ``l<i>.`` with ``norm1 / norm1b / norm2 / norm2b`` (stored
as the offset from one), ``ls1 / ls2``, ``mix.*`` and ``mlp.{up, down, act}``. Layers that run several times
appear once; the run order is the configuration's (``extra["layer_runs"]``). Projections that read the same
input are stacked into one matrix."""
from __future__ import annotations

import json
from pathlib import Path

import torch

from ..config import ModelConfig
from .attention_mixer import AttentionMixerWeights, stack_rows
from .general_delta import GeneralDeltaWeights
from .hybrid import HybridBlock, HybridWeights


def build_pamasun_weights(get, cfg: ModelConfig, dtype=torch.bfloat16, device="cpu") -> HybridWeights:
    """``get(name)`` returns a stored tensor."""
    mat = lambda n: get(n).to(device=device, dtype=dtype).contiguous()                 # noqa: E731
    vec = lambda n: get(n).to(device=device, dtype=torch.float32).contiguous()         # noqa: E731
    layers = []
    for i, spec in enumerate(cfg.extra["layer_specs"]):
        p, m = f"l{i}.", spec["mixer"]
        x = p + "mix."
        if spec["type"] == "attention":
            attn = AttentionMixerWeights(
                w_in=stack_rows([mat(x + n) for n in "qkvg"]), out_proj=mat(x + "o"), heads=m["heads"], kv_heads=m["kv_heads"],
                dim=m["dim"], vdim=m["vdim"], scale=m["scale"], gated=True, q_norm=vec(x + "q.norm"), k_norm=vec(x + "k.norm"),
                r1=vec(x + "r1"), r2=vec(x + "r2"), sinks=vec(x + "sink"))
            blk = HybridBlock("attention_mixer", vec(p + "norm1"), attn=attn)
        else:
            delta = GeneralDeltaWeights(
                w_in=stack_rows([mat(x + n) for n in ("r", "k", "v", "g", "a", "w1")]), w2=mat(x + "w2"), w0=vec(x + "w0"),
                a_bias=vec(x + "a.b"), norm_w=vec(x + "norm"), out_proj=mat(x + "o"), heads=m["heads"], dim=m["dim"])
            blk = HybridBlock("general_delta", vec(p + "norm1"), mamba=delta)
        blk.post_norm, blk.layer_scale = vec(p + "norm1b"), vec(p + "ls1")
        blocks = [blk]
        if spec["mlp"]:
            blocks.append(HybridBlock("mlp", vec(p + "norm2"), up=mat(p + "mlp.up"), down=mat(p + "mlp.down"), act="polynorm",
                                      act_coef=vec(p + "mlp.act"), post_norm=vec(p + "norm2b"), layer_scale=vec(p + "ls2")))
        layers.append(blocks)
    runs = cfg.extra["layer_runs"]
    return HybridWeights(embed=mat("embed"), blocks=[b for bs in layers for b in bs], final_norm=vec("final.norm"),
                         lm_head=mat("head"), runs=[layers[i] for i in runs])


def load_pamasun_weights(path, cfg: ModelConfig, dtype=torch.bfloat16, device="cpu") -> HybridWeights:
    from ..loading.checkpoint import TensorSource

    src = TensorSource(path)

    def get(name):
        if not src.has(name):
            raise KeyError(f"{path}: missing tensor {name}")
        return src.get(name)

    return build_pamasun_weights(get, cfg, dtype, device)


def pamasun_shapes(cfg: ModelConfig, rank: int | None = None) -> dict[str, tuple]:
    """Tensor names and shapes of a checkpoint of this configuration. ``rank``: width of the low-rank decay
    projection (a checkpoint decides it by its tensors; default: a sixteenth of the mixer, at least 4)."""
    H, V = cfg.hidden_size, cfg.vocab_size
    out = {"embed": (V, H), "head": (V, H), "final.norm": (H,)}
    for i, spec in enumerate(cfg.extra["layer_specs"]):
        p, m = f"l{i}.", spec["mixer"]
        x = p + "mix."
        out.update({p + "norm1": (H,), p + "norm1b": (H,), p + "ls1": (H,)})
        if spec["type"] == "attention":
            h, g, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            out.update({x + "q": (h * dk, H), x + "k": (g * dk, H), x + "v": (g * dv, H), x + "g": (h * dv, H), x + "o": (H, h * dv),
                        x + "q.norm": (dk,), x + "k.norm": (dk,), x + "r1": (h,), x + "r2": (h,), x + "sink": (h,)})
        else:
            hd = m["heads"] * m["dim"]
            r = rank or max(4, hd // 16)
            out.update({x + n: (hd, H) for n in ("r", "k", "v", "g", "a")})
            out.update({x + "a.b": (hd,), x + "w0": (hd,), x + "norm": (hd,), x + "w1": (r, H), x + "w2": (hd, r), x + "o": (H, hd)})
        if spec["mlp"]:
            ff = spec["mlp"]["ff"]
            out.update({p + "norm2": (H,), p + "norm2b": (H,), p + "ls2": (H,), p + "mlp.up": (ff, H), p + "mlp.down": (H, ff),
                        p + "mlp.act": (4,)})
    return out


def random_pamasun_tensors(cfg: ModelConfig, seed: int = 0, dtype=torch.bfloat16, device="cpu", rank: int | None = None) -> dict:
    """Random tensors under the checkpoint's names, scaled so that activations and decays stay in a sane range."""
    g = torch.Generator(device=device).manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g, device=device)                          # noqa: E731
    out = {}
    for name, shape in pamasun_shapes(cfg, rank).items():
        leaf = name.rsplit("mix.", 1)[-1].rsplit("mlp.", 1)[-1].split(".", 1)[-1] if name.startswith("l") else name
        if len(shape) == 2:
            t = r(*shape) * (1.0 if name == "embed" else shape[1] ** -0.5)
        elif leaf in ("norm", "q.norm", "k.norm", "ls1", "ls2") or name.endswith((".q.norm", ".k.norm", "mix.norm")):
            t = 1 + 0.2 * r(*shape)
        elif leaf.startswith("norm") or name == "final.norm":
            t = 0.2 * r(*shape)
        elif leaf in ("r1", "r2"):
            t = 0.1 + torch.rand(*shape, generator=g, device=device)
        elif leaf == "act":
            t = torch.tensor([0.8, 0.4, 0.2, 0.1], device=device) + 0.05 * r(*shape)
        elif leaf == "w0":
            t = -3 + 2 * r(*shape)
        else:
            t = r(*shape)
        out[name] = t.to(dtype)
    return out


def random_pamasun_weights(cfg: ModelConfig, seed: int = 0, dtype=torch.bfloat16, device="cpu", rank: int | None = None):
    t = random_pamasun_tensors(cfg, seed, torch.bfloat16 if dtype == torch.bfloat16 else torch.float32, device, rank)
    return build_pamasun_weights(t.__getitem__, cfg, dtype, device)


def pamasun_config_dict(cfg: ModelConfig) -> dict:
    return dict(architecture="Pamasun", vocab=cfg.vocab_size, width=cfg.hidden_size, layers=cfg.extra["layer_specs"],
                loop=cfg.extra.get("loop"), embedding=dict(scale=cfg.embed_scale), norm=dict(eps=cfg.rms_norm_eps))


def save_pamasun_checkpoint(path, cfg: ModelConfig, tensors: dict) -> None:
    from safetensors.torch import save_file

    path = Path(path)
    path.mkdir(parents=True, exist_ok=True)
    save_file({k: v.detach().cpu().contiguous() for k, v in tensors.items()}, str(path / "model.safetensors"))
    (path / "config.json").write_text(json.dumps(pamasun_config_dict(cfg)))
