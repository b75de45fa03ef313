"""Fusolix checkpoints: tensors by name -> :class:`HybridWeights` of the hybrid executor's stream layout with several streams.

Names: ``embed``, ``head``, ``final.norm`` (+ ``.b``) and per layer ``l<i>.`` with ``mix.left.* / mix.right.*``, ``mlp.*`` and per
sub-layer q (1: mixer, 2: feed-forward) ``norm<q>`` (+ ``.b``), ``canon<q>`` (the short convolution) and ``hc<q>.{in, out, mix}``. The
attention's output bias, times the attention's factor, is added in fp32 where the streams are mixed."""
from __future__ import annotations

import json
from pathlib import Path

import torch

from ..config import ModelConfig
from ..ops.reference import rope_inv_freq
from ..ops.streams import Sublayer
from .attention_mixer import AttentionMixerWeights
from .hybrid import HybridBlock, HybridWeights
from .moe import MoeBlockWeights
from .parallel_mixer import ParallelMixerWeights, join_columns, stack_parallel
from .retention import RetentionWeights

GLU_SLOPE = 1.702                 # slope of the gate's sigmoid in the dense feed-forward


def build_fusolix_weights(get, cfg: ModelConfig, dtype=torch.bfloat16, device="cpu") -> HybridWeights:
    """``get(name)`` returns a stored tensor."""
    mat = lambda n: get(n).to(device=device, dtype=dtype).contiguous()                 # noqa: E731
    vec = lambda n: get(n).to(device=device, dtype=torch.float32).contiguous()         # noqa: E731
    layers = []
    for i, spec in enumerate(cfg.extra["layer_specs"]):
        p, m = f"l{i}.", spec["mixer"]
        a, r, x, y = m["left"], m["right"], p + "mix.left.", p + "mix.right."

        def around(q, bias=None):
            return Sublayer(w_in=vec(f"{p}hc{q}.in"), w_out=vec(f"{p}hc{q}.out"), mix=vec(f"{p}hc{q}.mix"), norm_w=vec(f"{p}norm{q}"),
                            norm_b=vec(f"{p}norm{q}.b"), taps=vec(f"{p}canon{q}").t().contiguous(), bias=bias)

        w_in, b_in = stack_parallel([mat(x + n) for n in "qkv"], [mat(x + n + ".b") for n in "qkv"], [mat(y + n) for n in "qkvg"])
        blocks = [HybridBlock("parallel_mixer", None, parallel=ParallelMixerWeights(
            attn=AttentionMixerWeights(w_in=None, out_proj=None, heads=a["heads"], kv_heads=a["kv_heads"], dim=a["dim"], vdim=a["vdim"],
                                       scale=a["scale"], window=a["mask"]["size"], means=a["mask"]["pool"], gain=m["left_scale"]),
            ret=RetentionWeights(inv_freq=rope_inv_freq(r["rot"]["dims"], r["rot"]["base"], None)[0].to(device),
                                 decay=torch.tensor(r["decay"], dtype=torch.float32, device=device), heads=r["heads"], dim=r["dim"],
                                 vdim=r["vdim"], gain=m["right_scale"]),
            w_in=w_in, b_in=b_in, w_out=join_columns(mat(x + "o"), mat(y + "o"))), around=around(1, vec(x + "o.b") * m["left_scale"]))]
        mlp, z = spec["mlp"], p + "mlp."
        pair = lambda n: torch.cat([mat(z + n + "gate"), mat(z + n + "up")], 0)      # noqa: E731,B023
        if mlp and mlp["kind"] == "dense":
            blocks.append(HybridBlock("mlp", None, up=pair(""), down=mat(z + "down"), gated=True, act="clipped_swiglu", act_alpha=GLU_SLOPE,
                                      act_limit=mlp["limit"], around=around(2)))
        elif mlp:
            route = mlp["router"]
            blocks.append(HybridBlock("moe_stream", None, around=around(2), moe=MoeBlockWeights(
                router=mat(z + "router"), correction=None, gate_up=torch.stack([pair(f"e{n}.") for n in range(route["experts"])]),
                down=torch.stack([mat(f"{z}e{n}.down") for n in range(route["experts"])]), top=route["top"], scale=1.0, limit=0.0, alpha=1.0,
                act="silu", groups=(route["groups"]["count"], route["groups"]["keep"]), normalise=True)))
        layers.append(blocks)
    return HybridWeights(embed=mat("embed"), blocks=[b for bs in layers for b in bs], final_norm=vec("final.norm"),
                         final_norm_b=vec("final.norm.b"), lm_head=mat("head"), runs=layers, streams=cfg.extra["streams"])


def load_fusolix_weights(path, cfg: ModelConfig, dtype=torch.bfloat16, device="cpu") -> HybridWeights:
    from ..loading.checkpoint import TensorSource

    src = TensorSource(path)

    def get(name):
        if not src.has(name):
            raise KeyError(f"{path}: missing tensor {name}")
        return src.get(name)

    return build_fusolix_weights(get, cfg, dtype, device)


def fusolix_shapes(cfg: ModelConfig) -> dict[str, tuple]:
    """Tensor names and shapes of a checkpoint of this configuration."""
    H, V, S, K = cfg.hidden_size, cfg.vocab_size, cfg.extra["streams"], cfg.extra["taps"]
    out = {"embed": (V, H), "head": (V, H), "final.norm": (H,), "final.norm.b": (H,)}
    for i, spec in enumerate(cfg.extra["layer_specs"]):
        p, mlp = f"l{i}.", spec["mlp"]
        for q in (1, 2) if mlp else (1,):
            out.update({f"{p}norm{q}": (H,), f"{p}norm{q}.b": (H,), f"{p}canon{q}": (H, K), f"{p}hc{q}.in": (S,), f"{p}hc{q}.out": (S,),
                        f"{p}hc{q}.mix": (S, S)})
        a, r = spec["mixer"]["left"], spec["mixer"]["right"]
        rows = dict(q=a["heads"] * a["dim"], k=a["kv_heads"] * a["dim"], v=a["kv_heads"] * a["vdim"])
        out.update({f"{p}mix.left.{n}": (k, H) for n, k in rows.items()})
        out.update({f"{p}mix.left.{n}.b": (k,) for n, k in rows.items()})
        out.update({p + "mix.left.o": (H, a["heads"] * a["vdim"]), p + "mix.left.o.b": (H,), p + "mix.right.o": (H, r["heads"] * r["vdim"])})
        out.update({f"{p}mix.right.{n}": (r["heads"] * r[d], H) for n, d in (("q", "dim"), ("k", "dim"), ("v", "vdim"), ("g", "vdim"))})
        if mlp and mlp["kind"] == "moe":
            out[p + "mlp.router"] = (mlp["router"]["experts"], H)
        parts = [] if not mlp else [("", mlp["ff"])] if mlp["kind"] == "dense" else [(f"e{n}.", mlp["expert"]["ff"]) for n in range(mlp["router"]["experts"])]
        for name, ff in parts:
            out.update({f"{p}mlp.{name}gate": (ff, H), f"{p}mlp.{name}up": (ff, H), f"{p}mlp.{name}down": (H, ff)})
    return out


def random_fusolix_tensors(cfg: ModelConfig, seed: int = 0, dtype=torch.bfloat16, device="cpu") -> dict:
    """Random tensors under the checkpoint's names: projections of unit gain, norm weights around one, streams that differ
    and keep their size."""
    g = torch.Generator(device=device).manual_seed(seed)
    out, S = {}, cfg.extra["streams"]
    for name, shape in fusolix_shapes(cfg).items():
        t, leaf = torch.randn(*shape, generator=g, device=device), name.rsplit(".", 1)[-1]
        if ".hc" in name:
            t = {"in": (1 + 0.3 * t) / S, "out": 1 + 0.3 * t}.get(leaf, t)
            if leaf == "mix":
                t = 0.8 * torch.eye(S, device=device) + 0.2 / S + 0.05 * t
        elif len(shape) == 2:
            t = t * (0.5 if leaf.startswith("canon") else 1.0) * shape[1] ** -0.5
        elif leaf == "b":
            t = 0.1 * t
        else:
            t = 1 + 0.2 * t
        out[name] = t.to(dtype)
    return out


def random_fusolix_weights(cfg: ModelConfig, seed: int = 0, dtype=torch.bfloat16, device="cpu") -> HybridWeights:
    t = random_fusolix_tensors(cfg, seed, torch.bfloat16 if dtype == torch.bfloat16 else torch.float32, device)
    return build_fusolix_weights(t.__getitem__, cfg, dtype, device)


def fusolix_config_dict(cfg: ModelConfig) -> dict:
    return dict(architecture="Fusolix", vocab=cfg.vocab_size, width=cfg.hidden_size, layers=cfg.extra["layer_specs"],
                streams=cfg.extra["streams"], canon=dict(taps=cfg.extra["taps"]), embedding=dict(scale=cfg.embed_scale),
                norm=dict(eps=cfg.rms_norm_eps))


def save_fusolix_checkpoint(path, cfg: ModelConfig, tensors: dict) -> None:
    from safetensors.torch import save_file

    path = Path(path)
    path.mkdir(parents=True, exist_ok=True)
    save_file({k: v.detach().cpu().contiguous() for k, v in tensors.items()}, str(path / "model.safetensors"))
    (path / "config.json").write_text(json.dumps(fusolix_config_dict(cfg)))
