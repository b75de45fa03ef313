"""Plain, slow statement of the Govopel decoder (whole sequences, fp64 by default), one function per mechanism,
written from the model's equations. It takes the raw configuration record and the checkpoint's tensors by name
and shares no code with the package.

``with bf16_activations():`` rounds every activation between the operations to bf16 (inputs and results of the
projections, queries and keys, latents, head outputs), with everything else still exact: the error that
rounding alone causes, which bounds what a bf16 run may differ by."""
import contextlib
import math

import torch

_round = None


@contextlib.contextmanager
def bf16_activations():
    global _round
    _round = lambda x: x.to(torch.bfloat16).to(x.dtype)      # noqa: E731
    try:
        yield
    finally:
        _round = None


def act(x):
    return x if _round is None else _round(x)


def linear(x, w):
    return act(act(x) @ w.T)


def unit_rms(x, eps):
    """x over the root of (mean square + eps), along the last dimension."""
    return x / (x.pow(2).mean(-1, keepdim=True) + eps).sqrt()


def norm(x, w, eps):
    return unit_rms(x, eps) * w


def frequencies(rot):
    """(angle per position of every pair, factor on cosine and sine)."""
    n, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    plain = [base ** (-2 * i / n) for i in range(n // 2)]
    if not sc:
        return torch.tensor(plain, dtype=torch.float64), 1.0
    turn = lambda t: n * math.log(sc["original"] / (2 * math.pi * t)) / (2 * math.log(base))      # noqa: E731
    lo, hi = max(math.floor(turn(sc["fast"])), 0), min(math.ceil(turn(sc["slow"])), n - 1)
    out = []
    for i, f in enumerate(plain):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / sc["factor"] * ramp + f * (1 - ramp))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(sc["factor"]) + 1


def rotate(x, rot, start=0):
    """x [n, heads, width]: the first rot.dims dimensions of each head turned by the position's angles (dimension
    i goes with i + dims / 2); the rest passes."""
    f, m = frequencies(rot)
    half = rot["dims"] // 2
    a = (torch.arange(start, start + x.shape[0], dtype=torch.float64)[:, None] * f)[:, None]
    c, s = (a.cos() * m).to(x.dtype), (a.sin() * m).to(x.dtype)
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], -1)


def chunk_mask(n, size):
    """[query, key]: earlier or equal, and in the same run of ``size`` positions counted from the first."""
    p = torch.arange(n)
    return (p[None, :] <= p[:, None]) & (p[None, :] // size == p[:, None] // size)


def causal_mask(n):
    return torch.ones(n, n).tril().bool()


def soft_cap(s, cap):
    return cap * torch.tanh(s / cap)


def attend(scores, visible, v):
    return torch.softmax(scores.masked_fill(~visible, float("-inf")), -1) @ v


def attention(h, w, m, eps):
    """Mixer with values = projected keys. h [n, width] -> [n, width]; w: the mixer's tensors by short name."""
    n, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q, k = linear(h, w["q"]).view(n, H, D), linear(h, w["k"]).view(n, G, D)
    v = k
    q, k = (act(unit_rms(rotate(z, m["rot"]), eps)) for z in (q, k))
    vis = chunk_mask(n, m["mask"]["size"])
    out = [attend(soft_cap(q[:, a] @ k[:, a // (H // G)].T * m["scale"], m["softcap"]), vis, v[:, a // (H // G)]) for a in range(H)]
    return linear(torch.cat(out, -1), w["o"])


def latent_attention(h, w, m, eps):
    n, H, D, R, V, C = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = linear(norm(linear(h, w["dq"]), w["dq.norm"], eps), w["uq"]).view(n, H, D + R)
    d = linear(h, w["dkv"])
    c, kr = act(norm(d[:, :C], w["dkv.norm"], eps)), act(rotate(d[:, None, C:], m["rot"]))[:, 0]
    qn, qr = q[..., :D], act(rotate(q[..., D:], m["rot"]))
    kn, v = linear(c, w["uk"]).view(n, H, D), linear(c, w["uv"]).view(n, H, V)
    vis = causal_mask(n)
    out = [attend((qn[:, a] @ kn[:, a].T + qr[:, a] @ kr.T) * m["scale"], vis, v[:, a]) for a in range(H)]
    return linear(torch.cat(out, -1), w["o"])


def clipped_glu(g, u, limit):
    g, u = g.clamp(max=limit), u.clamp(-limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


def dense_mlp(h, w, limit):
    return linear(clipped_glu(linear(h, w["gate"]), linear(h, w["up"]), limit), w["down"])


def embed(tokens, table, w, eps):
    return norm(table[torch.as_tensor(tokens)], w, eps)


def forward(cfg, tensors, tokens, dtype=torch.float64, want_layers=False):
    """Logits [n, vocab] of one whole sequence (and the residual stream after every layer)."""
    t = {k: v.to(dtype) for k, v in tensors.items()}
    eps = cfg["norm"]["eps"]
    x = embed(tokens, t["embed"], t["embed.norm"], eps)
    stream = []
    for i, spec in enumerate(cfg["layers"]):
        p = f"l{i}."
        sub = lambda part: {k[len(p + part):]: v for k, v in t.items() if k.startswith(p + part)}  # noqa: E731
        mixer = attention if spec["type"] == "attention" else latent_attention
        x = x + norm(mixer(x, sub("mix."), spec["mixer"], eps), t[p + "norm1"], eps)
        if spec.get("mlp"):
            x = x + norm(dense_mlp(x, sub("mlp."), spec["mlp"]["limit"]), t[p + "norm2"], eps)
        stream.append(x)
    logits = soft_cap(act(norm(x, t["final.norm"], eps)) @ t["embed"].T, cfg["logit_softcap"])
    return (logits, torch.stack(stream)) if want_layers else logits


def random_tensors(cfg, seed, dtype=torch.float32):
    """Checkpoint of a configuration with random values: sharp query latents and projections of unit gain."""
    g = torch.Generator().manual_seed(seed)
    n = lambda *s: torch.randn(*s, generator=g)          # noqa: E731
    lin = lambda o, i: n(o, i) * i ** -0.5               # noqa: E731
    H, V = cfg["width"], cfg["vocab"]
    t = {"embed": lin(V, H) * 2, "embed.norm": 1 + 0.3 * n(H), "final.norm": 1 + 0.3 * n(H)}
    for i, spec in enumerate(cfg["layers"]):
        p, m = f"l{i}.", spec["mixer"]
        x, h, d = p + "mix.", m["heads"], m["dim"]
        t[p + "norm1"] = 1 + 0.3 * n(H)
        if spec["type"] == "attention":
            t.update({x + "q": lin(h * d, H), x + "k": lin(m["kv_heads"] * d, H), x + "o": lin(H, h * m["vdim"])})
        else:
            q, c, r, v = m["q_rank"], m["kv_rank"], m["rot_dim"], m["vdim"]
            t.update({x + "dq": lin(q, H), x + "dq.norm": 1.5 + 0.3 * n(q), x + "uq": lin(h * (d + r), q), x + "dkv": lin(c + r, H),
                      x + "dkv.norm": 1 + 0.3 * n(c), x + "uk": lin(h * d, c), x + "uv": lin(h * v, c), x + "o": lin(H, h * v)})
        if spec.get("mlp"):
            ff = spec["mlp"]["ff"]
            t.update({p + "norm2": 1 + 0.3 * n(H), p + "mlp.gate": lin(ff, H), p + "mlp.up": lin(ff, H), p + "mlp.down": lin(H, ff)})
    return {k: v.to(torch.bfloat16).to(dtype) for k, v in t.items()}


def _mlp(ff, limit):
    return None if ff is None else dict(kind="dense", ff=ff, limit=limit)


def attn_spec(heads, kv_heads, dim, rot, chunk, scale, softcap, ff, limit=1.5, base=3000.0, scaling=(2.5, 300, 20.0, 1.5)):
    r = dict(dims=rot, base=base)
    if scaling:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return dict(type="attention", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=scale, softcap=softcap, rot=r,
                                             mask=dict(size=chunk)), mlp=_mlp(ff, limit))


def latent_spec(heads, dim, rot, vdim, q_rank, kv_rank, scale, ff, limit=1.5, base=20000.0):
    return dict(type="latent_attention", mixer=dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank,
                                                    scale=scale, rot=dict(dims=rot, base=base)), mlp=_mlp(ff, limit))


def model_config(vocab, width, layers, eps=1e-5, logit_softcap=9.0):
    return dict(architecture="Govopel", vocab=vocab, width=width, layers=layers, norm=dict(eps=eps), logit_softcap=logit_softcap)


# Configurations of the tests: mixed orders, unequal layers, layers without feed-forward, chunks that do and do not fall on
# page borders, sizes no tensor-core tile or vector access divides, and values that happen to be equal or one.
CONFIGS = {
    "mixed": model_config(160, 96, [latent_spec(3, 32, 16, 24, 40, 56, 0.3, 112), attn_spec(6, 2, 48, 24, 20, 0.15, 6.0, 72),
                                    latent_spec(5, 24, 24, 40, 24, 32, 0.25, None), attn_spec(4, 1, 32, 32, 16, 0.2, 14.0, 80, 0.7)]),
    "odd": model_config(101, 75, [attn_spec(3, 3, 20, 10, 13, 0.3, 4.0, 50), latent_spec(3, 9, 6, 11, 17, 13, 0.5, 33, 3.0),
                                  attn_spec(5, 1, 33, 22, 1, 0.1, 2.0, None, scaling=None)], eps=1e-3, logit_softcap=25.0),
    "attention_only": model_config(128, 64, [attn_spec(2, 2, 64, 64, 64, 0.125, 10.0, 64, scaling=(1.0, 64, 1.0, 1.0)),
                                             attn_spec(8, 1, 16, 2, 129, 0.6, 30.0, 96, base=10.0, scaling=(40.0, 50, 32.0, 1.0))]),
    "latent_only": model_config(96, 64, [latent_spec(1, 8, 8, 8, 8, 8, 0.9, 64), latent_spec(8, 64, 64, 64, 64, 64, 0.12, 64, 1.0),
                                         latent_spec(2, 16, 2, 72, 120, 104, 0.4, None)]),
    "wide": model_config(264, 256, [latent_spec(20, 128, 64, 128, 96, 512, 0.1, 320), attn_spec(10, 2, 128, 64, 184, 0.1, 18.0, 256),
                                    latent_spec(4, 96, 40, 80, 160, 200, 0.12, 192)]),
}
