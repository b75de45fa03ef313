"""Plain, slow statement of the Pamasun decoder (whole sequences, fp64 by default), one function per
mechanism, written from the model's equations. It takes the raw configuration record and the checkpoint's
tensors by name and shares no code with the package.

``with bf16_activations():`` rounds every activation between the operations to bf16 (inputs and results of
the projections, normalised queries and keys, head outputs), with everything else still exact: the error
that rounding alone causes, which bounds what a bf16 run may differ by."""
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


def rms(x, eps):
    """x over the root of (mean square + eps), along the last dimension."""
    return x / (x.pow(2).mean(-1, keepdim=True) + eps).sqrt()


def around_zero_norm(x, w, eps):
    """RMS norm whose stored weight is the offset from one."""
    return rms(x, eps) * (1 + w)


def distance_bias(r1, r2, n):
    """[heads, n, n]: what the score of query i and key j loses, r1 ln(1 + r2 (i - j)) (0 above the diagonal)."""
    d = (torch.arange(n)[:, None] - torch.arange(n)[None, :]).clamp(min=0).to(r1.dtype)
    return r1[:, None, None] * torch.log(1 + r2[:, None, None] * d)


def sink_softmax(s, sink):
    """Softmax along the last dimension with one more term exp(sink) in the denominator."""
    m = torch.maximum(s.amax(-1, keepdim=True), sink)
    e = (s - m).exp()
    return e / (e.sum(-1, keepdim=True) + (sink - m).exp())


def attention(h, w, heads, kv_heads, dim, vdim, scale, eps):
    """w: the mixer's tensors by their short names. h [n, width] -> [n, width]."""
    n = h.shape[0]
    q = act(rms(linear(h, w["q"]).view(n, heads, dim), eps) * w["q.norm"])
    k = act(rms(linear(h, w["k"]).view(n, kv_heads, dim), eps) * w["k.norm"])
    v = linear(h, w["v"]).view(n, kv_heads, vdim)
    group = heads // kv_heads
    bias = distance_bias(w["r1"], w["r2"], n)
    out = torch.zeros(n, heads, vdim, dtype=h.dtype)
    for a in range(heads):
        s = q[:, a] @ k[:, a // group].T * scale - bias[a]
        s = s.masked_fill(torch.ones(n, n).triu(1).bool(), float("-inf"))
        out[:, a] = sink_softmax(s, w["sink"][a]) @ v[:, a // group]
    gated = out.reshape(n, heads * vdim) * torch.sigmoid(linear(h, w["g"]))
    return linear(gated, w["o"])


def delta_inputs(h, w, heads, dim):
    """Everything the recurrence reads, each [n, heads, dim]: r, k, v, decay, removal rate."""
    n = h.shape[0]
    r, k, v = (linear(h, w[x]).view(n, heads, dim) for x in ("r", "k", "v"))
    z = torch.tanh(linear(h, w["w1"])) @ w["w2"].T + w["w0"]
    decay = torch.exp(-math.exp(-0.5) * torch.sigmoid(z)).view(n, heads, dim)
    rate = torch.sigmoid(linear(h, w["a"]) + w["a.b"]).view(n, heads, dim)
    return r, k, v, decay, rate


def delta_recurrence(r, k, v, decay, rate, state=None):
    """Generalized delta rule token by token. Returns (o [n, heads, dim], last state [heads, dim, dim])."""
    n, heads, dim = r.shape
    s = torch.zeros(heads, dim, v.shape[-1], dtype=r.dtype) if state is None else state.clone()
    out = []
    for t in range(n):
        u = k[t] / (k[t].pow(2).sum(-1, keepdim=True) + 1e-6).sqrt()
        read = (u[:, :, None] * s).sum(1)                                  # u^T S of the old state
        s = decay[t][:, :, None] * s - (rate[t] * u)[:, :, None] * read[:, None, :] + k[t][:, :, None] * v[t][:, None, :]
        out.append((s * r[t][:, :, None]).sum(1))
    return torch.stack(out), s


def general_delta(h, w, heads, dim, eps):
    n = h.shape[0]
    o, _ = delta_recurrence(*delta_inputs(h, w, heads, dim))
    o = rms(o, eps).reshape(n, heads * dim) * w["norm"] * torch.sigmoid(linear(h, w["g"]))
    return linear(o, w["o"])


def polynorm(z, coef, eps):
    a, b, c, e = coef
    return a * rms(z, eps) + b * rms(z ** 2, eps) + c * rms(z ** 3, eps) + e


def dense_mlp(h, w, eps):
    return linear(polynorm(linear(h, w["up"]), w["act"], eps), w["down"])


def layer_order(cfg):
    """Indices of the layers in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


def forward(cfg, tensors, tokens, dtype=torch.float64, want_layers=False):
    """Logits [n, vocab] of one whole sequence (and the residual stream after every layer run)."""
    t = {k: v.to(dtype) for k, v in tensors.items()}
    eps = cfg["norm"]["eps"]
    x = t["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    stream = []
    for i in layer_order(cfg):
        spec, p = cfg["layers"][i], f"l{i}."
        sub = lambda part: {k[len(p + part):]: v for k, v in t.items() if k.startswith(p + part)}  # noqa: E731
        m, h = spec["mixer"], around_zero_norm(x, t[p + "norm1"], eps)
        if spec["type"] == "attention":
            y = attention(h, sub("mix."), m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], eps)
        else:
            y = general_delta(h, sub("mix."), m["heads"], m["dim"], eps)
        x = x + around_zero_norm(y, t[p + "norm1b"], eps) * t[p + "ls1"]
        if spec.get("mlp"):
            y = dense_mlp(around_zero_norm(x, t[p + "norm2"], eps), sub("mlp."), eps)
            x = x + around_zero_norm(y, t[p + "norm2b"], eps) * t[p + "ls2"]
        stream.append(x)
    logits = act(around_zero_norm(x, t["final.norm"], eps)) @ t["head"].T
    return (logits, torch.stack(stream)) if want_layers else logits


def random_tensors(cfg, seed, rank=5, dtype=torch.float32):
    """Checkpoint of a configuration with random values spread so that no mechanism is idle: gates and sinks
    of both signs, distance rates between 0.05 and 0.6, decays from near 1 down to their floor."""
    g = torch.Generator().manual_seed(seed)
    n = lambda *s: torch.randn(*s, generator=g)          # noqa: E731
    u = lambda *s: torch.rand(*s, generator=g)           # noqa: E731
    lin = lambda o, i: n(o, i) * i ** -0.5               # noqa: E731
    H, V = cfg["width"], cfg["vocab"]
    t = {"embed": n(V, H) * 0.7, "head": lin(V, H), "final.norm": 0.3 * n(H)}
    for i, spec in enumerate(cfg["layers"]):
        p, m = f"l{i}.", spec["mixer"]
        for k in ("norm1", "norm1b", "norm2", "norm2b"):
            t[p + k] = 0.3 * n(H)
        for k in ("ls1", "ls2"):
            t[p + k] = 0.5 + u(H)
        x = p + "mix."
        if spec["type"] == "attention":
            h, kv, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            t.update({x + "q": lin(h * dk, H), x + "k": lin(kv * dk, H), x + "v": lin(kv * dv, H), x + "g": lin(h * dv, H),
                      x + "o": lin(H, h * dv), x + "q.norm": 1 + 0.4 * n(dk), x + "k.norm": 1 + 0.4 * n(dk), x + "r1": 0.1 + u(h),
                      x + "r2": 0.05 + 0.55 * u(h), x + "sink": 2 * n(h)})
        else:
            hd = m["heads"] * m["dim"]
            t.update({x + k: lin(hd, H) for k in ("r", "k", "v", "g", "a")})
            t.update({x + "a.b": n(hd), x + "w0": -3 + 3 * n(hd), x + "norm": 1 + 0.3 * n(hd), x + "w1": lin(rank, H),
                      x + "w2": lin(hd, rank), x + "o": lin(H, hd)})
        if spec.get("mlp"):
            ff = spec["mlp"]["ff"]
            t.update({p + "mlp.up": lin(ff, H), p + "mlp.down": lin(H, ff), p + "mlp.act": torch.tensor([0.7, 0.5, 0.3, 0.2]) + 0.1 * n(4)})
        else:
            for k in ("norm2", "norm2b", "ls2"):
                del t[p + k]
    return {k: v.to(torch.bfloat16).to(dtype) for k, v in t.items()}


def attn_spec(heads, kv_heads, dim, vdim, scale, ff):
    return dict(type="attention", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale),
                mlp=None if ff is None else dict(kind="dense", ff=ff))


def delta_spec(heads, dim, ff):
    return dict(type="general_delta", mixer=dict(heads=heads, dim=dim), mlp=None if ff is None else dict(kind="dense", ff=ff))


def model_config(vocab, width, layers, loop, scale=3.0, eps=1e-5):
    return dict(architecture="Pamasun", vocab=vocab, width=width, layers=layers, loop=loop, embedding=dict(scale=scale),
                norm=dict(eps=eps))


# Configurations of the tests: mixed orders, unequal layers, a layer without feed-forward, sizes no
# tensor-core tile or vector access divides, and values that happen to be equal or one.
CONFIGS = {
    "mixed": model_config(160, 96, [delta_spec(3, 24, 112), attn_spec(6, 2, 48, 24, 0.17, 72), delta_spec(2, 32, None)],
                          dict(start=0, stop=2, times=2)),
    "odd": model_config(101, 75, [attn_spec(3, 1, 20, 13, 0.31, 50), delta_spec(1, 17, 33), attn_spec(4, 4, 12, 36, 0.2, None)],
                        dict(start=1, stop=3, times=3), scale=1.0, eps=1e-4),
    "attention_only": model_config(128, 64, [attn_spec(2, 2, 64, 64, 0.125, 64), attn_spec(8, 1, 16, 72, 0.3, 96)], None),
    "delta_only": model_config(96, 64, [delta_spec(1, 64, 48), delta_spec(2, 132, 40)], dict(start=1, stop=2, times=1)),
    "wide": model_config(264, 256, [attn_spec(10, 2, 128, 96, 0.09, 320), delta_spec(2, 128, 256)], dict(start=0, stop=2, times=2)),
}
