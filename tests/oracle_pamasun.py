"""Plain, slow statement of the Pamasun decoder (whole sequences, fp64 by default), one function per
mechanism, written from the model's equations. It takes the raw configuration record and the checkpoint's
tensors by name and shares no code with the package."""
import math

import torch


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
    q = rms((h @ w["q"].T).view(n, heads, dim), eps) * w["q.norm"]
    k = rms((h @ w["k"].T).view(n, kv_heads, dim), eps) * w["k.norm"]
    v = (h @ w["v"].T).view(n, kv_heads, vdim)
    group = heads // kv_heads
    bias = distance_bias(w["r1"], w["r2"], n)
    out = torch.zeros(n, heads, vdim, dtype=h.dtype)
    for a in range(heads):
        s = q[:, a] @ k[:, a // group].T * scale - bias[a]
        s = s.masked_fill(torch.ones(n, n).triu(1).bool(), float("-inf"))
        out[:, a] = sink_softmax(s, w["sink"][a]) @ v[:, a // group]
    gated = out.reshape(n, heads * vdim) * torch.sigmoid(h @ w["g"].T)
    return gated @ w["o"].T


def delta_inputs(h, w, heads, dim):
    """Everything the recurrence reads, each [n, heads, dim]: r, k, v, decay, removal rate."""
    n = h.shape[0]
    r, k, v = ((h @ w[x].T).view(n, heads, dim) for x in ("r", "k", "v"))
    z = torch.tanh(h @ w["w1"].T) @ w["w2"].T + w["w0"]
    decay = torch.exp(-math.exp(-0.5) * torch.sigmoid(z)).view(n, heads, dim)
    rate = torch.sigmoid(h @ w["a"].T + w["a.b"]).view(n, heads, dim)
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
    o = rms(o, eps).reshape(n, heads * dim) * w["norm"] * torch.sigmoid(h @ w["g"].T)
    return o @ w["o"].T


def polynorm(z, coef, eps):
    a, b, c, e = coef
    return a * rms(z, eps) + b * rms(z ** 2, eps) + c * rms(z ** 3, eps) + e


def dense_mlp(h, w, eps):
    return polynorm(h @ w["up"].T, w["act"], eps) @ w["down"].T


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
    logits = around_zero_norm(x, t["final.norm"], eps) @ t["head"].T
    return (logits, torch.stack(stream)) if want_layers else logits
