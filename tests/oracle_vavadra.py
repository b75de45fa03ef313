"""Plain, slow statement of the Vavadra decoder (whole sequences, fp64 by default), one function per mechanism, written
from the model's equations. It takes the raw configuration record and the checkpoint's tensors by name and shares no code
with the package.

``with bf16_activations():`` rounds every activation between the operations to bf16 (inputs and results of the
projections, keys, latents, head outputs), with everything else still exact: the error that rounding alone causes, which
bounds what a bf16 run may differ by."""
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


def linear(x, w, b=None):
    y = act(x) @ w.T
    return act(y if b is None else y + b)


def unit_rms(x, eps):
    """x over the root of (mean square + eps), along the last dimension."""
    return x / (x.pow(2).mean(-1, keepdim=True) + eps).sqrt()


def norm(x, w, eps):
    return unit_rms(x, eps) * w


def rotate(x, rot, start=0):
    """x [n, heads, width]: neighbouring dimensions (0, 1), (2, 3), .. of the first rot.dims turned by the position's
    angles; the rest passes."""
    n = rot["dims"]
    f = torch.tensor([rot["base"] ** (-2 * i / n) for i in range(n // 2)], dtype=torch.float64)
    a = (torch.arange(start, start + x.shape[0], dtype=torch.float64)[:, None] * f)[:, None]
    c, s = a.cos().to(x.dtype), a.sin().to(x.dtype)
    out = x.clone()
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    out[..., 0:n:2], out[..., 1:n:2] = u * c - v * s, v * c + u * s
    return out


def chunk_mask(n, size):
    """[query, key]: earlier or equal, and in the same run of ``size`` positions counted from the first."""
    p = torch.arange(n)
    return (p[None, :] <= p[:, None]) & (p[None, :] // size == p[:, None] // size)


def window_mask(n, size):
    """[query, key]: itself and the size - 1 positions before it."""
    d = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    return (d >= 0) & (d < size)


def attend(scores, visible, v, sink=None):
    s = scores.masked_fill(~visible, float("-inf"))
    if sink is not None:
        s = torch.cat([s, sink.expand(s.shape[0], 1)], -1)
    return torch.softmax(s, -1)[:, :v.shape[0]] @ v


def map_weight(w, diff):
    """The factor of the second map."""
    return torch.exp((w["lq1"] * w["lk1"]).sum()) - torch.exp((w["lq2"] * w["lk2"]).sum()) + diff


def combine_maps(a1, a2, lam, diff, eps):
    return unit_rms(a1 - lam * a2, eps) * (1 - diff)


def attention(h, w, m, eps):
    """Differential attention over chunks. h [n, width] -> [n, width]; w: the mixer's tensors by short name."""
    n, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k = linear(h, w["q"], w["q.b"]).view(n, H, 2, D), linear(h, w["k"], w["k.b"]).view(n, G, 2, D)
    v = linear(h, w["v"], w["v.b"]).view(n, G, V)
    lam, vis, out = map_weight(w, m["diff"]), chunk_mask(n, m["mask"]["size"]), []
    for a in range(H):
        g = a // (H // G)
        maps = [attend(q[:, a, i] @ k[:, g, i].T * m["scale"], vis, v[:, g]) for i in (0, 1)]
        out.append(combine_maps(*maps, lam, m["diff"], eps))
    return linear(torch.cat(out, -1), w["o"])


def latent_attention(h, w, m, eps):
    n, H, D, R, V, C = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = linear(h, w["q"]).view(n, H, D + R)
    d = linear(h, w["dkv"])
    c, kr = act(norm(d[:, :C], w["dkv.norm"], eps)), act(rotate(d[:, None, C:], m["rot"]))[:, 0]
    qn, qr = q[..., :D], act(rotate(q[..., D:], m["rot"]))
    kn, v = linear(c, w["uk"]).view(n, H, D), linear(c, w["uv"]).view(n, H, V)
    vis = window_mask(n, m["mask"]["size"])
    out = [attend((qn[:, a] @ kn[:, a].T + qr[:, a] @ kr.T) * m["scale"], vis, v[:, a], w["sink"][a]) for a in range(H)]
    return linear(torch.cat(out, -1), w["o"])


def short_conv(x, taps):
    """Causal convolution per channel: taps [channels, K], the last column for the current token; then silu."""
    n, K = x.shape[0], taps.shape[1]
    padded = torch.cat([x.new_zeros(K - 1, x.shape[1]), x], 0)
    y = sum(padded[j:j + n] * taps[:, j] for j in range(K))
    return act(y * torch.sigmoid(y))


def unit(x):
    return x / (x.pow(2).sum(-1, keepdim=True) + 1e-6).sqrt()


def delta_rates(h, w):
    """(write rate, decay) per token and head."""
    z = act(h) @ w["a"].T + w["dt_bias"]
    soft = torch.log1p(torch.exp(-z.abs())) + z.clamp(min=0)
    return torch.sigmoid(act(h) @ w["b"].T), torch.exp(-torch.exp(w["A_log"]) * soft)


def delta_memory(q, k, v, beta, g):
    """q, k [n, H, D], v [n, H, V], beta, g [n, H] -> read-outs [n, H, V]; the state starts at zero."""
    S, out = q.new_zeros(q.shape[1], q.shape[2], v.shape[2]), []
    for t in range(q.shape[0]):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out)


def delta(h, w, m, eps):
    n, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (short_conv(linear(h, w[z]), w[z + ".conv"]) for z in "qkv")
    q, k = unit(q.view(n, G, D)) * D ** -0.5, unit(k.view(n, G, D))
    q, k = q.repeat_interleave(H // G, 1), k.repeat_interleave(H // G, 1)
    beta, g = delta_rates(h, w)
    o = norm(delta_memory(q, k, v.view(n, H, V), beta, g), w["norm"], eps).reshape(n, H * V)
    gate = linear(h, w["g"])
    return linear(o * gate * torch.sigmoid(gate), w["o"])


def clipped_glu(g, u, limit):
    g, u = g.clamp(max=limit), u.clamp(-limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


def dense_mlp(h, w, limit):
    return linear(clipped_glu(linear(h, w["gate"]), linear(h, w["up"]), limit), w["down"])


def choose(z, correction, top, scale):
    """Router logits [n, E] -> (chosen experts [n, top], their weights)."""
    s = torch.softmax(z, -1)
    ids = (s + correction).topk(top, -1)[1]
    return ids, s.gather(1, ids) * scale


def experts(h, w, spec):
    r = spec["router"]
    ids, wts = choose(act(h) @ w["router"].T, w["correction"], r["top"], r["scale"])
    out = torch.zeros_like(h)
    for e in range(r["experts"] + r["identity"]):
        tok, slot = torch.nonzero(ids == e, as_tuple=True)
        if tok.numel():
            sub = {k: w.get(f"e{e}.{k}") for k in ("gate", "up", "down")}
            y = act(h[tok]) if e >= r["experts"] else dense_mlp(h[tok], sub, spec["expert"]["limit"])
            out[tok] += y * wts[tok, slot][:, None]
    sh = spec.get("shared")
    return out if not sh else out + dense_mlp(h, {k: w["shared." + k] for k in ("gate", "up", "down")}, sh["limit"])


MIXERS = {"attention": lambda *a: attention(*a), "latent_attention": lambda *a: latent_attention(*a), "delta": lambda *a: delta(*a)}


def layer_runs(cfg):
    """(layer, number of the pass it begins or None) in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    passes = [(i, t if i == a else None) for t in range(loop["times"]) for i in range(a, b)]
    return [(i, None) for i in range(a)] + passes + [(i, None) for i in range(b, n)]


def before_pass(x, first, step, t):
    """The stream as pass t of the loop gets it; ``first`` is the embedding."""
    return (x if t == 0 else x + first) + step[t]


def forward(cfg, tensors, tokens, dtype=torch.float64, want_layers=False):
    """Logits [n, vocab] of one whole sequence (and the residual stream after every layer)."""
    t = {k: v.to(dtype) for k, v in tensors.items()}
    eps = cfg["norm"]["eps"]
    first = t["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    x, stream = first, []
    for i, number in layer_runs(cfg):
        spec, p = cfg["layers"][i], f"l{i}."
        sub = lambda part: {k[len(p + part):]: v for k, v in t.items() if k.startswith(p + part)}  # noqa: E731
        if number is not None:
            x = before_pass(x, first, t["loop.step"], number)
        x = x + MIXERS[spec["type"]](norm(x, t[p + "norm1"], eps), sub("mix."), spec["mixer"], eps)
        if spec.get("mlp"):
            x = x + experts(norm(x, t[p + "norm2"], eps), sub("mlp."), spec["mlp"])
        stream.append(x)
    logits = act(norm(x, t["final.norm"], eps)) @ t["embed"].T * cfg["logit_scale"]
    return (logits, torch.stack(stream)) if want_layers else logits


# ----------------------------------------------------------------------------- configurations
def _shapes_mlp(p, H, mlp):
    r, out = mlp["router"], {p + "mlp.router": (mlp["router"]["experts"] + mlp["router"]["identity"], H)}
    out[p + "mlp.correction"] = (r["experts"] + r["identity"],)
    parts = [(f"e{e}", mlp["expert"]["ff"]) for e in range(r["experts"])] + ([("shared", mlp["shared"]["ff"])] if mlp.get("shared") else [])
    for name, ff in parts:
        out.update({f"{p}mlp.{name}.gate": (ff, H), f"{p}mlp.{name}.up": (ff, H), f"{p}mlp.{name}.down": (H, ff)})
    return out


def random_tensors(cfg, seed, dtype=torch.float32):
    """Checkpoint of a configuration with random values: projections of unit gain, decays of short and long memory, a
    router whose choices stand apart."""
    gen = torch.Generator().manual_seed(seed)
    n = lambda *s: torch.randn(*s, generator=gen)          # noqa: E731
    lin = lambda o, i: n(o, i) * i ** -0.5               # noqa: E731
    H = cfg["width"]
    t = {"embed": lin(cfg["vocab"], H) * 2, "final.norm": 1 + 0.3 * n(H)}
    if cfg.get("loop"):
        t["loop.step"] = n(cfg["loop"]["times"], H) * 0.7
    for i, spec in enumerate(cfg["layers"]):
        p, m = f"l{i}.", spec["mixer"]
        x, h, d, v = p + "mix.", m["heads"], m["dim"], m["vdim"]
        t[p + "norm1"] = 1 + 0.3 * n(H)
        if spec["type"] == "attention":
            g = m["kv_heads"]
            t.update({x + "q": lin(h * 2 * d, H) * 1.5, x + "k": lin(g * 2 * d, H) * 1.5, x + "v": lin(g * v, H), x + "o": lin(H, h * v),
                      x + "q.b": n(h * 2 * d) * 0.5, x + "k.b": n(g * 2 * d) * 0.5, x + "v.b": n(g * v) * 0.5})
            t.update({x + z: n(d) * 0.6 * d ** -0.25 for z in ("lq1", "lk1", "lq2", "lk2")})
        elif spec["type"] == "latent_attention":
            c, r = m["kv_rank"], m["rot_dim"]
            t.update({x + "q": lin(h * (d + r), H) * 1.5, x + "dkv": lin(c + r, H), x + "dkv.norm": 1 + 0.3 * n(c), x + "uk": lin(h * d, c),
                      x + "uv": lin(h * v, c), x + "sink": n(h) + 1, x + "o": lin(H, h * v)})
        else:
            g, K = m["kv_heads"], m["conv"]
            for z, rows in (("q", g * d), ("k", g * d), ("v", h * v)):
                t.update({x + z: lin(rows, H), f"{x}{z}.conv": n(rows, K) * K ** -0.5})
            t.update({x + "b": lin(h, H), x + "a": lin(h, H), x + "A_log": n(h) * 0.5, x + "dt_bias": n(h) - 2, x + "norm": 1 + 0.3 * n(v),
                      x + "g": lin(h * v, H), x + "o": lin(H, h * v)})
        if spec.get("mlp"):
            t[p + "norm2"] = 1 + 0.3 * n(H)
            for name, shape in _shapes_mlp(p, H, spec["mlp"]).items():
                t[name] = 0.2 * n(*shape) if len(shape) == 1 else lin(*shape) * (4 if name.endswith("router") else 1)
    return {k: v.to(torch.bfloat16).to(dtype) for k, v in t.items()}


def moe(ff, n_experts, identity, top, limit=1.2, scale=1.7, shared=None, shared_limit=0.9):
    return dict(kind="moe", expert=dict(ff=ff, limit=limit), router=dict(experts=n_experts, identity=identity, top=top, scale=scale),
                shared=dict(ff=shared, limit=shared_limit) if shared else None)


def attn_spec(heads, kv_heads, dim, vdim, chunk, scale, diff, mlp):
    return dict(type="attention", mlp=mlp, mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, diff=diff,
                                                      mask=dict(size=chunk)))


def latent_spec(heads, dim, rot, vdim, kv_rank, window, scale, mlp, base=9000.0):
    return dict(type="latent_attention", mlp=mlp, mixer=dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=kv_rank, scale=scale,
                                                             mask=dict(size=window), rot=dict(dims=rot, base=base)))


def delta_spec(heads, kv_heads, dim, vdim, conv, mlp):
    return dict(type="delta", mlp=mlp, mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv))


def model_config(vocab, width, layers, loop=None, eps=1e-5, embed_scale=3.0, logit_scale=0.8):
    return dict(architecture="Vavadra", vocab=vocab, width=width, layers=layers, norm=dict(eps=eps), embedding=dict(scale=embed_scale),
                logit_scale=logit_scale, loop=dict(zip(("start", "stop", "times"), loop)) if loop else None)


# Configurations of the tests: mixed orders, unequal layers, layers without feed-forward, loops at the start, in the middle
# and over the end, windows and chunks that do and do not fall on page borders, sizes no tensor-core tile or vector access
# divides, and values that happen to be equal or one.
CONFIGS = {
    "mixed": model_config(160, 96, [
        delta_spec(4, 2, 32, 48, 3, moe(40, 5, 2, 2, shared=56)), latent_spec(3, 24, 16, 40, 48, 21, 0.25, moe(32, 6, 1, 3, 0.7, shared=24)),
        attn_spec(6, 2, 16, 40, 18, 0.3, 0.45, None), latent_spec(5, 32, 8, 24, 40, 33, 0.2, moe(48, 4, 3, 2, 2.0, 1.0, 72, 1.6))],
        loop=(1, 3, 3)),
    "odd": model_config(101, 75, [
        attn_spec(3, 3, 9, 11, 13, 0.35, 0.2, moe(33, 3, 1, 1, shared=17)), delta_spec(3, 1, 10, 7, 5, moe(21, 7, 0, 4, 3.0, 0.6)),
        latent_spec(3, 9, 6, 11, 13, 1, 0.4, None), delta_spec(2, 2, 33, 12, 1, None)],
        loop=(0, 2, 2), eps=1e-3, embed_scale=1.0, logit_scale=1.0),
    "attention_only": model_config(128, 64, [
        attn_spec(2, 1, 32, 64, 64, 0.18, 0.8, moe(64, 4, 1, 2, shared=64)), attn_spec(8, 8, 8, 16, 129, 0.5, 0.1, None)], loop=(1, 2, 3)),
    "latent_only": model_config(96, 64, [
        latent_spec(1, 8, 8, 8, 8, 16, 0.9, moe(64, 2, 2, 2, shared=64)), latent_spec(8, 64, 64, 64, 64, 64, 0.12, None),
        latent_spec(2, 16, 2, 72, 104, 200, 0.4, moe(16, 9, 1, 5, shared=32))], loop=(2, 3, 2)),
    "delta_only": model_config(128, 64, [
        delta_spec(2, 2, 16, 16, 4, moe(32, 4, 2, 3, shared=32)), delta_spec(6, 3, 64, 24, 2, None)]),
    "wide": model_config(264, 256, [
        latent_spec(20, 64, 32, 64, 256, 90, 0.1, moe(128, 8, 2, 3, shared=192)), delta_spec(4, 2, 128, 128, 4, moe(96, 16, 4, 6, 0.8)),
        attn_spec(10, 2, 64, 128, 72, 0.12, 0.5, moe(64, 12, 2, 3, shared=64)), attn_spec(4, 4, 40, 72, 48, 0.16, 0.3, None)], loop=(1, 4, 2)),
}
