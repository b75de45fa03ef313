"""Plain, slow statement of the Fusolix decoder (whole sequences, fp64 by default), one function per mechanism, written
from the model's equations. It takes the raw configuration record and the checkpoint's tensors by name and shares no code
with the package.

``with bf16_activations():`` rounds every activation between the operations to bf16 (inputs and results of the
projections, keys, values and their means, head outputs), with everything else still exact: the error that rounding alone
causes, which bounds what a bf16 run may differ by."""
import contextlib

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


def layer_norm(x, w, b, eps):
    c = x - x.mean(-1, keepdim=True)
    return c / (c.pow(2).mean(-1, keepdim=True) + eps).sqrt() * w + b


def unit_rms(x, eps):
    return x / (x.pow(2).mean(-1, keepdim=True) + eps).sqrt()


def silu(x):
    return x * torch.sigmoid(x)


# ----------------------------------------------------------------------------- around a sub-layer
def short_conv(h, taps):
    """h plus its causal convolution per channel: taps [channels, K], the last column for the current token."""
    n, K = h.shape[0], taps.shape[1]
    padded = torch.cat([h.new_zeros(K - 1, h.shape[1]), h], 0)
    return h + sum(padded[j:j + n] * taps[:, j] for j in range(K))


def gather_streams(x, w_in):
    """x [n, streams, width] -> the sub-layer's input [n, width]."""
    return (x * w_in[:, None]).sum(1)


def spread(x, y, mix, w_out):
    """The streams behind a sub-layer with result y: stream t is sum_s mix[s, t] x_s + out[t] y."""
    return torch.einsum("nsd,st->ntd", x, mix) + w_out[:, None] * y[:, None]


# ----------------------------------------------------------------------------- mixer
def tokens_seen(n, size):
    """[query, token]: itself and the size - 1 positions before it."""
    d = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    return (d >= 0) & (d < size)


def blocks_seen(n, size, pool):
    """[query, block]: every token of the block lies before the query's window."""
    last = torch.arange(n // pool) * pool + pool - 1
    return last[None, :] <= torch.arange(n)[:, None] - size


def block_means(x, pool):
    """x [n, heads, width] -> means of the full blocks [n // pool, heads, width]."""
    full = x.shape[0] // pool
    return act(x[:full * pool].reshape(full, pool, *x.shape[1:]).mean(1))


def attend(scores, visible, v):
    return torch.softmax(scores.masked_fill(~visible, float("-inf")), -1) @ v


def pooled_attention(h, w, m):
    """Heads of the windowed attention with block means [n, heads * vdim]."""
    n, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    size, pool = m["mask"]["size"], m["mask"]["pool"]
    q, k = linear(h, w["q"], w["q.b"]).view(n, H, D), linear(h, w["k"], w["k.b"]).view(n, G, D)
    v = linear(h, w["v"], w["v.b"]).view(n, G, V)
    keys, vals = torch.cat([k, block_means(k, pool)]), torch.cat([v, block_means(v, pool)])
    visible = torch.cat([tokens_seen(n, size), blocks_seen(n, size, pool)], 1)
    return torch.cat([attend(q[:, a] @ keys[:, a // (H // G)].T * m["scale"], visible, vals[:, a // (H // G)]) for a in range(H)], -1)


def rotate(x, rot, start=0):
    """x [n, heads, width]: dimension i turned with i + dims / 2 by the position's angles, i < dims / 2; the rest passes."""
    half = rot["dims"] // 2
    f = torch.tensor([rot["base"] ** (-2 * i / rot["dims"]) for i in range(half)], dtype=torch.float64)
    a = (torch.arange(start, start + x.shape[0], dtype=torch.float64)[:, None] * f)[:, None]
    c, s = a.cos().to(x.dtype), a.sin().to(x.dtype)
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], -1)


def retain(q, k, v, decay):
    """q, k [n, H, D], v [n, H, V], decay [H] -> read-outs [n, H, V]; the state starts at zero."""
    S, out = q.new_zeros(q.shape[1], q.shape[2], v.shape[2]), []
    for t in range(q.shape[0]):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out)


def retention(h, w, m, eps):
    """Gated heads of the retention [n, heads * vdim]."""
    n, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k = (rotate(linear(h, w[z]).view(n, H, D), m["rot"]) for z in "qk")
    o = retain(q, k * D ** -0.5, linear(h, w["v"]).view(n, H, V), torch.tensor(m["decay"], dtype=h.dtype))
    return unit_rms(o, eps).reshape(n, H * V) * silu(linear(h, w["g"]))


def side_by_side(left, right, m):
    return m["left_scale"] * left + m["right_scale"] * right


def parallel(h, w, m, eps):
    part = lambda p: {k[len(p):]: v for k, v in w.items() if k.startswith(p)}      # noqa: E731
    lw, rw = part("left."), part("right.")
    return side_by_side(linear(pooled_attention(h, lw, m["left"]), lw["o"], lw["o.b"]), linear(retention(h, rw, m["right"], eps), rw["o"]), m)


# ----------------------------------------------------------------------------- feed-forward
def clipped_glu(g, u, limit):
    g, u = g.clamp(max=limit), u.clamp(-limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


def dense(h, w, spec):
    return linear(clipped_glu(linear(h, w["gate"]), linear(h, w["up"]), spec["limit"]), w["down"])


def best_groups(s, groups):
    """[n, experts] of scores -> which experts lie in the groups with the largest scores."""
    per = s.shape[1] // groups["count"]
    best = s.view(s.shape[0], groups["count"], per).amax(-1).topk(groups["keep"], -1)[1]
    return (torch.arange(s.shape[1])[None, :, None] // per == best[:, None, :]).any(-1)


def choose(z, top, groups):
    """Router logits [n, E] -> (chosen experts [n, top], their weights)."""
    s = torch.softmax(z, -1)
    ids = s.masked_fill(~best_groups(s, groups), -1.0).topk(top, -1)[1]
    w = s.gather(1, ids)
    return ids, w / (w.sum(-1, keepdim=True) + 1e-20)


def experts(h, w, spec):
    r = spec["router"]
    ids, wts = choose(act(h) @ w["router"].T, r["top"], r["groups"])
    out = torch.zeros_like(h)
    for e in range(r["experts"]):
        tok, slot = torch.nonzero(ids == e, as_tuple=True)
        if tok.numel():
            y = linear(silu(linear(h[tok], w[f"e{e}.gate"])) * linear(h[tok], w[f"e{e}.up"]), w[f"e{e}.down"])
            out[tok] += y * wts[tok, slot][:, None]
    return out


FEED_FORWARD = {"dense": lambda *a: dense(*a), "moe": lambda *a: experts(*a)}


def embedding(table, tokens, scale):
    return table[torch.as_tensor(tokens)] * scale


def forward(cfg, tensors, tokens, dtype=torch.float64, want_layers=False):
    """Logits [n, vocab] of one whole sequence (and the sum of the streams after every layer)."""
    t = {k: v.to(dtype) for k, v in tensors.items()}
    eps = cfg["norm"]["eps"]
    x = embedding(t["embed"], tokens, cfg["embedding"]["scale"])[:, None].repeat(1, cfg["streams"], 1)
    sums = []
    for i, spec in enumerate(cfg["layers"]):
        p = f"l{i}."
        sub = lambda part: {k[len(p + part):]: v for k, v in t.items() if k.startswith(p + part)}  # noqa: E731

        def sublayer(x, q, f):
            hc, nm = sub(f"hc{q}."), f"{p}norm{q}"
            h = layer_norm(gather_streams(x, hc["in"]), t[nm], t[nm + ".b"], eps)
            return spread(x, f(act(short_conv(h, t[f"{p}canon{q}"]))), hc["mix"], hc["out"])

        x = sublayer(x, 1, lambda h: parallel(h, sub("mix."), spec["mixer"], eps))
        if spec.get("mlp"):
            x = sublayer(x, 2, lambda h: FEED_FORWARD[spec["mlp"]["kind"]](h, sub("mlp."), spec["mlp"]))
        sums.append(x.sum(1))
    logits = act(layer_norm(x.sum(1), t["final.norm"], t["final.norm.b"], eps)) @ t["head"].T
    return (logits, torch.stack(sums)) if want_layers else logits


# ----------------------------------------------------------------------------- configurations
def random_tensors(cfg, seed, dtype=torch.float32):
    """Checkpoint of a configuration with random values: projections of unit gain, streams that differ and stay of the
    same size, a router whose choices stand apart."""
    gen = torch.Generator().manual_seed(seed)
    n = lambda *s: torch.randn(*s, generator=gen)          # noqa: E731
    lin = lambda o, i: n(o, i) * i ** -0.5               # noqa: E731
    H, S, K = cfg["width"], cfg["streams"], cfg["canon"]["taps"]
    t = {"embed": lin(cfg["vocab"], H) * 2, "head": lin(cfg["vocab"], H), "final.norm": 1 + 0.3 * n(H), "final.norm.b": 0.3 * n(H)}
    for i, spec in enumerate(cfg["layers"]):
        p, a, r = f"l{i}.", spec["mixer"]["left"], spec["mixer"]["right"]
        x = p + "mix."
        for q in (1, 2) if spec.get("mlp") else (1,):
            t.update({f"{p}norm{q}": 1 + 0.3 * n(H), f"{p}norm{q}.b": 0.3 * n(H), f"{p}canon{q}": n(H, K) * 0.5 * K ** -0.5,
                      f"{p}hc{q}.in": (1 + 0.5 * n(S)) / S, f"{p}hc{q}.out": 1 + 0.5 * n(S),
                      f"{p}hc{q}.mix": 0.7 * torch.eye(S) + 0.3 / S + 0.15 * n(S, S)})
        t.update({x + "left.q": lin(a["heads"] * a["dim"], H) * 1.5, x + "left.k": lin(a["kv_heads"] * a["dim"], H) * 1.5,
                  x + "left.v": lin(a["kv_heads"] * a["vdim"], H), x + "left.o": lin(H, a["heads"] * a["vdim"])})
        t.update({f"{x}left.{z}.b": n(t[f"{x}left.{z}"].shape[0]) * 0.5 for z in "qkvo"})
        t.update({x + "right.q": lin(r["heads"] * r["dim"], H), x + "right.k": lin(r["heads"] * r["dim"], H),
                  x + "right.v": lin(r["heads"] * r["vdim"], H), x + "right.g": lin(r["heads"] * r["vdim"], H),
                  x + "right.o": lin(H, r["heads"] * r["vdim"])})
        mlp, y = spec.get("mlp"), p + "mlp."
        if mlp and mlp["kind"] == "dense":
            t.update({y + "gate": lin(mlp["ff"], H) * 1.5, y + "up": lin(mlp["ff"], H) * 1.5, y + "down": lin(H, mlp["ff"])})
        elif mlp:
            t[y + "router"] = 4 * lin(mlp["router"]["experts"], H)
            for e in range(mlp["router"]["experts"]):
                ff = mlp["expert"]["ff"]
                t.update({f"{y}e{e}.gate": lin(ff, H), f"{y}e{e}.up": lin(ff, H), f"{y}e{e}.down": lin(H, ff)})
    return {k: v.to(torch.bfloat16).to(dtype) for k, v in t.items()}


def dense_mlp(ff, limit=1.2):
    return dict(kind="dense", ff=ff, limit=limit)


def moe(ff, n_experts, count, keep, top):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=n_experts, groups=dict(count=count, keep=keep), top=top))


def left_spec(heads, kv_heads, dim, vdim, size, pool, scale=None):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale or 1.1 * dim ** -0.5, mask=dict(size=size, pool=pool))


def right_spec(heads, dim, vdim, rot, decay=None, base=9000.0):
    return dict(heads=heads, dim=dim, vdim=vdim, rot=dict(dims=rot, base=base), decay=decay or [1 - 2.0 ** -(2 + 1.5 * i) for i in range(heads)])


def layer_spec(left, right, mlp, scales=(0.7, 1.2)):
    return dict(type="parallel", mlp=mlp, mixer=dict(left=left, right=right, left_scale=scales[0], right_scale=scales[1]))


def model_config(vocab, width, layers, streams=3, taps=4, eps=1e-5, embed_scale=2.0):
    return dict(architecture="Fusolix", vocab=vocab, width=width, layers=layers, norm=dict(eps=eps), embedding=dict(scale=embed_scale),
                streams=streams, canon=dict(taps=taps))


# Configurations of the tests: unequal layers, layers without feed-forward, windows and blocks that do and do not fall on
# page borders (blocks wider than a page or a window too), one and many streams and taps, sizes no tensor-core tile or
# vector access divides, and values that happen to be equal or one.
CONFIGS = {
    "mixed": model_config(160, 96, [
        layer_spec(left_spec(4, 2, 32, 40, 18, 4), right_spec(2, 24, 40, 16), moe(40, 9, 3, 2, 3)),
        layer_spec(left_spec(6, 3, 16, 24, 11, 6), right_spec(3, 32, 16, 32, [0.5, 0.97, 1.0]), None, (1.0, 0.4)),
        layer_spec(left_spec(5, 1, 24, 16, 27, 16), right_spec(4, 16, 32, 4), dense_mlp(136), (0.3, 1.0))]),
    "odd": model_config(101, 75, [
        layer_spec(left_spec(3, 3, 9, 11, 7, 3), right_spec(2, 10, 7, 6), dense_mlp(33, 0.8)),
        layer_spec(left_spec(2, 1, 13, 5, 1, 5), right_spec(1, 34, 13, 2), moe(21, 6, 6, 3, 2)),
        layer_spec(left_spec(4, 2, 8, 3, 19, 23), right_spec(3, 7, 33, 4), moe(17, 4, 1, 1, 1))], streams=1, taps=1, eps=1e-3, embed_scale=1.0),
    "narrow": model_config(128, 64, [
        layer_spec(left_spec(8, 8, 8, 16, 32, 2), right_spec(8, 8, 8, 8), moe(16, 12, 4, 1, 3), (1.0, 1.0)),
        layer_spec(left_spec(1, 1, 64, 8, 2, 1), right_spec(1, 64, 64, 64), dense_mlp(48, 3.0))], streams=5, taps=2),
    "wide": model_config(264, 256, [
        layer_spec(left_spec(12, 2, 64, 64, 50, 8), right_spec(4, 128, 64, 128), moe(96, 16, 4, 2, 5)),
        layer_spec(left_spec(16, 1, 128, 128, 33, 32), right_spec(2, 64, 128, 48), dense_mlp(320)),
        layer_spec(left_spec(4, 4, 40, 72, 21, 10), right_spec(5, 40, 24, 20), moe(64, 8, 2, 2, 4))], streams=2, taps=3),
    "repeated": model_config(96, 128, [
        layer_spec(left_spec(8, 4, 32, 32, 48, 12), right_spec(4, 32, 64, 24), dense_mlp(192)) for _ in range(3)], streams=8, taps=5),
}
