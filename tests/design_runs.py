"""Shared driver of the tests of designs without a library implementation: an engine over random weights, fed token by
token or in portions, with small pools so that pages and state slots come round again. ``O`` is the design's plain model."""
import torch

from mlxcel_b200.config import ModelConfig
from mlxcel_b200.engine import EngineConfig
from mlxcel_b200.llm import LLM
from mlxcel_b200.models.designs import design_fn


def llm_for(raw, tensors, device, dtype, **ecfg):
    cfg = ModelConfig.from_dict(raw)
    kw = dict(max_batch=4, max_prefill_seqs=4, state_slots=4, block_size=16, num_blocks=48, max_num_batched_tokens=768,
              max_model_len=768, prefix_cache=False, watermark=0.0)
    kw.update(ecfg)
    return LLM(cfg, design_fn(cfg.model_type, "build_{}_weights")(tensors.__getitem__, cfg, dtype, device), EngineConfig(**kw))


def tokens_for(raw, n, seed):
    return torch.randint(0, raw["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def cut(n, sizes):
    """n split into the given sizes, taken in turn."""
    out, i = [], 0
    while n > 0:
        out.append(min(n, sizes[i % len(sizes)]))
        n -= out[-1]
        i += 1
    return out


def run_alone(eng, toks, sizes):
    """Logits [n, vocab] of one sequence fed in portions of the given sizes (all places wanted)."""
    sid, at, out = eng.open_sequence(), 0, []
    for c in cut(len(toks), sizes):
        out.append(eng.feed([(sid, toks[at:at + c], list(range(c)))]).float().cpu())
        at += c
    eng.close_sequence(sid)
    return torch.cat(out)


def run_mixed(eng, seqs, schedule):
    """Several sequences in shared steps. ``schedule``: per step {sequence index: portion}; a sequence that
    is through is closed at once (its pages and slot go to the next)."""
    ids, at, got = {}, {}, {i: [] for i in range(len(seqs))}
    for step in schedule:
        entries, order = [], []
        for i, c in step.items():
            if i not in ids:
                ids[i], at[i] = eng.open_sequence(), 0
            entries.append((ids[i], seqs[i][at[i]:at[i] + c], list(range(c))))
            order.append((i, c))
        lg = eng.feed(entries).float().cpu()
        r = 0
        for i, c in order:
            got[i].append(lg[r:r + c])
            r, at[i] = r + c, at[i] + c
            if at[i] == len(seqs[i]):
                eng.close_sequence(ids[i])
    return [torch.cat(got[i]) for i in range(len(seqs))]


def interleave(lengths, portions, width=4):
    """Schedule over sequences of these lengths: at most ``width`` live, each advancing by its own portions."""
    left, nxt, live, steps, k = list(lengths), 0, [], [], 0
    while nxt < len(lengths) or live:
        while len(live) < width and nxt < len(lengths):
            live.append(nxt)
            nxt += 1
        step = {}
        for i in live:
            if (k + i) % 5 == 3 and len(live) > 1:
                continue                                  # left out of this step
            sizes = portions[i % len(portions)]
            step[i] = min(left[i], sizes[k % len(sizes)])
            left[i] -= step[i]
        live = [i for i in live if left[i]]
        if step:
            steps.append(step)
        k += 1
    return steps


def worst(got, want):
    """Largest root-mean-square difference of a position's logits (means taken off) over the logits' spread."""
    want = want.float()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    return float(d.pow(2).mean(-1).sqrt().max() / (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt())


def _errors(got, want):
    want = want.float()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt()


def bf16_ok(O, raw, tensors, toks, got, want):
    """A bf16 run against what rounding the activations alone causes: the mean error stays near that of
    rounding, and all but a few positions (ill-conditioned ones, where rounding decides a sign) stay within
    three times its largest error."""
    with O.bf16_activations():
        r = _errors(O.forward(raw, tensors, toks).float(), want)
    e = _errors(got, want)
    return float(e.median()) < 1.3 * float(r.median()) + 1e-3 and int((e > 3 * r.max()).sum()) <= max(1, len(toks) // 50)


def oracle_greedy(O, raw, tensors, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(O.forward(raw, tensors, toks)[-1].argmax()))
    return toks[len(prompt):]


# ----------------------------------------------------------------------------- kernels on paged pools
def assert_close(got, want, dtype, f32=2e-5, bf16=1.5e-2):
    """Error of every element relative to its size plus the tensor's root mean square."""
    tol = f32 if dtype == torch.float32 else bf16
    got, want = got.double().cpu(), want.double()
    err = (got - want).abs() / (want.abs() + want.pow(2).mean().sqrt())
    assert torch.isfinite(got).all() and err.max() < tol, float(err.max())


def paged_tables(lens, bs, seed=0):
    """Block tables of sequences of these lengths over a shuffled pool; (tables, blocks in the pool)."""
    need = [-(-n // bs) for n in lens]
    perm = torch.randperm(sum(need) + 3, generator=torch.Generator().manual_seed(seed)).tolist()
    tab, at = torch.zeros(len(lens), max(max(need), 1), dtype=torch.int32), 0
    for s, k in enumerate(need):
        tab[s, :k] = torch.tensor(perm[at:at + k], dtype=torch.int32)
        at += k
    return tab, len(perm)


def fill_pages(pool, tab, s, rows):
    """rows [n, heads, width] as the first n entries of sequence s."""
    bs = pool.shape[2]
    for i in range(rows.shape[0]):
        pool[int(tab[s, i // bs]), :, i % bs] = rows[i].to(pool.dtype)


def bounds(sizes):
    out = [0]
    for n in sizes:
        out.append(out[-1] + n)
    return out
