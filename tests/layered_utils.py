"""Helpers of the layer-by-layer decoders' tests: engines over random weights, feeding schedules, op-level batches on shuffled pages."""
from __future__ import annotations

import torch

import plain_nopelorn as plain
from miles_b200.engine.engine import Engine
from miles_b200.models import nopelorn
from miles_b200.models.config import ModelConfig
from miles_b200.models.convert import load_named_into_model
from miles_b200.models.qwen3 import SHORT_Q, ForwardMeta, RaggedBatch


def engine_for(cfg: dict, weights, device="cpu", dtype=torch.float32, blocks=24, block_size=16, slots=4, context=None, **kw) -> Engine:
    c = ModelConfig.from_hf_config(cfg)
    e = Engine(c, device=device, dtype=dtype, num_blocks=blocks, block_size=block_size, max_running_requests=slots,
               max_context_len=context or blocks * block_size, **kw)
    loaded = load_named_into_model(e.model, list(weights.items()), c, e.ps)
    assert loaded == {n for n, _ in e.model.named_parameters()}
    return e


def tokens_for(cfg: dict, n: int, seed: int = 0) -> list[int]:
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def sizes_for(total: int, pattern) -> list[int]:
    out, i = [], 0
    while total > 0:
        n = min(total, pattern[i % len(pattern)])
        out.append(n)
        total -= n
        i += 1
    return out


def feed_alone(engine: Engine, toks, sizes, rid="x") -> torch.Tensor:
    """Logits of every position of one request fed in pieces of these sizes."""
    r = engine.open_request(rid)
    rows, at = [], 0
    for n in sizes:
        rows.append(engine.feed([(r, toks[at:at + n], list(range(n)))]).cpu())
        at += n
    engine.close_request(rid)
    return torch.cat(rows)


def feed_together(engine: Engine, schedule, sequences) -> dict:
    """`schedule`: steps of (name, tokens) entries; a request is opened at its first entry and closed after its last token."""
    live, at, rows = {}, {n: 0 for n in sequences}, {n: [] for n in sequences}
    for step in schedule:
        entries = []
        for name, n in step:
            if name not in live:
                live[name] = engine.open_request(name)
            n = min(n, len(sequences[name]) - at[name])
            entries.append((live[name], sequences[name][at[name]:at[name] + n], list(range(n))))
            at[name] += n
        out = engine.feed(entries).cpu()
        k = 0
        for (name, _), (_, toks, _) in zip(step, entries):
            rows[name].append(out[k:k + len(toks)])
            k += len(toks)
            if at[name] == len(sequences[name]):
                engine.close_request(name)
                del live[name]
    assert not live
    return {n: torch.cat(r) for n, r in rows.items()}


def random_schedule(lengths: dict, seed: int, together: int = 3) -> list:
    """Steps for `feed_together`: up to `together` requests at a time, pieces of some beside single tokens of others, now and then one
    left out."""
    g = torch.Generator().manual_seed(seed)
    left, schedule, order = dict(lengths), [], list(lengths)
    live: list[str] = []
    while left:
        while len(live) < together and any(n not in live for n in left):
            live.append(next(n for n in order if n in left and n not in live))
        step = []
        for n in live:
            if torch.rand((), generator=g) < 0.85:
                k = int([1, 1, 2, 3, 9, 17, 40][int(torch.randint(0, 7, (), generator=g))])
                step.append((n, min(k, left[n])))
        if not step:
            continue
        for n, k in step:
            left[n] -= k
            if not left[n]:
                del left[n]
                live.remove(n)
        schedule.append(step)
    return schedule


def row_errors(got: torch.Tensor, want: torch.Tensor) -> torch.Tensor:
    """Every row's error relative to the rows' root mean square (means taken off)."""
    got, want = got.double().cpu(), want.double().cpu()
    d = (got - want) - (got - want).mean(-1, keepdim=True)
    return d.square().mean(-1).sqrt() / want.square().mean().sqrt()


def rel(got: torch.Tensor, want: torch.Tensor) -> float:
    """Largest of `row_errors`."""
    return float(row_errors(got, want).max())


# ---- op level: several sequences on shuffled pages, any pieces ---------------------------------------------------------------

class Pages:
    def __init__(self, lengths, block_size=16, device="cpu", seed=0):
        self.bs, self.device = block_size, device
        need = [-(-n // block_size) for n in lengths]
        perm = torch.randperm(sum(need) + 2, generator=torch.Generator().manual_seed(seed)).tolist()
        self.num_blocks = len(perm)
        self.blocks = [[perm.pop() for _ in range(k)] for k in need]
        self.slots = torch.randperm(len(lengths), generator=torch.Generator().manual_seed(seed + 1)).tolist()

    def meta(self, pieces, decode_form=False) -> ForwardMeta:
        """pieces: (sequence, start, end), long ones first.  decode_form: the one-token-per-row form without offsets."""
        assert pieces == sorted(pieces, key=lambda p: p[2] - p[1] <= SHORT_Q)
        pos, slot, seq, cu = [], [], [], [0]
        bt = torch.zeros(len(pieces), max(len(b) for b in self.blocks), dtype=torch.int32)
        for i, (b, s, e) in enumerate(pieces):
            bt[i, :len(self.blocks[b])] = torch.tensor(self.blocks[b], dtype=torch.int32)
            pos += range(s, e)
            slot += [self.blocks[b][p // self.bs] * self.bs + p % self.bs for p in range(s, e)]
            seq += [i] * (e - s)
            cu.append(cu[-1] + e - s)
        n_long = sum(e - s > SHORT_Q for _, s, e in pieces)
        i32 = dict(dtype=torch.int32, device=self.device)
        rg = RaggedBatch() if decode_form else RaggedBatch(
            cu_q=torch.tensor(cu, **i32), token_seq=torch.tensor(seq, **i32), q_lens=[e - s for _, s, e in pieces],
            seq_lens=[e for _, _, e in pieces], n_long=n_long, t_long=cu[n_long])
        return ForwardMeta(positions=torch.tensor(pos, **i32), block_table=bt.to(self.device),
                           slot_mapping=torch.tensor(slot, dtype=torch.int64, device=self.device),
                           state_slots=torch.tensor([self.slots[b] for b, _, _ in pieces], **i32), ragged=rg)


def run_pieces(pages: Pages, inputs, schedule, fn):
    """Run `fn(rows, meta)` step by step over (sequence, n) pieces; returns every sequence's outputs in order.  Steps in which every
    piece is one token use the decode form."""
    at, out = [0] * len(inputs), [[] for _ in inputs]
    for step in schedule:
        pieces = sorted([(b, at[b], min(at[b] + n, len(inputs[b]))) for b, n in step if at[b] < len(inputs[b])],
                        key=lambda p: p[2] - p[1] <= SHORT_Q)
        if not pieces:
            continue
        m = pages.meta(pieces, decode_form=all(e - s == 1 for _, s, e in pieces))
        y = fn(torch.cat([inputs[b][s:e] for b, s, e in pieces]).to(pages.device), m).cpu()
        k = 0
        for b, s, e in pieces:
            out[b].append(y[k:k + e - s])
            k += e - s
            at[b] = e
    return [torch.cat(o) for o in out]


def latent_case(m: dict, T: int, seed=0):
    """Inputs whose projections ARE the layer's input: h = [queries | latent | rotated key part], selection matrices as weights.
    Returns (h [T, ·] bf16-exact, oracle weights with the prefix 'x.')."""
    g = torch.Generator().manual_seed(seed)
    nq, nk = m["heads"] * (m["dim"] + m["rot_dim"]), m["kv_rank"] + m["rot_dim"]
    h = torch.randn(T, nq + nk, generator=g).bfloat16().double()
    eye = torch.eye(nq + nk, dtype=torch.float64)
    r = m["kv_rank"]
    W = {"x.q": eye[:nq], "x.dkv": eye[nq:], "x.dkv.norm": (1 + 0.2 * torch.randn(r, generator=g)).bfloat16().double(),
         "x.uk": (torch.randn(m["heads"] * m["dim"], r, generator=g) / r ** 0.5).bfloat16().double(),
         "x.uv": (torch.randn(m["heads"] * m["vdim"], r, generator=g) / r ** 0.5).bfloat16().double(),
         "x.sink": torch.randn(m["heads"], generator=g).bfloat16().double(), "x.o": torch.eye(m["heads"] * m["vdim"], dtype=torch.float64)}
    return h, W


def point_at(h, W, m, eps, query: int, key: int, strength: float):
    """Make the unrotated query of token `query` parallel to the unrotated key of token `key` in every head."""
    c, _ = plain.latent_of(h[key:key + 1], W, "x.", m, eps)
    k = (c @ W["x.uk"].T).view(m["heads"], m["dim"])
    q = h[query, : m["heads"] * (m["dim"] + m["rot_dim"])].view(m["heads"], -1)
    q[:, : m["dim"]] = (strength * k / k.norm(dim=-1, keepdim=True)).bfloat16().double()
    q[:, m["dim"]:] = 0


def latent_fn(m: dict, W, cache, dtype, device, eps):
    """fn(rows, meta) → attention output through the package's op."""
    from miles_b200.ops import mixers as MX

    spec = nopelorn._mixer("latent_attention", m)
    freq, mag = spec.rotary.table()
    lay = MX.LatentLayout(m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"])
    t = {k: v.to(device=device, dtype=dtype) for k, v in W.items()}
    w_ukv = torch.cat([t["x.uk"], t["x.uv"]]).contiguous()
    freq = torch.tensor(freq, dtype=torch.float64, device=device)
    return lambda x, meta: MX.latent_attention(x.to(dtype), lay, cache, meta, freq=freq, magnitude=mag, scale=spec.scale, window=spec.window,
                                               sink=t["x.sink"], w_ukv=w_ukv, kv_norm=t["x.dkv.norm"], eps=eps)


def latent_cache(m: dict, pages: Pages, dtype):
    from miles_b200.ops import mixers as MX

    lay = MX.LatentLayout(m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"])
    # pages that were used before: what lies outside a sequence's own positions must not matter
    return (50 * torch.randn(pages.num_blocks, pages.bs, lay.pitch, generator=torch.Generator().manual_seed(9))).to(dtype).to(pages.device)
