"""The Dobepel design through the library, against the plain implementation in
`tests/plain/dobepel_plain.py`: each mechanism alone (kernels against plain functions), models of few layers
in every cut (whole, token by token, portions down to two tokens, batches of unequal requests, slots and pages
used again), keys far away, at page borders and on either side of the window's and the kept tokens' edges, the
first tokens, long decoding, sizes that make special cases (one key head or as many as query heads, keys and
values of different widths, one head, windows of one key and of none, nothing kept, more kept than a page or
than the prompt, one expert, all experts, no shared expert, no feed-forward, an odd width), and greedy
generation through the library's entry point.

Weights are random; where random weights would hide a fault they are reshaped: the attention's scale is large
so that the softmax is peaked, and slopes of many heads reach far, so that one far key, a window's edge or a
kept token decides a row of logits.
"""
import json
import os

import pytest
import torch

from harness import run_batch, run_chunks, run_tail, run_whole
from plain import dobepel_plain as P
from util import random_tokens

pytestmark = pytest.mark.gpu

FP32_TOL = 2e-4          # of the logits' spread; two float32 computations in different orders of summation
VOCAB = 101
DEV = "cuda"


def _moe(experts=5, top=2, ff=20, shared=28):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def _dense(ff=36):
    return {"kind": "dense", "ff": ff}


def _left(heads=4, kv_heads=2, dim=16, vdim=24, scale=0.4, size=21, keep=5):
    out = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if size:
        out["mask"] = {"size": size, "keep_first": keep}
    return out


def _right(heads=3, dim=12, vdim=20, decay=None):
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay or [0.3, 0.93, 0.998, 0.75, 1.0, 0.0][:heads]}


def _layer(left=None, right=None, mlp="dense"):
    return {"type": "parallel", "mixer": {"left": left or _left(), "right": right or _right()},
            "mlp": _dense() if mlp == "dense" else _moe() if mlp == "moe" else mlp}


def _config(layers, width=40, eps=1e-5, mult=0.7, buckets=53, mul_prev=37, mul_cur=11):
    return {"architecture": "Dobepel", "vocab": VOCAB, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
            "embedding": {"bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}},
            "layers": json.loads(json.dumps(layers))}


def _make(tmp_path, name, config, seed, std=0.12, bias=0.4, change=None):
    """A model folder with random weights for `config` (`change(tensors)` may edit them); returns (folder, plain
    tensors, config)."""
    from picolm_b200.config import config_from_dict
    from picolm_b200.weights import random_tensors, save_safetensors
    cfg = config_from_dict(config)
    tensors = random_tensors(cfg, seed, std=std, norm_std=0.2)
    g = torch.Generator().manual_seed(seed + 1000)
    for n in list(tensors):
        t = tensors[n]
        if n.endswith(".router.b"):
            tensors[n] = (bias * torch.randn(t.shape, generator=g)).to(t.dtype)
        elif n in ("embed", "bigram"):
            tensors[n] = torch.randn(t.shape, generator=g).to(t.dtype)
    if change is not None:
        change(tensors)
    d = str(tmp_path / name)
    os.makedirs(d, exist_ok=True)
    save_safetensors(os.path.join(d, "model.safetensors"), tensors)
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg.to_dict(), f)
    return d, P.read_safetensors(os.path.join(d, "model.safetensors")), cfg.to_dict()


def _plain(tensors, config, tokens, dtype=torch.float64):
    return P.PlainDobepel(config, tensors, dtype).logits(tokens).to(torch.float32)


def _close(got, want, tol=FP32_TOL, what=""):
    err = (got.double() - want.double()).abs().max().item()
    spread = want.double().std().item()
    assert err <= tol * spread, f"{what}: max |diff| {err:.3e} is {err / spread:.2e} of the logits' spread (limit {tol})"


def _engine(d, dtype="float32", max_tokens=64 * 40, **kw):
    from picolm_b200.engine import Engine
    return Engine.from_folder(d, dtype=dtype, max_tokens=max_tokens, **kw)


class _Step:
    """What the kernels read of a step, for sequences that bring `lens` tokens each from position `starts`."""

    def __init__(self, lens, slots, starts=None, tokens=None):
        offs = [0]
        for n in lens:
            offs.append(offs[-1] + n)
        i32 = dict(dtype=torch.int32, device=DEV)
        starts = starts or [0] * len(lens)
        self.n_seqs, self.n_tokens, self.max_new = len(lens), offs[-1], max(lens)
        self.is_decode = all(n == 1 for n in lens)
        self.seq_start, self.seq_slot = torch.tensor(offs, **i32), torch.tensor(slots, **i32)
        self.seq_kv_len = torch.tensor([s + n for s, n in zip(starts, lens)], **i32)
        self.tok_seq = torch.tensor([b for b, n in enumerate(lens) for _ in range(n)], **i32)
        self.tok_pos = torch.tensor([s + i for s, n in zip(starts, lens) for i in range(n)], **i32)
        self.max_position = max(s + n - 1 for s, n in zip(starts, lens))
        if tokens is not None:
            self.tok_ids = torch.tensor(tokens, **i32)


def _in_cuts(lens, cuts):
    """For every step of `cuts` (per sequence a (from, to) or None): the live sequences' numbers and their ranges."""
    for cut in cuts:
        yield [(i, c) for i, c in enumerate(cut) if c is not None]


# ------------------------------------------------------------------------------------------- kernels alone
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("d,buckets,mul_prev,mul_cur", [(40, 53, 37, 11), (42, 1, 5, 3), (256, 97, 1_000_003, 2_000_000_011), (8, 7, 0, 1)])
def test_token_and_pair_rows(dtype, d, buckets, mul_prev, mul_cur):
    """Row of the token plus row of the pair, products that exceed 32 bits among them, over ragged steps that go on from
    a state; slots used again after zeroing start without a token before."""
    from picolm_b200 import ops
    g = torch.Generator().manual_seed(d)
    table = torch.randn(VOCAB, d, generator=g).to(dtype)
    pairs = torch.randn(buckets + 1, d, generator=g).to(dtype)
    seqs = [random_tokens(n, VOCAB, n) for n in (9, 1, 14)]
    seqs[2][0] = seqs[2][1] = 0                       # token 0 as the token before is not "no token before"
    want = [(table[s].double() + pairs[P.pair_rows(s, buckets, mul_prev, mul_cur)].double()) for s in seqs]
    state = torch.full((5, 1), 77, dtype=torch.int32, device=DEV)
    slots = [3, 0, 1]
    for turn in range(2):
        state[slots] = 0
        got = [torch.zeros(len(s), d) for s in seqs]
        for live in _in_cuts(seqs, [[(0, 4), (0, 1), (0, 1)], [(4, 5), None, (1, 13)], [(5, 9), None, (13, 14)]]):
            step = _Step([c[1] - c[0] for _, c in live], [slots[i] for i, _ in live], tokens=[t for i, c in live for t in seqs[i][c[0]:c[1]]])
            x = ops.embed_pair(step, table.to(DEV), pairs.to(DEV), state, mul_prev, mul_cur).cpu()
            o = 0
            for i, c in live:
                got[i][c[0]:c[1]] = x[o:o + c[1] - c[0]]
                o += c[1] - c[0]
        for i in range(3):
            assert (got[i].double() - want[i]).abs().max() < 1e-5, f"sequence {i}, turn {turn}"
        assert state[:, 0].tolist() == [seqs[1][-1] + 1, seqs[2][-1] + 1, 77, seqs[0][-1] + 1, 77]


def _paged(k, v, order, hd, dtype, junk=True):
    """Keys and values [n, G, .] of one sequence in pages of 64 in the order `order`, padded to heads of `hd`; places that
    hold nothing are filled with large numbers."""
    n, G = k.shape[:2]
    pages = torch.full((max(order) + 2, G, 64, hd), 300.0 if junk else 0.0)
    vals = pages.clone()
    for i in range(n):
        pages[order[i // 64], :, i % 64] = 0
        vals[order[i // 64], :, i % 64] = 0
        pages[order[i // 64], :, i % 64, :k.shape[2]] = k[i]
        vals[order[i // 64], :, i % 64, :v.shape[2]] = v[i]
    return pages.to(dtype).to(DEV), vals.to(dtype).to(DEV)


class _KV:
    def __init__(self, k, v, table, window, keep):
        self.k, self.v, self.block_table, self.window, self.keep_first, self.writable = k, v, table, window, keep, True


@pytest.mark.parametrize("how", ["prompt", "portion", "single", "many_ranges"])
@pytest.mark.parametrize("hd,H,G,dtype", [(16, 4, 2, torch.float32), (64, 4, 1, torch.bfloat16), (128, 6, 3, torch.bfloat16),
                                          (48, 20, 1, torch.bfloat16), (80, 3, 3, torch.bfloat16)])
@pytest.mark.parametrize("size,keep", [(1, 0), (21, 5), (64, 64), (65, 70), (130, 1), (70, 300), (None, 0)])
def test_attention_with_slopes_and_kept_tokens(hd, H, G, dtype, size, keep, how):
    """Every attention kernel (CUDA cores, tcgen05 at 64 and 128, mma.sync prompts and decode, with few and with many key
    ranges) with slopes under a window that keeps the first tokens: queries are aimed in turn at the key just inside
    the window, just outside it, the last kept one and the first that is not, so that one token off shows."""
    from picolm_b200 import ops
    T = 300
    g = torch.Generator().manual_seed(hd + (size or 0))
    k, v = torch.randn(T, G, hd, generator=g), torch.randn(T, G, hd, generator=g)
    q = 0.1 * torch.randn(T, H, hd, generator=g)
    slopes = [0.02 * 2.0 ** (-3.0 * h / H) for h in range(H)]
    scale = 8.0 / hd
    for i in range(T):
        w = size or 40
        target = [max(0, i - w + 1), max(0, i - w), max(0, min(i, keep - 1)), min(i, keep)][i % 4]
        q[i] += k[target].repeat_interleave(H // G, dim=0) * 1.5
    q, k, v = (t.to(dtype).double() for t in (q, k, v))

    def exact(size, keep):
        s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(H // G, dim=1)) * scale
        i = torch.arange(T, dtype=torch.float64)
        s = s - torch.tensor(slopes, dtype=torch.float64)[:, None, None] * (i[:, None] - i[None, :])
        s = s.masked_fill(~P.window_mask(T, size, keep), float("-inf"))
        return torch.einsum("hij,jhd->ihd", torch.softmax(s, dim=-1), v.repeat_interleave(H // G, dim=1))

    want = exact(size, keep)
    tol = 2e-5 if dtype == torch.float32 else 0.03
    if size and keep < T:
        wrong = [(size + 1, keep)] + ([(size - 1, keep)] if size > 1 else []) + ([(size, keep + 1)] if size + keep < 290 else []) \
            + ([(size, keep - 1)] if keep and size + keep < 290 else [])
        for s2, k2 in wrong:
            assert (exact(s2, k2) - want).abs().amax(dim=(1, 2)).gt(10 * tol).sum() >= 2, f"{s2}, {k2} would not show"
    order = [4, 1, 5, 2, 3]
    kp, vp = _paged(k.float(), v.float(), order, hd, dtype)
    table = torch.tensor([[0] * 5, order], dtype=torch.int32, device=DEV)
    kv = _KV(kp, vp, table, size, keep if size else 0)
    sl = torch.tensor(slopes, dtype=torch.float32, device=DEV)
    qd = q.to(dtype).to(DEV)

    def run(lo, hi, seq_first):
        n = hi - lo
        # a first sequence of one token on the null page, so that ours starts at an offset
        lens, starts = ([1, n], [0, lo]) if seq_first else ([n], [lo])
        step = _Step(lens, list(range(len(lens))), starts)
        kv.block_table = table if seq_first else table[1:].contiguous()
        rows = torch.cat([qd[:1], qd[lo:hi]]) if seq_first else qd[lo:hi].contiguous()
        return ops.attention(rows, kv, step, G, scale, slopes=sl).float().cpu().view(-1, H, hd)[-n:]

    if how == "prompt":
        got, rng = run(0, T, True), range(T)
    elif how == "portion":
        got, rng = run(149, T, False), range(149, T)
    elif how == "single":
        rng = [0, 1, 4, 5, 20, 21, 63, 64, 65, 100, 128, 129, 150, 191, 192, 200, 255, 256, 299]
        got = torch.cat([run(i, i + 1, False) for i in rng])
    else:
        rng = [0, 64, 130, 299]
        if dtype == torch.float32:
            pytest.skip("the CUDA-core kernel has no key ranges")
        got = []
        for i in rng:
            for splits, scratch in ((3, False), (8, False), (5, True), (11, True)):
                out = ops.attention_decode(qd[i:i + 1].contiguous(), kp, vp, torch.tensor([i], dtype=torch.int32, device=DEV),
                                           torch.tensor([1], dtype=torch.int32, device=DEV), table, G, scale, splits, window=size,
                                           scratch=scratch, keep_first=keep if size else 0, slopes=sl)
                err = (out.float().cpu().view(H, hd).double() - want[i]).abs().max()
                assert err < tol * 4, f"query {i} in {splits} ranges: {err:.2e}"
            got.append(out.float().cpu().view(1, H, hd))
        got = torch.cat(got)
    err = (got.double() - want[list(rng)]).abs().amax(dim=(1, 2))
    assert err.max() < tol * 4, f"query {list(rng)[int(err.argmax())]}: {err.max():.2e}"


def test_attention_with_kept_tokens_and_no_slopes():
    """A window that keeps the first tokens without slopes (the other instance of the tcgen05 kernel)."""
    from picolm_b200 import ops
    T, H, G, hd, size, keep = 260, 4, 2, 64, 40, 70
    g = torch.Generator().manual_seed(1)
    q, k, v = (torch.randn(T, n, hd, generator=g).bfloat16().double() for n in (H, G, G))
    s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(2, dim=1)) * 0.2
    s = s.masked_fill(~P.window_mask(T, size, keep), float("-inf"))
    want = torch.einsum("hij,jhd->ihd", torch.softmax(s, dim=-1), v.repeat_interleave(2, dim=1))
    order = [2, 4, 1, 5, 3]
    kp, vp = _paged(k.float(), v.float(), order, hd, torch.bfloat16)
    kv = _KV(kp, vp, torch.tensor([order], dtype=torch.int32, device=DEV), size, keep)
    got = ops.attention(q.bfloat16().to(DEV), kv, _Step([T], [0]), G, 0.2).float().cpu().view(T, H, hd)
    assert (got.double() - want).abs().max() < 0.05


@pytest.mark.parametrize("dtype,N,P_", [(torch.float32, 12, 20), (torch.float32, 40, 33), (torch.bfloat16, 16, 8), (torch.bfloat16, 64, 72),
                                        (torch.bfloat16, 128, 136), (torch.bfloat16, 80, 64), (torch.bfloat16, 20, 24), (torch.bfloat16, 144, 16)])
@pytest.mark.parametrize("cut", ["whole", "mixed", "single"])
def test_constant_decay_recurrence(dtype, N, P_, cut):
    """The recurrence with SiLU on its inputs over ragged steps, from zero, from a state, in one pass and in segments,
    chunk by chunk on the tensor cores and token by token: outputs and states; decays of 1, 0, next to 1 and in between;
    column slices of a wider matrix; state rows wider than the state."""
    from picolm_b200 import ops
    H = 5
    decay = [0.3, 0.9995, 1.0, 0.0, 0.93]
    lens = [700, 1, 130]
    g = torch.Generator().manual_seed(N + P_)
    cols = 2 * H * N + H * P_
    pad = (-cols) % 8 + 8
    rows = [torch.randn(n, cols + pad, generator=g).to(dtype) for n in lens]
    want, states = [], []
    for r in rows:
        x = P.silu(r[:, :cols].double())
        if dtype == torch.bfloat16:
            x = x.to(dtype).double()
        n = len(x)
        o, S = P.decayed_scan(x[:, :H * N].view(n, H, N), x[:, H * N:2 * H * N].view(n, H, N), x[:, 2 * H * N:].view(n, H, P_),
                              torch.tensor(decay, dtype=torch.float32).double())
        want.append(o.reshape(n, H * P_))
        states.append(S.reshape(-1))
    width = H * N * P_ + 12
    state = torch.full((5, width), 7.0, device=DEV)
    slots = [2, 0, 3]
    dd, powers = torch.tensor(decay, dtype=torch.float32, device=DEV), ops.decay_powers(decay).to(DEV)
    cuts = {"whole": [[(0, 700), (0, 1), (0, 130)]],
            "mixed": [[(0, 290), (0, 1), (0, 2)], [(290, 291), None, (2, 34)], [(291, 570), None, (34, 129)], [(570, 700), None, (129, 130)]],
            "single": [[(0, 660), None, (0, 100)]] + [[(660 + i, 661 + i), (0, 1) if i == 3 else None, (100 + i, 101 + i) if i < 30 else None]
                                                       for i in range(40)]}[cut]
    state[slots] = 0.0
    state[:, H * N * P_:] = 5.0
    got = [torch.zeros(n, H * P_) for n in lens]
    for live in _in_cuts(lens, cuts):
        step = _Step([c[1] - c[0] for _, c in live], [slots[i] for i, _ in live])
        x = torch.cat([rows[i][c[0]:c[1]] for i, c in live]).to(DEV)
        y = ops.decay_scan(x[:, :H * N], x[:, H * N:2 * H * N], x[:, 2 * H * N:cols], dd, powers, state, step, H, N, P_,
                           activation="silu").cpu()
        o = 0
        for i, c in live:
            got[i][c[0]:c[1]] = y[o:o + c[1] - c[0]]
            o += c[1] - c[0]
    # bfloat16: inputs are exact on both sides up to a SiLU that rounds the other way now and then
    tol = 3e-6 if dtype == torch.float32 else 2e-3
    for i in range(3):
        for h in range(H):
            w, o = want[i][:, h * P_:(h + 1) * P_], got[i][:, h * P_:(h + 1) * P_].double()
            assert (o - w).abs().max() < tol * max(w.abs().max().item(), 1e-3), f"sequence {i}, head {h} (decay {decay[h]})"
        S = state[slots[i], :H * N * P_].cpu().double()
        assert (S - states[i]).abs().max() < tol * states[i].abs().max(), f"state of sequence {i}"
    assert (state[[1, 4]][:, :H * N * P_] == 7.0).all() and (state[:, H * N * P_:] == 5.0).all()


def test_long_memory_keeps_its_digits():
    """A decay of 0.99995 over 6,000 tokens in float32: the state stays within float32 rounding of the exact sum."""
    from picolm_b200 import ops
    H, N, P_, T = 1, 16, 16, 6000
    g = torch.Generator().manual_seed(3)
    x = torch.randn(T, 3 * N, generator=g).abs()
    decay = [0.99995]
    d = torch.tensor(decay, dtype=torch.float32).double()
    k, v = P.silu(x[:, N:2 * N].double()), P.silu(x[:, 2 * N:].double())
    w = d ** torch.arange(T - 1, -1, -1, dtype=torch.float64)
    want = torch.einsum("tn,tp->np", k * w[:, None], v)
    state = torch.zeros(2, N * P_, device=DEV)
    xd = x.to(DEV)
    ops.decay_scan(xd[:, :N], xd[:, N:2 * N], xd[:, 2 * N:], d.float().to(DEV), ops.decay_powers(decay).to(DEV), state, _Step([T], [0]),
                   H, N, P_, activation="silu")
    assert ((state[0].view(N, P_).cpu().double() - want) / want).abs().max() < 2e-5


@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("d", [40, 1028, 2048, 5120])
def test_joined_norms_into_the_stream(d, out_dtype):
    """Two results each behind its norm, their mean behind the closing norm with its factor, the add, the opening norm."""
    from picolm_b200 import ops
    g = torch.Generator().manual_seed(d)
    x, a, b = (torch.randn(7, d, generator=g) * s for s in (1.0, 3.0, 0.2))
    ws = [1 + 0.3 * torch.randn(d, generator=g) for _ in range(4)]
    y = 0.5 * (P.rms_norm(a.double(), ws[0].double(), 1e-5) + P.rms_norm(b.double(), ws[1].double(), 1e-4))
    nx = x.double() + P.rms_norm(y, ws[2].double(), 1e-3)
    want = P.rms_norm(nx, ws[3].double(), 1e-2)
    xd = x.to(DEV)
    wd = [w.to(DEV) for w in ws]
    got = ops.joined_post_pre_norm(xd, a.to(DEV), wd[0], 1e-5, b.to(DEV), wd[1], 1e-4, 0.5, wd[2], 1e-3, wd[3], 1e-2, out_dtype)
    assert (xd.cpu().double() - nx).abs().max() < 1e-5
    assert (got.float().cpu().double() - want).abs().max() < (1e-5 if out_dtype == torch.float32 else 2e-2)


@pytest.mark.parametrize("M,K,F,dtype", [(1, 64, 128, torch.bfloat16), (8, 192, 200, torch.bfloat16), (50, 512, 1000, torch.bfloat16),
                                         (8, 64, 38016, torch.bfloat16), (100, 128, 256, torch.bfloat16), (300, 1024, 520, torch.bfloat16),
                                         (1024, 512, 4096, torch.bfloat16), (90, 4096, 256, torch.bfloat16), (640, 2048, 768, torch.bfloat16),
                                         (13, 40, 36, torch.bfloat16), (33, 50, 70, torch.float32)])
def test_product_with_the_exact_gelu(M, K, F, dtype):
    """W_up's product with the exact GELU behind it, in every form the product takes (few rows, their walk over many
    tiles, single CTAs, pairs, K in parts, the stream of stages, the CUDA cores)."""
    from picolm_b200 import ops
    g = torch.Generator().manual_seed(M + F)
    a, w = torch.randn(M, K, generator=g).to(dtype), (1.5 / K ** 0.5 * torch.randn(F, K, generator=g)).to(dtype)
    want = P.gelu_erf(a.double() @ w.double().T)
    got = ops.linear_act(a.to(DEV), w.to(DEV), dtype, "gelu_erf").float().cpu().double()
    assert (got - want).abs().max() < (2e-5 if dtype == torch.float32 else 0.04)
    ops.check_status()


@pytest.mark.parametrize("E,top", [(5, 2), (12, 4), (1, 1), (7, 7), (40, 3)])
def test_router_choice_by_biased_logits(E, top):
    """The largest logits with the router's bias inside them; weights are the softmax over the chosen ones alone, also
    for logits far from zero."""
    from picolm_b200 import ops
    g = torch.Generator().manual_seed(E)
    z, b = 30.0 * torch.randn(50, E, generator=g), 20.0 * torch.randn(E, generator=g)
    ids, weights = P.choose(z.double() + b.double(), top)
    got_ids, got_w, _ = ops.route_topk(z.to(DEV), E, top, b.to(DEV), scores="logits")
    assert (got_ids.cpu() == ids).all()
    assert (got_w.cpu().double() - weights).abs().max() < 1e-5


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("C", [1024, 2052, 6000])
def test_wide_gate_and_norm(dtype, C):
    """The norm over all heads together with its gate, rows wide enough for a block each."""
    from picolm_b200 import ops
    g = torch.Generator().manual_seed(C)
    x, w = torch.randn(9, C, generator=g) * 2, 1 + 0.3 * torch.randn(C, generator=g)
    rows = torch.randn(9, C + 8, generator=g).to(dtype)
    want = P.rms_norm(x.double(), w.double(), 1e-4) * torch.sigmoid(rows[:, 8:].double())
    got = ops.gated_norm(x.to(DEV), dtype, weight=w.to(DEV), eps=1e-4, gate=rows.to(DEV)[:, 8:], gate_mode=ops.GATE_AFTER_NORM,
                         activation="sigmoid")
    assert (got.float().cpu().double() - want).abs().max() < (2e-5 if dtype == torch.float32 else 3e-2)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("D,Dv,hd", [(16, 24, 32), (64, 64, 64), (24, 8, 32)])
def test_heads_into_pages_as_they_are(dtype, D, Dv, hd):
    """A QKV product's rows to queries and pages without anything done to them, padded to the cache's head size."""
    from picolm_b200 import ops
    H, G, lens, starts = 4, 2, [70, 1], [3, 64]
    g = torch.Generator().manual_seed(D)
    cols = H * D + G * (D + Dv)
    wide = torch.randn(71, cols + 24, generator=g).to(dtype).to(DEV)
    kp = torch.full((6, G, 64, hd), 9.0, dtype=dtype, device=DEV)
    vp = kp.clone()
    table = torch.tensor([[3, 1], [4, 2]], dtype=torch.int32, device=DEV)
    step = _Step(lens, [0, 1], starts)
    q = torch.empty(71, H, hd, dtype=dtype, device=DEV)
    ops.qk_norm_rope_store(wide[:, 8:8 + cols], None, None, None, 0.0, q, _KV(kp, vp, table, None, 0), None, step, H, G, D, Dv)
    rows = wide[:, 8:8 + cols].cpu()
    assert (q.cpu()[:, :, :D] == rows[:, :H * D].view(71, H, D)).all() and (q[:, :, D:] == 0).all()
    at = [(0, 3 + i) for i in range(70)] + [(1, 64)]
    written = torch.zeros(6, 64, dtype=torch.bool)
    for t, (b, pos) in enumerate(at):
        page = int(table[b, pos // 64])
        written[page, pos % 64] = True
        assert (kp[page, :, pos % 64, :D].cpu() == rows[t, H * D:(H + G) * D].view(G, D)).all() and (kp[page, :, pos % 64, D:] == 0).all()
        assert (vp[page, :, pos % 64, :Dv].cpu() == rows[t, (H + G) * D:].view(G, Dv)).all() and (vp[page, :, pos % 64, Dv:] == 0).all()
    assert (kp.cpu().permute(0, 2, 1, 3)[~written] == 9.0).all(), "places of other tokens were touched"


# ------------------------------------------------------------------------------------------------- models
MODELS = {
    "dense": ([_layer(), _layer(_left(heads=2, kv_heads=1, dim=24, vdim=8, size=64, keep=64), _right(heads=1, dim=16, vdim=32, decay=[0.97]))], {}),
    "routed": ([_layer(mlp="moe"), _layer(_left(heads=3, kv_heads=3, dim=16, vdim=16, size=65, keep=0), mlp=_moe(experts=3, top=3, shared=None))], {"mult": 0.5}),
    # no window, a window of one key, one that keeps more than a page, one that keeps more than any prompt has; no
    # feed-forward, one expert, a decay of exactly 1 and 0
    "mixed": ([_layer(_left(size=None), _right(heads=6), mlp=None), _layer(_left(heads=1, kv_heads=1, size=1, keep=0), mlp=_moe(experts=1, top=1)),
               _layer(_left(heads=6, kv_heads=2, size=30, keep=70), mlp="moe"), _layer(_left(size=5, keep=500), mlp=None)], {"mult": 1.0}),
    # an odd width, head sizes that are no multiples of anything, one bucket, multipliers of zero and beyond 32 bits
    "odd": ([_layer(_left(heads=3, kv_heads=1, dim=10, vdim=6, size=17, keep=3), _right(heads=2, dim=7, vdim=9), mlp=_dense(30)),
             _layer(_left(heads=2, kv_heads=2, dim=5, vdim=11, size=40, keep=1), _right(heads=1, dim=3, vdim=5, decay=[0.9]), mlp=_moe(experts=4, top=1, ff=13, shared=9))],
            {"width": 42, "buckets": 1, "mul_prev": 0, "mul_cur": 3}),
    "pairs": ([_layer(mlp=None)], {"buckets": 89, "mul_prev": 4_000_000_007, "mul_cur": 3_000_000_019, "mult": 0.25, "eps": 1e-2}),
}


@pytest.mark.parametrize("name", sorted(MODELS))
def test_float32_model_matches_plain_in_every_cut(tmp_path, name):
    """Whole prompts, a prompt and 90 single tokens over a page border, token by token from the first, portions down
    to two tokens, a batch of unequal requests, and the same again on slots and pages that were given back."""
    layers, kw = MODELS[name]
    d, tensors, config = _make(tmp_path, name, _config(layers, **kw), seed=len(name))
    reqs = [random_tokens(n, VOCAB, 100 + i) for i, n in enumerate([230, 40, 1, 129])]
    want = [_plain(tensors, config, t) for t in reqs]
    eng = _engine(d)
    for turn in range(2):
        _close(run_whole(eng, reqs[0]), want[0], what="whole")
        _close(run_tail(eng, reqs[0], tail=90), want[0], what="a prompt and 90 single tokens")
        _close(run_tail(eng, reqs[1], tail=40), want[1], what="token by token from the first")
        _close(run_chunks(eng, reqs[0], [2, 62, 3, 61, 2, 33, 67]), want[0], what="portions")
        outs = run_batch(eng, reqs, [64, 7, 1, 129])
        for i, (got, ref) in enumerate(zip(outs, want)):
            _close(got, ref, what=f"batch, request {i}, turn {turn}")
    eng.cache.check()
    assert eng.cache.slots.used == 0


def test_few_wanted_rows(tmp_path):
    """A step of which few rows are wanted narrows the stream in its last layer, with and without a feed-forward there;
    a step of which nothing is wanted leaves the caches right."""
    for name in ("dense", "routed", "mixed", "odd"):
        layers, kw = MODELS[name]
        d, tensors, config = _make(tmp_path, "few" + name, _config(layers, **kw), seed=31)
        t, u = random_tokens(100, VOCAB, 12), random_tokens(9, VOCAB, 13)
        want_t, want_u = _plain(tensors, config, t), _plain(tensors, config, u)
        eng = _engine(d)
        a, b = eng.new_sequence(), eng.new_sequence()
        got = eng.step([(a, t[:70]), (b, u[:5])], [[69, 3], [4]]).float().cpu()
        _close(got, torch.stack([want_t[69], want_t[3], want_u[4]]), what=f"{name}: three rows of a batch")
        assert eng.step([(a, t[70:90]), (b, u[5:])], [[], []]) is None
        got = eng.step([(a, t[90:])], [[9]]).float().cpu()
        _close(got, want_t[99:100], what=f"{name}: after a step of which nothing was wanted")
        eng.end_sequence(a), eng.end_sequence(b)


def test_pages_before_the_window_go_back_and_kept_ones_stay(tmp_path):
    """Over a long sequence a windowed group holds the kept tokens' pages and the window's, whatever the length; the
    pages that went back serve another sequence meanwhile; logits stay right."""
    layers = [_layer(_left(heads=2, kv_heads=1, size=70, keep=67, scale=1.2), mlp=None), _layer(_left(size=30, keep=0), mlp="moe")]
    d, tensors, config = _make(tmp_path, "pages", _config(layers), seed=6)
    t, u = random_tokens(640, VOCAB, 1), random_tokens(90, VOCAB, 2)
    want_t, want_u = _plain(tensors, config, t), _plain(tensors, config, u)
    eng = _engine(d, max_tokens=64 * 12, max_seq_tokens=700)
    a = eng.new_sequence()
    got = [eng.step([(a, t[:130])], [list(range(130))]).float().cpu()]
    b = None
    for o in range(130, 640):
        if o == 500:
            b = eng.new_sequence()
            _close(eng.step([(b, u)], [list(range(90))]).float().cpu(), want_u, what="another sequence on pages that went back")
        got.append(eng.step([(a, t[o:o + 1])], [[0]]).float().cpu())
        held = [len([p for p in g.pages[a] if p]) for g in eng.cache.kv_groups]
        assert max(held) <= 2 + 3 and min(held) <= 2, held
    _close(torch.cat(got), want_t, what="640 tokens")
    eng.end_sequence(a), eng.end_sequence(b)
    eng.cache.check()


# ------------------------------------------------------------------------------- windows, kept tokens, far keys
@pytest.mark.parametrize("size,keep", [(5, 2), (64, 1), (65, 64), (63, 65), (130, 20)])
def test_window_and_kept_edges_decide_logits_and_are_right(tmp_path, size, keep):
    """With a peaked softmax one key often holds most of a row's weight: a window or a kept range that is one token off
    changes rows' logits by far more than the tolerance (the test first makes sure of that with the plain
    implementation), in prompts, in portions that start around the edges and in single tokens."""
    left = _left(heads=6, kv_heads=1, dim=16, vdim=8, size=size, keep=keep, scale=3.0)
    layers = [_layer(left, mlp=None), _layer(_left(heads=6, kv_heads=2, dim=16, vdim=16, size=size + 3, keep=keep + 2, scale=3.0))]
    d, tensors, config = _make(tmp_path, f"w{size}", _config(layers, mult=1.0), seed=size)
    t = random_tokens(330, VOCAB, size)
    want = _plain(tensors, config, t)
    for key in ("size", "keep_first"):
        for off in (-1, 1):
            other = json.loads(json.dumps(config))
            other["layers"][0]["mixer"]["left"]["mask"][key] += off
            diff = (_plain(tensors, other, t) - want).abs().amax(dim=1) / want.std()
            assert (diff > 50 * FP32_TOL).sum() >= 3, f"the weights do not make {key} show"
    eng = _engine(d)
    _close(run_whole(eng, t), want, what="whole")
    _close(run_tail(eng, t, tail=200), want, what="single tokens over the edges")
    _close(run_chunks(eng, t, [size - 1, 2, size, 3, 330 - 2 * size - 4]), want, what="portions around the edges")
    outs = run_batch(eng, [t, t[:size + keep + 1], t[:3]], [size, size - 1, 1])
    _close(outs[0], want, what="batch")
    _close(outs[1], want[:size + keep + 1], what="batch, a request that just leaves a window")
    eng.cache.check()


def test_far_keys_first_tokens_and_slow_states(tmp_path):
    """Kept tokens ten pages away, a layer that sees everything and decays next to 1: changing token 3 of 660 moves the
    last 60 rows of logits through each of them alone, in prompts, portions and 200 single tokens alike."""
    for name, layers in {
            "kept": [_layer(_left(heads=8, kv_heads=1, size=40, keep=6, scale=2.5), _right(decay=[0.1, 0.2, 0.0]))],
            "all": [_layer(_left(heads=8, kv_heads=2, size=None, scale=2.5), _right(decay=[0.1, 0.2, 0.0]), mlp="moe")],
            "slow": [_layer(_left(size=3, keep=0), _right(decay=[1.0, 0.9999, 0.999]))]}.items():
        d, tensors, config = _make(tmp_path, name, _config(layers, mult=1.0), seed=21)
        t = random_tokens(660, VOCAB, 8)
        want = _plain(tensors, config, t)
        changed = list(t)
        changed[3] = (changed[3] + 1) % VOCAB
        assert (_plain(tensors, config, changed)[-60:] - want[-60:]).abs().max() > 20 * FP32_TOL * want.std(), name
        eng = _engine(d)
        _close(run_whole(eng, t), want, what=f"{name}: whole")
        _close(run_tail(eng, t, tail=200), want, what=f"{name}: 200 single tokens")
        _close(run_chunks(eng, t, [333, 67, 2, 258]), want, what=f"{name}: portions")


def test_the_token_before_is_carried(tmp_path):
    """With the mixers all but silent the pair's row decides a position's logits: the first token of a portion or of a
    step that decodes looks at the last token of the step before, of its own sequence, and a slot that is used again
    starts without one.  (The test first shows that a wrong token before moves the logits.)"""
    d, tensors, config = _make(tmp_path, "before", _config([_layer(mlp=None)], mult=0.05), seed=4)
    t, u = random_tokens(60, VOCAB, 1), random_tokens(60, VOCAB, 2)
    want_t, want_u = _plain(tensors, config, t), _plain(tensors, config, u)
    assert (_plain(tensors, config, [u[9]] + t[10:])[1] - want_t[10]).abs().max() > 1000 * FP32_TOL * want_t.std()
    eng = _engine(d, max_seqs=2)
    for _ in range(3):
        outs = run_batch(eng, [t, u], [10, 33])
        _close(outs[0], want_t, what="first"), _close(outs[1], want_u, what="second")
        _close(run_chunks(eng, u, [1, 1, 2, 20, 36]), want_u, what="portions")


def test_every_part_of_a_layer_shows(tmp_path):
    """Planted mistakes in the plain implementation (a half of the mixer left out or unnormed, slopes or the factor on
    the residual forgotten, the shared expert, the router's bias or the gate left out) move its logits far beyond the
    tolerance that the library meets, so the comparison can see each of them."""
    d, tensors, config = _make(tmp_path, "shows", _config([_layer(mlp="moe"), _layer(mlp="moe")]), seed=14)
    t = random_tokens(90, VOCAB, 5)
    want = _plain(tensors, config, t)
    _close(run_whole(_engine(d), t), want, what="whole")

    def moved(config=config, **edit):
        other = dict(tensors)
        for end, fn in edit.items():
            for n in other:
                if n.endswith(end.replace("__", ".")):
                    other[n] = fn(other[n])
        return (_plain(other, config, t) - want).abs().max() > 100 * FP32_TOL * want.std()

    zero = torch.zeros_like
    assert moved(left__out=zero) and moved(right__out=zero) and moved(shared__down=zero) and moved(router__b=zero) and moved(right__g=zero)
    assert moved(norm1b=torch.ones_like) and moved(norm2b=torch.ones_like) and moved(bigram=zero)
    assert moved(config=dict(config, residual_mult=1.0)) and moved(config=dict(config, norm={"eps": 1e-1}))
    flat = P.head_slopes
    try:
        P.head_slopes = lambda n: [2.0 ** (-8.0 * h / n) for h in range(n)]
        assert moved()
    finally:
        P.head_slopes = flat


# ------------------------------------------------------------------------------------------------ bfloat16
@pytest.mark.parametrize("name", ["wide_heads", "serving"])
def test_bfloat16_follows_the_plain_implementation(tmp_path, name):
    """The serving precision stays within rounding of the exact logits, and its own cuts agree with each other far
    more closely than that.  `wide_heads`: head sizes 64 and 128 (the tcgen05 prompt attention), the recurrence on the
    tensor cores; `serving`: 48 and 80 (the mma.sync kernels), routed layers whose sizes take the tensor-core products."""
    if name == "wide_heads":
        layers = [_layer(_left(heads=4, kv_heads=2, dim=64, vdim=32, size=70, keep=9, scale=0.11), _right(heads=2, dim=64, vdim=64), mlp=_dense(256)),
                  _layer(_left(heads=2, kv_heads=1, dim=96, vdim=128, size=90, keep=66, scale=0.09), _right(heads=1, dim=128, vdim=72, decay=[0.99]), mlp=_moe(experts=6, top=3, ff=64, shared=64))]
    else:
        layers = [_layer(_left(heads=4, kv_heads=2, dim=48, vdim=32, size=33, keep=3, scale=0.2), _right(heads=3, dim=16, vdim=40), mlp=_moe(experts=6, top=3, ff=64, shared=32)),
                  _layer(_left(heads=8, kv_heads=2, dim=72, vdim=72, size=100, keep=20, scale=0.1), _right(heads=2, dim=48, vdim=16), mlp=_dense(200)),
                  _layer(_left(heads=4, kv_heads=4, dim=16, vdim=16, size=None), _right(heads=2, dim=80, vdim=24), mlp=None)]
    d, tensors, config = _make(tmp_path, "bf16" + name, _config(layers, width=128), seed=3, std=0.08)
    t, u = random_tokens(300, VOCAB, 5), random_tokens(31, VOCAB, 6)
    want = _plain(tensors, config, t)
    eng = _engine(d, dtype="bfloat16")
    whole = run_whole(eng, t)
    rel = ((whole - want).double().pow(2).mean().sqrt() / want.double().std()).item()
    assert rel < 0.05, f"bfloat16 logits are {rel:.3f} of the spread away from the exact ones"
    for got in (run_tail(eng, t, tail=120), run_chunks(eng, t, [64, 2, 134, 31, 69]), run_batch(eng, [u, t], [11, 130])[1]):
        rel = ((got - whole).double().pow(2).mean().sqrt() / want.double().std()).item()
        assert rel < 0.03, f"two cuts of the same request differ by {rel:.3f} of the spread"
    eng.cache.check()


@pytest.mark.parametrize("name", ["odd", "mixed"])
def test_bfloat16_at_sizes_the_tensor_cores_refuse(tmp_path, name):
    """An odd width and odd head sizes in the serving precision: other kernels, the same logits within rounding."""
    layers, kw = MODELS[name]
    d, tensors, config = _make(tmp_path, "bf16" + name, _config(layers, **kw), seed=11, std=0.08)
    t = random_tokens(140, VOCAB, 9)
    want = _plain(tensors, config, t)
    eng = _engine(d, dtype="bfloat16")
    whole = run_whole(eng, t)
    rel = ((whole - want).double().pow(2).mean().sqrt() / want.double().std()).item()
    assert rel < 0.05, f"bfloat16 logits are {rel:.3f} of the spread away from the exact ones"
    for got in (run_tail(eng, t, tail=70), run_chunks(eng, t, [64, 2, 74])):
        rel = ((got - whole).double().pow(2).mean().sqrt() / want.double().std()).item()
        assert rel < 0.03, f"two cuts of the same request differ by {rel:.3f} of the spread"


def test_overlapping_launches_see_what_the_ones_before_wrote(tmp_path):
    """Steps whose kernels are queued far ahead of the GPU (a slow recurrence in front of routed layers whose prompts
    take the grouped products): neighbouring launches then overlap, and a value read before the kernel in front has
    written it shows as wrong logits.  The same step again and again, on memory that earlier steps used for other things."""
    layers = [_layer(_left(heads=2, kv_heads=2, dim=48, vdim=8, size=17, keep=20, scale=0.07), _right(heads=1, dim=160, vdim=4, decay=[0.0]),
                     mlp=_moe(experts=3, top=1, ff=128, shared=None)),
              _layer(_left(heads=16, kv_heads=2, dim=64, vdim=16, size=100, keep=0, scale=0.2), _right(heads=3, dim=160, vdim=4),
                     mlp=_moe(experts=3, top=2, ff=64, shared=64)),
              _layer(_left(heads=4, kv_heads=1, dim=96, vdim=16, size=65, keep=100, scale=0.1), _right(heads=4, dim=48, vdim=4, decay=[0.999, 0.6, 0.9, 0.5]),
                     mlp=_dense(100))]
    d, tensors, config = _make(tmp_path, "overlap", _config(layers, width=160, mult=0.5), seed=315, std=0.08, bias=2.0)
    reqs = [random_tokens(n, VOCAB, 70 + i) for i, n in enumerate([1, 160, 100])]
    want = torch.cat([_plain(tensors, config, t) for t in reqs])
    eng = _engine(d, dtype="bfloat16")
    for turn in range(8):
        slots = [eng.new_sequence() for _ in reqs]
        got = eng.step(list(zip(slots, reqs)), [list(range(len(t))) for t in reqs]).float().cpu()
        rel = (got - want).double().pow(2).mean(dim=1).sqrt() / want.double().std()
        assert rel.median() < 0.02, f"turn {turn}: half of the rows are {rel.median().item():.3f} of the spread away"
        for s in slots:
            eng.end_sequence(s)


# ---------------------------------------------------------------------------------------------- generation
GEN = [_layer(_left(size=6, keep=2), mlp="dense"), _layer(_left(heads=2, kv_heads=1, dim=8, vdim=16, size=70, keep=0), mlp="moe"), _layer(mlp=None)]


def _greedy(tensors, config, p, n):
    return P.greedy(P.PlainDobepel(config, tensors), p, n)


def test_greedy_generation_through_the_entry_point(tmp_path):
    """`generate` (batch planning, captured decode steps, sampled ids fed back on the device) gives the plain
    implementation's greedy tokens; more requests than fit one batch, so slots and pages are used again."""
    from picolm_b200.api import generate, model_load
    d, tensors, config = _make(tmp_path, "gen", _config(GEN), seed=13)
    prompts = [random_tokens(n, VOCAB, 30 + i) for i, n in enumerate([5, 70, 1, 19, 33])]
    want = [_greedy(tensors, config, p, 8) for p in prompts]
    eng = model_load(d, dtype="float32", max_batch=2)
    got, stats = generate(eng, prompts, max_tokens=8, temperature=0.0, stop_ids=[], return_stats=True)
    assert got == want
    assert stats.batches == 3 and eng.cache.slots.used == 0
    assert eng.use_graphs, "decode steps of this design are meant to replay captured graphs"
    eng.cache.check()


def test_long_generation(tmp_path):
    """160 tokens from a short prompt, over page borders, windows and kept tokens: every token is the plain
    implementation's choice for the sequence as it stands."""
    from picolm_b200.api import generate, model_load
    d, tensors, config = _make(tmp_path, "long", _config(GEN), seed=19)
    p = random_tokens(7, VOCAB, 3)
    eng = model_load(d, dtype="float32", max_batch=1)
    got = generate(eng, [p], max_tokens=160, temperature=0.0, stop_ids=[])[0]
    logits = _plain(tensors, config, p + got)
    for i, tok in enumerate(got):
        row = logits[len(p) - 1 + i]
        assert row[tok] >= row.max() - FP32_TOL * row.std(), f"token {i}"


def test_bfloat16_generation_with_captured_prompt_steps(tmp_path):
    """In bfloat16 `generate` replays captured graphs for the prompts' step too: every generated token is, by the logits
    of the same prompts launched kernel by kernel, the best or within rounding of it."""
    from picolm_b200.api import generate, model_load
    d, tensors, config = _make(tmp_path, "pgraph", _config(GEN, width=64), seed=23, std=0.08)
    prompts = [random_tokens(n, VOCAB, 60 + i) for i, n in enumerate([70, 9, 200])]
    eng = model_load(d, dtype="bfloat16", max_batch=4)
    assert eng.prompt_graphs, "every part of the design declares itself safe for captured prompt steps"
    plain_eng = _engine(d, dtype="bfloat16", use_graphs=False)
    for turn in range(2):                               # the second time from graphs that were captured before
        got = generate(eng, prompts, max_tokens=6, temperature=0.0, stop_ids=[])
        assert eng._prompt_graphs, "the prompts' step was not replayed from a graph"
        slots = [plain_eng.new_sequence() for _ in prompts]
        logits = plain_eng.step(list(zip(slots, prompts))).float().cpu()
        for step in range(6):
            for i, row in enumerate(logits):
                tok = got[i][step]
                assert row[tok] >= row.max() - 0.03 * row.std(), f"turn {turn}, request {i}, step {step}: graph and single launches disagree"
            logits = plain_eng.step([(s, [got[i][step]]) for i, s in enumerate(slots)]).float().cpu()
        for s in slots:
            plain_eng.end_sequence(s)
    eng.cache.check()


def test_trace_replay_as_a_user_runs_it(tmp_path):
    """bin/trace_run on a Dobepel folder: a batch of unequal prompts, single tokens until the shorter requests end,
    a request alone afterwards in the slot that was given back."""
    from test_gpu_trace_run import Replay
    d, tensors, config = _make(tmp_path, "replay", _config(GEN), seed=17)
    reqs = {f"q{i}": random_tokens(n, VOCAB, 300 + i) for i, n in enumerate([70, 9, 1, 30, 3, 2])}
    ref = {k: _plain(tensors, config, t) for k, t in reqs.items()}
    rp = Replay(d, "float32", str(tmp_path / "out"), max_tokens=128)
    try:
        batch = ["q0", "q1", "q2", "q4", "q5"]
        pos = {"q0": 50, "q1": 4, "q2": 1, "q4": 2, "q5": 1}
        got = rp.send([{"id": k, "tokens": reqs[k][:pos[k]], "want": [pos[k] - 1]} for k in batch],
                      end=[k for k in batch if pos[k] == len(reqs[k])])
        for row, k in enumerate(batch):
            _close(got[row:row + 1], ref[k][pos[k] - 1:pos[k]], what=f"prompt of {k}")
        live = [k for k in batch if pos[k] < len(reqs[k])]
        while live:
            ending = [k for k in live if pos[k] + 1 == len(reqs[k])]
            got = rp.send([{"id": k, "tokens": [reqs[k][pos[k]]], "want": [0]} for k in live], end=ending)
            for row, k in enumerate(live):
                _close(got[row:row + 1], ref[k][pos[k]:pos[k] + 1], what=f"{k} at {pos[k]}")
                pos[k] += 1
            live = [k for k in live if pos[k] < len(reqs[k])]
        got = rp.send([{"id": "again", "tokens": reqs["q3"], "want": [0, 29]}], end=["again"])
        _close(got, ref["q3"][[0, 29]], what="alone, afterwards")
    finally:
        rp.close()


def test_command_line(tmp_path):
    """The library's command line on a Dobepel folder: random weights from a config.json, greedy tokens equal to the
    plain implementation's, sampling, the per-layer benchmark with a row for every layer."""
    import re
    import subprocess
    import sys
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    exe = [sys.executable, os.path.join(root, "bin", "picolm_b200")]
    cfg_path = str(tmp_path / "config.json")
    with open(cfg_path, "w") as f:
        json.dump(_config(GEN), f)
    d = str(tmp_path / "model")
    r = subprocess.run(exe + ["--random-weights", cfg_path, "--out", d, "-s", "3"], capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    tensors = P.read_safetensors(os.path.join(d, "model.safetensors"))
    with open(os.path.join(d, "config.json")) as f:
        config = json.load(f)
    r = subprocess.run(exe + [d, "-p", "5,6,7; 9", "-n", "6", "-t", "0", "--dtype", "float32", "--stop-id", "-1"],
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [[int(t) for t in ln.split()] for ln in r.stdout.strip().splitlines()] == [_greedy(tensors, config, [5, 6, 7], 6),
                                                                                    _greedy(tensors, config, [9], 6)]
    r = subprocess.run(exe + [d, "-p", "5,6,7; 9", "-n", "6", "-t", "0.8", "-k", "40", "--top-p", "0.9", "-s", "5", "--stop-id", "-1"],
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [len(ln.split()) for ln in r.stdout.strip().splitlines()] == [6, 6]
    r = subprocess.run(exe + [d, "-p", "5,6,7,8", "-n", "5", "--benchmark"], capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    rows = [ln.split(",") for ln in r.stderr.splitlines() if re.fullmatch(r"\d+,[0-9.]+,[0-9.]+,[0-9.]+,\d+", ln)]
    assert [int(x[0]) for x in rows] == [0, 1, 2] * 3
    r = subprocess.run(exe + [d, "--list-tensors"], capture_output=True, text=True, timeout=60)
    assert "l1.mlp.router.b\t[5]\tBF16" in r.stdout and "bigram\t[54, 40]\tBF16" in r.stdout and "l2.mix.right.out" in r.stdout
