"""The Laperax design through the library, against the plain implementation in
`tests/plain/laperax_plain.py`: each mechanism alone (kernels against plain functions), models of few layers
in every cut (whole, token by token, portions down to two tokens, batches of unequal requests, slots and pages
used again), keys far away, at page borders and on either side of the window's edge, the first tokens, long
decoding, sizes that make special cases (one key head or as many as query heads, keys and values of different
widths, one head, no rotation and rotations of part of a head, a window of one key and none, one convolution
tap, one expert, all experts, no feed-forward, an odd width), and greedy generation through the library's entry
point.

Weights are random; where random weights would hide a fault they are reshaped: the attention's scale is large
so that the softmax is peaked, and decays lie next to 1, so that one far key, a window's edge or a lost state
decides a row of logits.
"""
import json
import os

import pytest
import torch

from harness import run_batch, run_chunks, run_tail, run_whole
from plain import laperax_plain as P
from util import random_tokens

pytestmark = pytest.mark.gpu

FP32_TOL = 2e-4          # of the logits' spread; two float32 computations in different orders of summation
VOCAB = 101
DEV = "cuda"


def _moe(experts=5, top=2, ff=20, scale=1.7):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}


def _layer(kind, mixer, mlp):
    return {"type": kind, "mixer": {k: v for k, v in mixer.items() if v is not None}, "mlp": _moe() if mlp == "moe" else mlp}


def _ret(heads=3, dim=12, vdim=20, decay=None, rot=(5000.0, 8), mlp="moe"):
    return _layer("retention", {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay or [0.3, 0.93, 0.998, 0.75, 1.0, 0.0][:heads],
                                "rot": {"base": rot[0], "dims": rot[1]} if rot else None}, mlp)


def _att(heads=4, kv_heads=2, dim=16, vdim=24, scale=0.7, size=21, rot=(300.0, 12), mlp="moe"):
    return _layer("attention", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                                "rot": {"base": rot[0], "dims": rot[1]} if rot else None, "mask": {"size": size} if size else None}, mlp)


def _del(heads=4, kv_heads=2, dim=12, vdim=20, conv=3, mlp="moe"):
    return _layer("delta", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, mlp)


def _config(layers, width=40, eps=1e-5, logit_scale=0.4, cap=6.0):
    return {"architecture": "Laperax", "vocab": VOCAB, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale,
            "logit_softcap": cap, "layers": json.loads(json.dumps(layers))}


def _make(tmp_path, name, config, seed, std=0.12, change=None):
    """A model folder with random weights for `config` (`change(tensors)` may edit them); returns (folder, plain
    tensors, config)."""
    from picolm_b200.config import config_from_dict
    from picolm_b200.weights import random_tensors, save_safetensors
    cfg = config_from_dict(config)
    tensors = random_tensors(cfg, seed, std=std, norm_std=0.2)
    g = torch.Generator().manual_seed(seed + 1000)
    for n in list(tensors):
        t = tensors[n]
        if n.endswith(".router"):                             # scores that differ, so that the choice is not close
            tensors[n] = (2.0 / t.shape[1] ** 0.5 * torch.randn(t.shape, generator=g)).to(t.dtype)
        elif n in ("embed", "head"):
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
    return P.PlainLaperax(config, tensors, dtype).logits(tokens).to(torch.float32)


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


def _live(cuts):
    """For every step of `cuts` (per sequence a (from, to) or None): the live sequences' numbers and their ranges."""
    for cut in cuts:
        yield [(i, c) for i, c in enumerate(cut) if c is not None]


def _rotation(dims, base, n):
    """cos and sin of positions 0 .. n - 1 as the kernels take them."""
    from picolm_b200 import ops
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    ang = torch.arange(n, dtype=torch.float64)[:, None] * f[None, :]
    return ops.Rotation(ang.cos().float().to(DEV).contiguous(), ang.sin().float().to(DEV).contiguous(), dims, "half")


# ------------------------------------------------------------------------------------------- kernels alone
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("d,eps", [(40, 1e-5), (43, 0.3), (2048, 1e-6), (16000, 1e-2)])
def test_normed_embedding(dtype, d, eps):
    from picolm_b200 import ops
    g = torch.Generator().manual_seed(d)
    table, w = torch.randn(VOCAB, d, generator=g).to(dtype), (1 + 0.3 * torch.randn(d, generator=g)).to(dtype)
    t = [0, 100, 7, 7, 3]
    got = ops.embed_norm(torch.tensor(t, dtype=torch.int32, device=DEV), table.to(DEV), w.to(DEV), eps).cpu()
    assert got.dtype == torch.float32
    assert (got.double() - P.rms_norm(table[t].double(), w.double(), eps)).abs().max() < 2e-5


@pytest.mark.parametrize("n", [1, 3, 4, 1001, 700_000])
def test_logits_scaled_and_capped(n):
    from picolm_b200 import ops
    g = torch.Generator().manual_seed(n)
    x = torch.randn(n, generator=g) * 40
    x[0] = 1e30
    want = P.squash(x.double() * 0.3, 5.0)
    xd = x.to(DEV)
    assert ops.squash(xd, 0.3, 5.0) is xd and (xd.cpu().double() - want).abs().max() < 2e-6
    y = torch.randn(n + 1, generator=g).to(DEV)[1:]                       # not on a 16-byte boundary
    want = P.squash(y.cpu().double() * 2.0, 0.5)
    assert (ops.squash(y, 2.0, 0.5).cpu().double() - want).abs().max() < 1e-6


@pytest.mark.parametrize("dtype,N,P_,rot", [
    (torch.float32, 12, 20, 8), (torch.float32, 40, 33, 40), (torch.float32, 7, 9, 2), (torch.bfloat16, 16, 8, 16), (torch.bfloat16, 64, 72, 64),
    (torch.bfloat16, 128, 136, 128), (torch.bfloat16, 128, 256, 48), (torch.bfloat16, 80, 64, 32), (torch.bfloat16, 48, 64, 20),
    (torch.bfloat16, 32, 40, 2), (torch.bfloat16, 96, 24, 0), (torch.bfloat16, 20, 24, 12), (torch.bfloat16, 144, 16, 64), (torch.bfloat16, 16, 6, 16)])
@pytest.mark.parametrize("cut", ["whole", "mixed", "single"])
def test_rotated_recurrence(dtype, N, P_, rot, cut):
    """The constant-decay recurrence over rotated queries and scaled rotated keys, in ragged steps that go on from a
    state and from positions far from 0, in one pass and in segments, chunk by chunk on the tensor cores and token by
    token: outputs and states.  In bfloat16 the rows are exact on both sides, so what the products take in two terms
    must show sixteen bits: the tolerance lies well below a bfloat16 rounding of a rotated row."""
    from picolm_b200 import ops
    H, base, k_scale = 5, 900.0, 0.37
    decay = [0.3, 0.9995, 1.0, 0.0, 0.93]
    lens, starts = [700, 1, 130], [0, 77, 1000]
    g = torch.Generator().manual_seed(N + P_ + rot)
    cols = 2 * H * N + H * P_
    pad = (-cols) % 8 + 8
    rows = [torch.randn(n, cols + pad, generator=g).to(dtype) for n in lens]
    want, states = [], []
    for r, s0 in zip(rows, starts):
        x, n = r[:, :cols].double(), len(r)
        q, k = x[:, :H * N].view(n, H, N), x[:, H * N:2 * H * N].view(n, H, N)
        if rot:
            q, k = P.rotate(q, range(s0, s0 + n), rot, base), P.rotate(k, range(s0, s0 + n), rot, base)
        k, v, d64 = k * k_scale, x[:, 2 * H * N:].view(n, H, P_), torch.tensor(decay, dtype=torch.float32).double()
        want.append(P.decayed_scan(q, k, v, d64).reshape(n, H * P_))
        w = d64[:, None] ** torch.arange(n - 1, -1, -1, dtype=torch.float64)
        states.append(torch.einsum("thn,thp,ht->hnp", k, v, w).reshape(-1))
    width = H * N * P_ + 12
    state = torch.full((5, width), 7.0, device=DEV)
    slots = [2, 0, 3]
    rotation = _rotation(rot, base, 1200) if rot else None
    dd, powers = torch.tensor(decay, dtype=torch.float32, device=DEV), ops.decay_powers(decay).to(DEV)
    cuts = {"whole": [[(0, 700), (0, 1), (0, 130)]],
            "mixed": [[(0, 290), (0, 1), (0, 2)], [(290, 291), None, (2, 34)], [(291, 570), None, (34, 129)], [(570, 700), None, (129, 130)]],
            "single": [[(0, 660), None, (0, 100)]] + [[(660 + i, 661 + i), (0, 1) if i == 3 else None, (100 + i, 101 + i) if i < 30 else None]
                                                       for i in range(40)]}[cut]
    state[slots] = 0.0
    state[:, H * N * P_:] = 5.0
    got = [torch.zeros(n, H * P_) for n in lens]
    for live in _live(cuts):
        step = _Step([c[1] - c[0] for _, c in live], [slots[i] for i, _ in live], [starts[i] + c[0] for i, c in live])
        x = torch.cat([rows[i][c[0]:c[1]] for i, c in live]).to(DEV)
        y = ops.decay_scan(x[:, :H * N], x[:, H * N:2 * H * N], x[:, 2 * H * N:cols], dd, powers, state, step, H, N, P_,
                           rotation=rotation, k_scale=k_scale).cpu()
        o = 0
        for i, c in live:
            got[i][c[0]:c[1]] = y[o:o + c[1] - c[0]]
            o += c[1] - c[0]
    tol = 3e-6 if dtype == torch.float32 else 1e-4
    for i in range(3):
        for h in range(H):
            w, o = want[i][:, h * P_:(h + 1) * P_], got[i][:, h * P_:(h + 1) * P_].double()
            assert (o - w).abs().max() < tol * max(w.abs().max().item(), 1e-3), f"sequence {i}, head {h} (decay {decay[h]})"
        S = state[slots[i], :H * N * P_].cpu().double()
        assert (S - states[i]).abs().max() < tol * states[i].abs().max(), f"state of sequence {i}"
    assert (state[[1, 4]][:, :H * N * P_] == 7.0).all() and (state[:, H * N * P_:] == 5.0).all()


def test_rotated_recurrence_refuses_what_it_cannot_do():
    from picolm_b200 import ops
    x = torch.zeros(2, 48, device=DEV)
    dd, powers, state = torch.ones(1, device=DEV), ops.decay_powers([1.0]).to(DEV), torch.zeros(2, 256, device=DEV)

    def run(rotation, **kw):
        return ops.decay_scan(x[:, :16], x[:, 16:32], x[:, 32:], dd, powers, state, _Step([2], [0], [8]), 1, 16, 16, rotation=rotation, **kw)

    run(_rotation(16, 10.0, 10))
    r = _rotation(16, 10.0, 10)
    for rotation, kw in ((_rotation(16, 10.0, 9), {}), (_rotation(18, 10.0, 10), {}), (ops.Rotation(r.cos, r.sin, 16, "adjacent"), {}), (r, {"activation": "silu"})):
        with pytest.raises(ops.KernelError):
            run(rotation, **kw)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("N,Pv,H,hpg", [(12, 20, 4, 2), (32, 64, 3, 3), (64, 40, 2, 1), (100, 128, 2, 2), (200, 24, 1, 1), (1, 5, 2, 1),
                                        (16, 8, 2, 2), (48, 72, 4, 2), (128, 136, 2, 1), (112, 64, 2, 2)])
def test_delta_rule_with_one_decay_a_head(dtype, N, Pv, H, hpg):
    """Unit queries and keys, decays and write strengths, and the recurrence chunk by chunk (in bfloat16 on the tensor
    cores where the sizes allow it) and token by token, from zero and from a state: outputs and states; decays from next to 1
    to next to 0; neighbouring keys that are nearly the same."""
    from picolm_b200 import ops
    G = H // hpg
    lens, slots = [230, 1, 67], [3, 0, 1]
    g = torch.Generator().manual_seed(N + Pv)
    rows = [torch.randn(n, 2 * G * N + H * Pv + 2 * H + 8, generator=g).to(dtype) for n in lens]
    for r in rows:                                         # a key like the one before, over a chunk's border too
        for lo, hi in ((20, 26), (62, 67)):
            r[lo:hi, 4 + G * N:4 + 2 * G * N] = r[lo:lo + 1, 4 + G * N:4 + 2 * G * N].clone()
    a_log = torch.linspace(-9.0, 1.5, H) if H > 1 else torch.tensor([-2.0])
    bias = torch.randn(H, generator=g)

    def parts(r):
        o, out = 4, []
        for n in (G * N, G * N, H * Pv, H, H):
            out.append(r[:, o:o + n])
            o += n
        return out

    want, states = [], []
    for r in rows:
        q, k, v, z, b = (t.double() for t in parts(r))
        n = len(r)
        q, k, v = q.view(n, G, N), k.view(n, G, N), v.view(n, H, Pv)
        q = q / torch.sqrt((q * q).sum(-1, keepdim=True) + 1e-6) * N ** -0.5
        k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
        fade = torch.exp(-torch.exp(a_log.double()) * P.softplus(z + bias.double()))
        heads = [P.delta_rule(q[:, h // hpg], k[:, h // hpg], v[:, h], fade[:, h], torch.sigmoid(b[:, h]), with_state=True) for h in range(H)]
        want.append(torch.cat([o for o, _ in heads], dim=1))
        states.append(torch.stack([S for _, S in heads]).reshape(-1))
    state = torch.zeros(5, H * N * Pv + 4, device=DEV)
    for name, cuts in (("whole", [[(0, 230), (0, 1), (0, 67)]]),
                       ("cut", [[(0, 33), (0, 1), (0, 2)], [(33, 34), None, (2, 40)], [(34, 200), None, (40, 41)]]
                               + [[(i, i + 1), None, (i - 159, i - 158) if i < 226 else None] for i in range(200, 230)])):
        state.zero_()
        got = [torch.zeros(n, H * Pv) for n in lens]
        for live in _live(cuts):
            step = _Step([c[1] - c[0] for _, c in live], [slots[i] for i, _ in live])
            q, k, v, z, b = parts(torch.cat([rows[i][c[0]:c[1]] for i, c in live]).to(DEV))
            qn, kn, qk, decay, beta = ops.delta_prep(q, k, z, b, a_log.to(DEV), bias.to(DEV), 1e-6, N ** -0.5, H, N, heads_per_group=hpg,
                                                     head_decay=True)
            assert decay.shape == (step.n_tokens, H)
            y = ops.delta_scan(qn, kn, qk, decay, beta, v, state[:, :H * N * Pv], step, H, N, Pv, heads_per_group=hpg, head_decay=True).cpu()
            o = 0
            for i, c in live:
                got[i][c[0]:c[1]] = y[o:o + c[1] - c[0]]
                o += c[1] - c[0]
        for i in range(3):
            tol = 2e-5 if dtype == torch.float32 or N % 16 or N > 128 or Pv % 8 else 1e-4
            err = (got[i].double() - want[i]).abs().max()
            assert err < tol * want[i].abs().max(), f"{name}, sequence {i}: {err:.2e}"
            err = (state[slots[i], :H * N * Pv].cpu().double() - states[i]).abs().max()
            assert err < tol * states[i].abs().max(), f"{name}, state of sequence {i}: {err:.2e}"
        assert (state[:, H * N * Pv:] == 0).all() and (state[[2, 4]] == 0).all()


class _KV:
    def __init__(self, k, v, table):
        self.k, self.v, self.block_table, self.window, self.keep_first, self.writable = k, v, table, None, 0, True


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("D,Dv,rot", [(16, 24, 12), (64, 64, 64), (10, 6, 2), (128, 64, 32), (16, 16, 0)])
def test_norm_behind_the_rotation(dtype, D, Dv, rot):
    """Queries and keys into the pages, rotated and then divided by each head's root mean square, the constant in it large
    enough to show; values as they are."""
    from picolm_b200 import ops
    H, G, T, eps = 4, 2, 70, 0.2
    hd = -(-max(D, Dv) // 16) * 16
    g = torch.Generator().manual_seed(D)
    qkv = torch.randn(T, H * D + G * (D + Dv), generator=g)
    pos = list(range(3, 3 + T))
    kp, vp = torch.zeros(4, G, 64, hd, dtype=dtype, device=DEV), torch.zeros(4, G, 64, hd, dtype=dtype, device=DEV)
    table = torch.tensor([[3, 1]], dtype=torch.int32, device=DEV)
    q = torch.empty(T, H, hd, dtype=dtype, device=DEV)
    ones = torch.ones(D, dtype=dtype, device=DEV)
    ops.qk_norm_rope_store(qkv.to(DEV), None, ones, ones, eps, q, _KV(kp, vp, table), _rotation(rot, 50.0, 100) if rot else None,
                           _Step([T], [0], [3]), H, G, D, Dv, per_head=True)

    def unit(x, n):
        x = x.double().view(T, n, D)
        return P.unit_rms(P.rotate(x, pos, rot, 50.0) if rot else x, eps)

    tol = 1e-5 if dtype == torch.float32 else 2e-2
    assert (q.cpu()[:, :, :D].double() - unit(qkv[:, :H * D], H)).abs().max() < tol
    keys = torch.stack([kp[table[0, p // 64], :, p % 64, :D] for p in pos]).cpu().double()
    vals = torch.stack([vp[table[0, p // 64], :, p % 64, :Dv] for p in pos]).cpu().double()
    assert (keys - unit(qkv[:, H * D:(H + G) * D], G)).abs().max() < tol
    assert (vals - qkv[:, (H + G) * D:].double().view(T, G, Dv)).abs().max() < tol


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,group", [(4, 20), (3, 64), (2, 256), (5, 7)])
def test_heads_normed_without_a_weight(dtype, heads, group):
    from picolm_b200 import ops
    C = heads * group
    g = torch.Generator().manual_seed(C)
    x, rows = torch.randn(9, C, generator=g) * 2, torch.randn(9, C + 8, generator=g).to(dtype)
    want = P.unit_rms(x.double().view(9, heads, group), 1e-3).reshape(9, C) * P.silu(rows[:, 8:].double())
    got = ops.gated_norm(x.to(DEV), dtype, eps=1e-3, group=group, gate=rows.to(DEV)[:, 8:], gate_mode=ops.GATE_AFTER_NORM, activation="silu")
    assert (got.float().cpu().double() - want).abs().max() < (2e-5 if dtype == torch.float32 else 5e-2)


@pytest.mark.parametrize("M,K,F,dtype", [(1, 64, 128, torch.bfloat16), (8, 192, 200, torch.bfloat16), (50, 512, 1000, torch.bfloat16),
                                         (100, 256, 512, torch.bfloat16), (300, 2048, 512, torch.bfloat16), (700, 1024, 1536, torch.bfloat16),
                                         (5, 40, 36, torch.bfloat16), (70, 40, 36, torch.float32)])
def test_products_with_a_squared_relu(M, K, F, dtype):
    """The activation in the product's epilogue (skinny, wide, paired and streamed forms) and as a kernel of its own."""
    from picolm_b200 import ops
    g = torch.Generator().manual_seed(M + F)
    a, w = torch.randn(M, K, generator=g).to(dtype), (torch.randn(F, K, generator=g) / K ** 0.5).to(dtype)
    want = torch.clamp(a.double() @ w.double().T, min=0) ** 2
    got = ops.linear_act(a.to(DEV), w.to(DEV), dtype, "relu2").float().cpu().double()
    assert ((got - want).abs() <= (1e-5 if dtype == torch.float32 else 1.2e-2) * (1 + want)).all()


@pytest.mark.parametrize("dtype,T,E,top,d,F", [
    (torch.float32, 9, 5, 2, 40, 20), (torch.float32, 300, 4, 3, 36, 70), (torch.bfloat16, 1, 8, 3, 64, 64), (torch.bfloat16, 8, 6, 2, 192, 96),
    (torch.bfloat16, 33, 3, 3, 128, 200), (torch.bfloat16, 7, 4, 1, 42, 13), (torch.bfloat16, 200, 3, 2, 128, 64), (torch.bfloat16, 300, 2, 2, 64, 72),
    (torch.bfloat16, 500, 5, 2, 200, 136), (torch.bfloat16, 700, 8, 3, 512, 320), (torch.bfloat16, 90, 1, 1, 64, 64)])
def test_experts_without_a_gate(tmp_path, dtype, T, E, top, d, F):
    """The routed feed-forward as the part does it, small tiles and tiles of 128 rows: choice, weights, both products and
    the weighted sum, alone and added to a sublayer's rows into the stream."""
    from picolm_b200.parts.feed_forward import RoutedMLP
    from picolm_b200.runtime import Runtime
    name = {torch.float32: "float32", torch.bfloat16: "bfloat16"}[dtype]
    part = RoutedMLP({"hidden_size": d, "experts": E, "top": top, "expert_size": F, "route_scale": 2.3, "activation": "relu2",
                      "router_name": "router", "expert_prefix": "e", "up_name": "up", "down_name": "down"}, Runtime.create(name, DEV))
    g = torch.Generator().manual_seed(T + F)
    tensors = {n: (torch.randn(ws.shape, generator=g) * (3.0 if n == "router" else 1.5) / ws.shape[1] ** 0.5).to(dtype)
               for n, ws in part.weight_specs().items()}
    assert set(tensors) == {"router"} | {f"e{e}.{w}" for e in range(E) for w in ("up", "down")}
    part.load({n: t.to(DEV) for n, t in tensors.items()})
    h = torch.randn(T, d, generator=g).to(dtype)
    get = {f"w.{n}": t.double() for n, t in tensors.items()}.__getitem__
    want = P.mixture(h.double(), "w", _moe(E, top, F, 2.3), get)
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    got = part.forward(h.to(DEV), None).cpu().double()
    assert (got - want).abs().max() < tol * want.abs().max()
    x, add = torch.randn(T, d, generator=g), torch.randn(T, d, generator=g)
    xd = x.to(DEV)
    part.forward(h.to(DEV), None, add=add.to(DEV), into=xd)
    assert (xd.cpu().double() - (x.double() + add.double() + want)).abs().max() < tol * want.abs().max()


# ------------------------------------------------------------------------------------------------- models
MODELS = {
    "retention": ([_ret(), _ret(heads=1, dim=16, vdim=32, decay=[0.97], rot=(100.0, 16), mlp=_moe(3, 3, 12, 0.6)), _ret(rot=None)], {}),
    "attention": ([_att(), _att(heads=3, kv_heads=3, dim=16, vdim=16, size=65, rot=(10.0, 2)), _att(heads=2, kv_heads=1, dim=24, vdim=8, size=64, rot=(1e6, 24), mlp=_moe(1, 1))], {"eps": 1e-2}),
    "delta": ([_del(), _del(heads=3, kv_heads=1, dim=8, vdim=16, conv=1), _del(heads=2, kv_heads=2, dim=40, vdim=8, conv=5, mlp=_moe(4, 1))], {}),
    # every mixer, with and without a feed-forward; no window, a window of one key, no rotation; decays of exactly 1 and 0
    "mixed": ([_att(size=None, rot=None, mlp=None), _del(mlp=None), _ret(heads=6, mlp=None), _att(heads=1, kv_heads=1, size=1), _ret(), _del()],
              {"logit_scale": 1.0, "cap": 3.0}),
    # an odd width, sizes that are no multiples of anything
    "odd": ([_ret(heads=2, dim=7, vdim=9, rot=(50.0, 6), mlp=_moe(4, 3, 13)), _att(heads=3, kv_heads=1, dim=10, vdim=6, size=17, rot=(70.0, 10)),
             _del(heads=3, kv_heads=3, dim=5, vdim=11, conv=2, mlp=_moe(7, 5, 9)), _att(heads=2, kv_heads=2, dim=5, vdim=11, size=40, rot=(9.0, 4))],
            {"width": 42, "logit_scale": 2.0, "cap": 40.0}),
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
    """A step of which few rows are wanted narrows the stream in its last layer (and the norm's rows that the feed-forward
    shares with the mixer), with and without a feed-forward there; a step of which nothing is wanted leaves the caches right."""
    for name in sorted(MODELS) + ["no_ff"]:
        layers, kw = MODELS[name] if name in MODELS else ([_ret(), _del(mlp=None)], {})
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


def test_pages_before_the_window_go_back(tmp_path):
    """Over a long sequence a windowed layer holds the window's pages, whatever the length; the pages that went back serve
    another sequence meanwhile; logits stay right."""
    layers = [_att(heads=2, kv_heads=1, size=70, scale=1.5, mlp=None), _ret(), _att(size=30)]
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
        assert max(held) <= 3 and min(held) <= 2, held
    _close(torch.cat(got), want_t, what="640 tokens")
    eng.end_sequence(a), eng.end_sequence(b)
    eng.cache.check()


# ------------------------------------------------------------------------------- windows, far keys, slow states
@pytest.mark.parametrize("size", [1, 5, 63, 64, 65, 130])
def test_window_edges_decide_logits_and_are_right(tmp_path, size):
    """With a peaked softmax one key often holds most of a row's weight: a window that is one token off changes rows'
    logits by far more than the tolerance (the test first makes sure of that with the plain implementation), in prompts, in
    portions that start around the edge and in single tokens."""
    layers = [_att(heads=6, kv_heads=1, dim=16, vdim=8, size=size, scale=1.2, mlp=None), _att(heads=6, kv_heads=2, dim=16, vdim=16, size=size + 3, scale=1.2)]
    d, tensors, config = _make(tmp_path, f"w{size}", _config(layers), seed=size)
    t = random_tokens(330, VOCAB, size)
    want = _plain(tensors, config, t)
    for off in (-1, 1):
        if size + off < 1:
            continue
        other = json.loads(json.dumps(config))
        other["layers"][0]["mixer"]["mask"]["size"] += off
        diff = (_plain(tensors, other, t) - want).abs().amax(dim=1) / want.std()
        assert (diff > 50 * FP32_TOL).sum() >= 3, "the weights do not make the window's edge show"
    eng = _engine(d)
    _close(run_whole(eng, t), want, what="whole")
    _close(run_tail(eng, t, tail=200), want, what="single tokens over the edges")
    _close(run_chunks(eng, t, [size + 1, 2, size, 3, 330 - 2 * size - 6]), want, what="portions around the edges")
    outs = run_batch(eng, [t, t[:size + 6], t[:3]], [size, size + 1, 1])
    _close(outs[0], want, what="batch")
    _close(outs[1], want[:size + 6], what="batch, a request that just leaves a window")
    eng.cache.check()


def test_far_keys_first_tokens_and_slow_states(tmp_path):
    """A layer that sees everything, decays next to 1 and a delta rule that hardly fades: changing token 3 of 660 moves the
    last 60 rows of logits through each of them alone, in prompts, portions and 200 single tokens alike."""

    def slow(tensors):
        for n in tensors:
            if n.endswith("A_log"):
                tensors[n].fill_(-9.0)
            elif n.endswith(".mix.b"):
                tensors[n].mul_(0.2)

    for name, layers in {"all": [_att(heads=8, kv_heads=2, size=None, scale=1.2)], "slow": [_ret(decay=[1.0, 0.9999, 0.999])],
                         "delta": [_del(dim=24, heads=2, kv_heads=1)]}.items():
        d, tensors, config = _make(tmp_path, name, _config(layers), seed=21, change=slow)
        t = random_tokens(660, VOCAB, 8)
        want = _plain(tensors, config, t)
        changed = list(t)
        changed[3] = (changed[3] + 1) % VOCAB
        assert (_plain(tensors, config, changed)[-60:] - want[-60:]).abs().max() > 20 * FP32_TOL * want.std(), name
        eng = _engine(d)
        _close(run_whole(eng, t), want, what=f"{name}: whole")
        _close(run_tail(eng, t, tail=200), want, what=f"{name}: 200 single tokens")
        _close(run_chunks(eng, t, [333, 67, 2, 258]), want, what=f"{name}: portions")


def test_every_part_of_a_layer_shows(tmp_path):
    """Planted mistakes in the plain implementation (a gate, a norm, a convolution or a scale left out, the norm of queries
    and keys or the rotation forgotten) move its logits far beyond the tolerance that the library meets, so the
    comparison can see each of them."""
    d, tensors, config = _make(tmp_path, "shows", _config([_ret(), _att(), _del(), _ret(mlp=None)], eps=1e-3), seed=14)
    t = random_tokens(90, VOCAB, 5)
    want = _plain(tensors, config, t)
    _close(run_whole(_engine(d), t), want, what="whole")

    def moved(config=config, **edit):
        other = dict(tensors)
        for end, fn in edit.items():
            hit = [n for n in other if n.endswith(end.replace("__", "."))]
            assert hit, end
            for n in hit:
                other[n] = fn(other[n])
        return (_plain(other, config, t) - want).abs().max() > 50 * FP32_TOL * want.std()

    zero, one = torch.zeros_like, torch.ones_like
    last_tap = lambda w: torch.cat([torch.zeros_like(w[:, 1:]), torch.ones_like(w[:, :1])], dim=1)        # noqa: E731
    assert moved(l0__mix__g=zero) and moved(l2__mix__g=zero) and moved(l2__mix__b=zero) and moved(l2__mix__a=zero)
    assert moved(A_log=zero) and moved(dt_bias=zero) and moved(l2__mix__norm=one) and moved(norm1=one) and moved(embed__norm=one)
    assert moved(q__conv=last_tap) and moved(v__conv=last_tap) and moved(router=zero) and moved(final__norm=one)
    for path, value in ((("logit_scale",), 0.5), (("logit_softcap",), 7.0), (("norm", "eps"), 0.1), (("layers", 0, "mixer", "decay", 1), 0.9),
                        (("layers", 0, "mixer", "rot", "dims"), 6), (("layers", 0, "mixer", "rot", "base"), 6000.0),
                        (("layers", 1, "mixer", "rot", "dims"), 10), (("layers", 1, "mixer", "scale"), 0.6),
                        (("layers", 2, "mlp", "router", "scale"), 1.6), (("layers", 2, "mlp", "router", "top"), 1)):
        other = json.loads(json.dumps(config))
        node = other
        for key in path[:-1]:
            node = node[key]
        node[path[-1]] = value
        assert moved(config=other), path
    unit, rotate = P.unit_rms, P.rotate
    try:
        P.unit_rms = lambda x, eps: x if x.shape[-1] == 16 else unit(x, eps)                # the attention's heads alone
        assert moved()
        P.unit_rms = unit
        P.rotate = lambda x, positions, dims, base: rotate(x, [p + 1 for p in positions], dims, base) if x.shape[1] == 2 else rotate(x, positions, dims, base)
        assert moved()                                                                          # keys one position off
    finally:
        P.unit_rms, P.rotate = unit, rotate


# ------------------------------------------------------------------------------------------------ bfloat16
@pytest.mark.parametrize("name", ["wide_heads", "serving"])
def test_bfloat16_follows_the_plain_implementation(tmp_path, name):
    """The serving precision stays within rounding of the exact logits, and its own cuts agree with each other far
    more closely than that.  `wide_heads`: head sizes 64 and 128 (the tcgen05 prompt attention), the recurrences on the
    tensor cores; `serving`: 48 and 80 (the mma.sync kernels); routed layers whose sizes take the tensor-core products."""
    if name == "wide_heads":
        layers = [_att(heads=4, kv_heads=2, dim=64, vdim=32, size=70, scale=0.11, rot=(1e4, 32), mlp=_moe(3, 2, 96)),
                  _ret(heads=2, dim=128, vdim=72, rot=(1e4, 128), mlp=_moe(2, 1, 128)), _del(heads=2, kv_heads=1, dim=64, vdim=128, conv=4, mlp=_moe(6, 3, 64)),
                  _att(heads=2, kv_heads=1, dim=96, vdim=128, size=90, scale=0.09, rot=(1e3, 96), mlp=None)]
    else:
        layers = [_ret(heads=3, dim=16, vdim=40, rot=(1e3, 12), mlp=_moe(6, 3, 64)), _att(heads=4, kv_heads=2, dim=48, vdim=32, size=33, scale=0.2, rot=(1e3, 8)),
                  _del(heads=4, kv_heads=4, dim=32, vdim=48, conv=2, mlp=_moe(2, 2, 72)), _att(heads=8, kv_heads=2, dim=72, vdim=72, size=None, scale=0.1, rot=None),
                  _ret(heads=2, dim=80, vdim=24, rot=None, mlp=None)]
    d, tensors, config = _make(tmp_path, "bf16" + name, _config(layers, width=128, cap=30.0), seed=3, std=0.08)
    t, u = random_tokens(300, VOCAB, 5), random_tokens(31, VOCAB, 6)
    want = _plain(tensors, config, t)
    eng = _engine(d, dtype="bfloat16")
    whole = run_whole(eng, t)

    def apart(x, y):                                        # rows where a close choice of experts fell the other way count little
        return ((x - y).double().pow(2).mean(dim=1).sqrt() / want.double().std()).median().item()

    assert apart(whole, want) < 0.05, f"bfloat16 logits are {apart(whole, want):.3f} of the spread away from the exact ones"
    for got in (run_tail(eng, t, tail=120), run_chunks(eng, t, [64, 2, 134, 31, 69]), run_batch(eng, [u, t], [11, 130])[1]):
        assert apart(got, whole) < 0.03, f"two cuts of the same request differ by {apart(got, whole):.3f} of the spread"
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

    def apart(x, y):
        return ((x - y).double().pow(2).mean(dim=1).sqrt() / want.double().std()).median().item()

    assert apart(whole, want) < 0.05, f"bfloat16 logits are {apart(whole, want):.3f} of the spread away from the exact ones"
    for got in (run_tail(eng, t, tail=70), run_chunks(eng, t, [64, 2, 74])):
        assert apart(got, whole) < 0.03, f"two cuts of the same request differ by {apart(got, whole):.3f} of the spread"


def test_overlapping_launches_see_what_the_ones_before_wrote(tmp_path):
    """Steps whose kernels are queued far ahead of the GPU (a slow recurrence in front of routed layers whose prompts
    take the grouped products): neighbouring launches then overlap, and a value read before the kernel in front has
    written it shows as wrong logits.  The same step again and again, on memory that earlier steps used for other things."""
    layers = [_ret(heads=1, dim=160, vdim=4, decay=[0.0], rot=(1e4, 160), mlp=_moe(3, 1, 128)), _del(heads=2, kv_heads=1, dim=200, vdim=8, mlp=_moe(3, 2, 64)),
              _att(heads=16, kv_heads=2, dim=64, vdim=16, size=100, scale=0.2, mlp=_moe(2, 2, 64)), _ret(heads=4, dim=48, vdim=8, decay=[0.999, 0.6, 0.9, 0.5], mlp=_moe(3, 1, 96))]
    d, tensors, config = _make(tmp_path, "overlap", _config(layers, width=160), seed=315, std=0.08)
    reqs = [random_tokens(n, VOCAB, 70 + i) for i, n in enumerate([1, 160, 100])]
    want = torch.cat([_plain(tensors, config, t) for t in reqs])
    eng = _engine(d, dtype="bfloat16")
    for turn in range(8):
        slots = [eng.new_sequence() for _ in reqs]
        got = eng.step(list(zip(slots, reqs)), [list(range(len(t))) for t in reqs]).float().cpu()
        rel = (got - want).double().pow(2).mean(dim=1).sqrt() / want.double().std()
        assert rel.median() < 0.03, f"turn {turn}: half of the rows are {rel.median().item():.3f} of the spread away"
        for s in slots:
            eng.end_sequence(s)


# ---------------------------------------------------------------------------------------------- generation
GEN = [_ret(), _att(heads=2, kv_heads=1, dim=8, vdim=16, size=6, rot=(100.0, 8)), _del(), _att(size=70, mlp=None)]


def _greedy(tensors, config, p, n):
    return P.greedy(P.PlainLaperax(config, tensors), p, n)


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
    """160 tokens from a short prompt, over page borders and windows: every token is the plain implementation's choice for
    the sequence as it stands."""
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
    layers = [_ret(dim=16, vdim=24, rot=(5000.0, 16)), _att(heads=2, kv_heads=1, dim=8, vdim=16, size=6, rot=(100.0, 8)), _del(dim=32), _att(size=70, mlp=None)]
    d, tensors, config = _make(tmp_path, "pgraph", _config(layers, width=64), seed=23, std=0.08)
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
    """bin/trace_run on a Laperax folder: a batch of unequal prompts, single tokens until the shorter requests end,
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
    """The library's command line on a Laperax folder: random weights from a config.json, greedy tokens equal to the
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
    assert [int(x[0]) for x in rows] == [0, 1, 2, 3] * 3
    r = subprocess.run(exe + [d, "--list-tensors"], capture_output=True, text=True, timeout=60)
    assert "l1.mlp.router\t[5, 40]\tBF16" in r.stdout and "embed.norm\t[40]\tBF16" in r.stdout and "l2.mix.dt_bias\t[4]" in r.stdout
