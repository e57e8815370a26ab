"""A plain, slow implementation of the Dobepel design: one function per
mechanism, written from the design's equations.  It shares no code with
picolm_b200 (it has its own safetensors reader) and runs on the CPU in float64
or float32.

The design in this file's notation.  `x_t = E[token_t] + B[bucket_t]`: beside
the token's row a row of a second table, picked by the pair (token before,
token).  Layers are listed one by one in config.json; a layer is
`x += m post1(mixer(pre1(x)))`, then, if it has a feed-forward,
`x += m post2(ff(pre2(x)))`, with RMS norms on both sides of each sublayer and
one constant m for the whole model.  One kind of mixer, two halves that read the
same rows: softmax attention whose scores fall off linearly with the distance
at a rate of the head's own, over a sliding window and the first few tokens of
the sequence; and a linear recurrence with one constant decay a head behind
SiLU on queries, keys and values, whose concatenated heads are normed, gated
and projected.  Each half's result passes a norm of its own, and their mean is
the mixer's result.  The feed-forward is two maps with the exact GELU between
them, or a mixture of gated experts chosen by biased router logits with a
shared expert beside them.  Final norm, logits against `head`.

`h` is a sublayer's input [T, width] for ONE sequence whose first row is
position 0; weights are stored [out, in] and applied as `W x`.
"""
import json
import math
import struct

import torch

_ST_DTYPES = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "I32": torch.int32}


def read_safetensors(path):
    """name -> tensor, read with nothing but the file format: 8 bytes of length, a JSON table, the data."""
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        table = json.loads(f.read(n))
        data = f.read()
    out = {}
    for name, ent in table.items():
        if name == "__metadata__":
            continue
        a, b = ent["data_offsets"]
        t = torch.frombuffer(bytearray(data[a:b]), dtype=_ST_DTYPES[ent["dtype"]])
        out[name] = t.reshape(ent["shape"]).clone()
    return out


# ----------------------------------------------------------------- small pieces
def silu(z):
    return z * torch.sigmoid(z)


def gelu_erf(z):
    return 0.5 * z * (1.0 + torch.special.erf(z / math.sqrt(2.0)))


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


def pair_rows(tokens, buckets, mul_prev, mul_cur):
    """Row of the pair table for every token: (before * mul_prev + token * mul_cur) mod buckets; the first token of
    a sequence has none before it and takes the extra row at the end."""
    rows = []
    for i, t in enumerate(tokens):
        rows.append(buckets if i == 0 else (int(tokens[i - 1]) * mul_prev + int(t) * mul_cur) % buckets)
    return rows


# ------------------------------------------------------------ softmax attention
def head_slopes(heads):
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


def visible(i, j, size, keep_first):
    """Whether position i sees position j: earlier or itself, and inside the window or among the kept first ones.
    size None: no window, every earlier key."""
    return j <= i and (size is None or i - j < size or j < keep_first)


def window_mask(T, size, keep_first):
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    ok = j <= i
    if size is not None:
        ok = ok & ((i - j < size) | (j < keep_first))
    return ok


def falling_attention(h, w, m, get):
    """Softmax attention with a penalty that grows linearly with the distance."""
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ get(w + ".q").T).view(T, H, D)
    k = (h @ get(w + ".k").T).view(T, G, D)
    v = (h @ get(w + ".v").T).view(T, G, Dv)
    mask = m.get("mask") or {}
    ok = window_mask(T, mask.get("size"), mask.get("keep_first", 0))
    pos = torch.arange(T, dtype=h.dtype)
    dist = pos[:, None] - pos[None, :]
    out = torch.zeros(T, H, Dv, dtype=h.dtype)
    for head, slope in enumerate(head_slopes(H)):
        g = head // (H // G)
        s = (q[:, head] @ k[:, g].T) * m["scale"] - slope * dist
        s = s.masked_fill(~ok, -math.inf)
        out[:, head] = torch.softmax(s, dim=-1) @ v[:, g]
    return out.reshape(T, H * Dv) @ get(w + ".o").T


# -------------------------------------------------------- the linear recurrence
def decayed_scan(q, k, v, decay):
    """q, k [T, H, N], v [T, H, P]: S_t = decay_h S_(t-1) + k_t v_t^T from zero, o_t = S_t^T q_t.  Returns (o, S)."""
    T, H, N = q.shape
    P = v.shape[2]
    d = torch.as_tensor(decay, dtype=q.dtype)[:, None, None]
    S = torch.zeros(H, N, P, dtype=q.dtype)
    out = torch.zeros(T, H, P, dtype=q.dtype)
    for t in range(T):
        S = d * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hn,hnp->hp", q[t], S)
    return out, S


def lightning_attention(h, w, m, eps, get):
    T = h.shape[0]
    H, N, P = m["heads"], m["dim"], m["vdim"]
    q = silu(h @ get(w + ".q").T).view(T, H, N)
    k = silu(h @ get(w + ".k").T).view(T, H, N)
    v = silu(h @ get(w + ".v").T).view(T, H, P)
    o, _ = decayed_scan(q, k, v, m["decay"])
    o = rms_norm(o.reshape(T, H * P), get(w + ".norm"), eps)
    return (o * torch.sigmoid(h @ get(w + ".g").T)) @ get(w + ".o").T


def side_by_side(h, w, m, eps, get):
    left = rms_norm(falling_attention(h, w + ".left", m["left"], get), get(w + ".left.out"), eps)
    right = rms_norm(lightning_attention(h, w + ".right", m["right"], eps, get), get(w + ".right.out"), eps)
    return 0.5 * (left + right)


# ---------------------------------------------------------------- feed-forwards
def two_maps(h, w, get):
    return gelu_erf(h @ get(w + ".up").T) @ get(w + ".down").T


def gated_expert(h, w, get):
    return (silu(h @ get(w + ".gate").T) * (h @ get(w + ".up").T)) @ get(w + ".down").T


def choose(logits, top):
    """The `top` largest logits of every row and the softmax over those alone: (ids, weights) [T, top]."""
    ids = torch.argsort(logits, dim=-1, descending=True, stable=True)[:, :top]
    return ids, torch.softmax(torch.gather(logits, 1, ids), dim=-1)


def mixture(h, w, m, get):
    z = h @ get(w + ".router").T + get(w + ".router.b")
    ids, weights = choose(z, m["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(m["router"]["experts"]):
        for t, slot in torch.nonzero(ids == e).tolist():
            out[t] += weights[t, slot] * gated_expert(h[t:t + 1], f"{w}.e{e}", get)[0]
    if m.get("shared"):
        out = out + gated_expert(h, w + ".shared", get)
    return out


def feed_forward(h, w, m, get):
    return two_maps(h, w, get) if m["kind"] == "dense" else mixture(h, w, m, get)


# ------------------------------------------------------------------- the model
class PlainDobepel:
    """logits(tokens) of one sequence from a model folder's config and tensors; `dtype` float64 or float32."""

    def __init__(self, config, tensors, dtype=torch.float64):
        self.config, self.dtype = config, dtype
        self.tensors = {n: t.to(dtype) for n, t in tensors.items()}

    def embed(self, tokens):
        b = self.config["embedding"]["bigram"]
        rows = pair_rows(tokens, b["buckets"], b["mul_prev"], b["mul_cur"])
        return self.tensors["embed"][list(tokens)] + self.tensors["bigram"][rows]

    def layer(self, i, x):
        c, get = self.config, self.tensors.__getitem__
        layer, w, eps, m = c["layers"][i], f"l{i}", c["norm"]["eps"], c["residual_mult"]
        y = side_by_side(rms_norm(x, get(w + ".norm1"), eps), w + ".mix", layer["mixer"], eps, get)
        x = x + m * rms_norm(y, get(w + ".norm1b"), eps)
        if layer.get("mlp") is not None:
            y = feed_forward(rms_norm(x, get(w + ".norm2"), eps), w + ".mlp", layer["mlp"], get)
            x = x + m * rms_norm(y, get(w + ".norm2b"), eps)
        return x

    def residuals(self, tokens):
        """The stream after every layer, [layers, T, width]."""
        x, out = self.embed(tokens), []
        for i in range(len(self.config["layers"])):
            x = self.layer(i, x)
            out.append(x)
        return torch.stack(out)

    def logits(self, tokens):
        x = self.residuals(tokens)[-1]
        return rms_norm(x, self.tensors["final.norm"], self.config["norm"]["eps"]) @ self.tensors["head"].T


def load(folder, dtype=torch.float64):
    with open(folder + "/config.json", encoding="utf-8") as f:
        config = json.load(f)
    return PlainDobepel(config, read_safetensors(folder + "/model.safetensors"), dtype)


def greedy(model, prompt, n):
    """n tokens of greedy continuation, every step from the whole sequence again."""
    tokens = list(prompt)
    for _ in range(n):
        tokens.append(int(torch.argmax(model.logits(tokens)[-1])))
    return tokens[len(prompt):]
