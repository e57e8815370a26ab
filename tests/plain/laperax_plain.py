"""A plain, slow implementation of the Laperax design: one function per
mechanism, written from the design's equations.  It shares no code with
picolm_b200 (it has its own safetensors reader) and runs on the CPU in float64
or float32.

The design in this file's notation.  The stream begins as a norm of the token's
row.  Layers are listed one by one in config.json; a layer has one norm, whose
rows both of its sublayers read: `h = norm(x)`, `x += mixer(h) + ff(h)`, the
second term only where the layer has a feed-forward.  Three kinds of mixer: a
linear recurrence with one constant decay a head over rotated queries and keys
("retention"), softmax attention over a sliding window whose rotated queries
and keys have a root mean square of one ("attention"), and a delta rule whose
state fades by one factor a head and token ("delta").  The feed-forward is a
mixture of ungated experts with a squared ReLU, weighted by normalised sigmoid
scores.  Final norm, then logits, scaled and squashed by a tanh.

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


def softplus(z):
    return torch.where(z > 30, z, torch.log1p(torch.exp(torch.clamp(z, max=30))))


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


def squash(z, cap):
    return cap * torch.tanh(z / cap)


def rotate(x, positions, dims, base):
    """x [T, heads, size]: component i < dims/2 of every head is paired with component i + dims/2 and the pair is
    turned by position * base^(-2i/dims); components from `dims` on stay."""
    half = dims // 2
    freq = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64)
    ang = torch.as_tensor(positions, dtype=torch.float64)[:, None] * freq[None, :]
    c, s = ang.cos().to(x.dtype)[:, None, :], ang.sin().to(x.dtype)[:, None, :]
    out = x.clone()
    u, v = x[..., :half], x[..., half:dims]
    out[..., :half] = u * c - v * s
    out[..., half:dims] = v * c + u * s
    return out


def short_conv(x, w):
    """Per channel: out[t] = sum_j w[:, j] x[t - (taps - 1) + j], zeros before the first row."""
    T, taps = x.shape[0], w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x])
    out = torch.zeros_like(x)
    for j in range(taps):
        out = out + padded[j:j + T] * w[:, j]
    return out


# -------------------------------------------------------------------- retention
def decayed_scan(q, k, v, decay):
    """q, k [T, H, N], v [T, H, P]: S_t = decay_h S_(t-1) + k_t v_t^T from zero, o_t = S_t^T q_t."""
    T, H, N = q.shape
    P = v.shape[2]
    d = torch.as_tensor(decay, dtype=q.dtype)[:, None, None]
    S = torch.zeros(H, N, P, dtype=q.dtype)
    out = torch.zeros(T, H, P, dtype=q.dtype)
    for t in range(T):
        S = d * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hn,hnp->hp", q[t], S)
    return out


def retention(h, w, m, eps, get):
    T = h.shape[0]
    H, N, P = m["heads"], m["dim"], m["vdim"]
    q = (h @ get(w + ".q").T).view(T, H, N)
    k = (h @ get(w + ".k").T).view(T, H, N)
    v = (h @ get(w + ".v").T).view(T, H, P)
    if m.get("rot"):
        q = rotate(q, range(T), m["rot"]["dims"], m["rot"]["base"])
        k = rotate(k, range(T), m["rot"]["dims"], m["rot"]["base"])
    o = decayed_scan(q, k * N ** -0.5, v, m["decay"])
    o = unit_rms(o, eps).reshape(T, H * P)
    return (o * silu(h @ get(w + ".g").T)) @ get(w + ".o").T


# ------------------------------------------------------------ softmax attention
def window_mask(T, size):
    """[T, T]: whether position i (row) sees position j: not a later one and fewer than `size` positions back
    (None: any earlier one)."""
    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (back >= 0) if size is None else (back >= 0) & (back < size)


def unit_attention(h, w, m, eps, get):
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ get(w + ".q").T).view(T, H, D)
    k = (h @ get(w + ".k").T).view(T, G, D)
    v = (h @ get(w + ".v").T).view(T, G, Dv)
    if m.get("rot"):
        q = rotate(q, range(T), m["rot"]["dims"], m["rot"]["base"])
        k = rotate(k, range(T), m["rot"]["dims"], m["rot"]["base"])
    q, k = unit_rms(q, eps), unit_rms(k, eps)
    ok = window_mask(T, m["mask"]["size"] if m.get("mask") else None)
    out = torch.zeros(T, H, Dv, dtype=h.dtype)
    for head in range(H):
        g = head // (H // G)
        s = ((q[:, head] @ k[:, g].T) * m["scale"]).masked_fill(~ok, -math.inf)
        out[:, head] = torch.softmax(s, dim=-1) @ v[:, g]
    return out.reshape(T, H * Dv) @ get(w + ".o").T


# ------------------------------------------------------------------- delta rule
def delta_rule(q, k, v, g, beta, with_state=False):
    """One head.  q, k [T, N], v [T, P], g, beta [T]: S <- g_t S; u = beta_t (v_t - S^T k_t); S <- S + k_t u^T;
    o_t = S^T q_t.  Returns o [T, P] (and the last S)."""
    T, N = k.shape
    S = torch.zeros(N, v.shape[1], dtype=q.dtype)
    out = torch.zeros(T, v.shape[1], dtype=q.dtype)
    for t in range(T):
        S = g[t] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + torch.outer(k[t], u)
        out[t] = S.T @ q[t]
    return (out, S) if with_state else out


def fading_delta(h, w, m, eps, get):
    T = h.shape[0]
    H, G, N, P = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(short_conv(h @ get(f"{w}.{n}").T, get(f"{w}.{n}.conv"))) for n in "qkv")
    q, k, v = q.view(T, G, N), k.view(T, G, N), v.view(T, H, P)
    q = q / torch.sqrt((q * q).sum(dim=-1, keepdim=True) + 1e-6) * N ** -0.5
    k = k / torch.sqrt((k * k).sum(dim=-1, keepdim=True) + 1e-6)
    beta = torch.sigmoid(h @ get(w + ".b").T)
    g = torch.exp(-torch.exp(get(w + ".A_log")) * softplus(h @ get(w + ".a").T + get(w + ".dt_bias")))
    gate = silu(h @ get(w + ".g").T).view(T, H, P)
    heads = []
    for head in range(H):
        src = head // (H // G)
        o = delta_rule(q[:, src], k[:, src], v[:, head], g[:, head], beta[:, head])
        heads.append(rms_norm(o, get(w + ".norm"), eps) * gate[:, head])
    return torch.cat(heads, dim=-1) @ get(w + ".o").T


MIXERS = {"retention": retention, "attention": unit_attention, "delta": fading_delta}


# ----------------------------------------------------------------- feed-forward
def square_expert(h, w, get):
    return torch.clamp(h @ get(w + ".up").T, min=0) ** 2 @ get(w + ".down").T


def choose(logits, top, scale):
    """The `top` largest sigmoid scores of every row, divided by their sum and times `scale`: (ids, weights) [T, top]."""
    s = torch.sigmoid(logits)
    ids = torch.argsort(s, dim=-1, descending=True, stable=True)[:, :top]
    picked = torch.gather(s, 1, ids)
    return ids, picked / (picked.sum(dim=-1, keepdim=True) + 1e-20) * scale


def mixture(h, w, m, get):
    ids, weights = choose(h @ get(w + ".router").T, m["router"]["top"], m["router"]["scale"])
    out = torch.zeros_like(h)
    for e in range(m["router"]["experts"]):
        rows, slots = torch.nonzero(ids == e, as_tuple=True)
        if rows.numel():
            out.index_add_(0, rows, weights[rows, slots][:, None] * square_expert(h[rows], f"{w}.e{e}", get))
    return out


# ------------------------------------------------------------------- the model
class PlainLaperax:
    """logits(tokens) of one sequence from a model folder's config and tensors; `dtype` float64 or float32."""

    def __init__(self, config, tensors, dtype=torch.float64):
        self.config, self.dtype = config, dtype
        self.tensors = {n: t.to(dtype) for n, t in tensors.items()}

    def embed(self, tokens):
        return rms_norm(self.tensors["embed"][list(tokens)], self.tensors["embed.norm"], self.config["norm"]["eps"])

    def layer(self, i, x):
        c, get = self.config, self.tensors.__getitem__
        layer, w, eps = c["layers"][i], f"l{i}", c["norm"]["eps"]
        h = rms_norm(x, get(w + ".norm1"), eps)
        y = MIXERS[layer["type"]](h, w + ".mix", layer["mixer"], eps, get)
        if layer.get("mlp") is not None:
            y = y + mixture(h, w + ".mlp", layer["mlp"], get)
        return x + y

    def residuals(self, tokens):
        """The stream after every layer, [layers, T, width]."""
        x, out = self.embed(tokens), []
        for i in range(len(self.config["layers"])):
            x = self.layer(i, x)
            out.append(x)
        return torch.stack(out)

    def logits(self, tokens):
        c = self.config
        x = rms_norm(self.residuals(tokens)[-1], self.tensors["final.norm"], c["norm"]["eps"])
        return squash(x @ self.tensors["head"].T * c["logit_scale"], c["logit_softcap"])


def load(folder, dtype=torch.float64):
    with open(folder + "/config.json", encoding="utf-8") as f:
        config = json.load(f)
    return PlainLaperax(config, read_safetensors(folder + "/model.safetensors"), dtype)


def greedy(model, prompt, n):
    """n tokens of greedy continuation, every step from the whole sequence again."""
    tokens = list(prompt)
    for _ in range(n):
        tokens.append(int(torch.argmax(model.logits(tokens)[-1])))
    return tokens[len(prompt):]
