"""A plain, slow statement of the Pafelorn decoder, one function per mechanism, in float64 on the CPU.

It shares no code with the engine: every function takes plain tensors and the numbers of its own section of
config.json and works on ONE sequence from its first token.  `forward` returns the logits of every position and
the residual stream after every layer.

Notation: T tokens, W the model width, x [T, W] the residual stream, h [T, W] a sub-layer's input.  Linear weights
are [out, in].
"""
from __future__ import annotations

import math

import torch

F = torch.float64


def lin(w, h, b=None):
    y = h @ w.to(F).t()
    return y if b is None else y + b.to(F)


def sub(w, prefix):
    return {k[len(prefix):]: t for k, t in w.items() if k.startswith(prefix)}


def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w.to(F)


# ---------------------------------------------------------------- embedding
def bigram_rows(tokens, bigram):
    """Row of the bigram table per token: a hash of (token before, token); the row behind the hashed ones for the first."""
    rows, before = [], None
    for t in tokens:
        rows.append(bigram["buckets"] if before is None
                    else (before * bigram["mul_prev"] + t * bigram["mul_cur"]) % bigram["buckets"])
        before = t
    return rows


def embedding(tokens, w, config):
    ids = torch.as_tensor(list(tokens), dtype=torch.long)
    x = w["embed"].to(F)[ids] * config["embedding"]["scale"]
    return x + w["bigram"].to(F)[torch.as_tensor(bigram_rows(list(tokens), config["embedding"]["bigram"]), dtype=torch.long)]


# ---------------------------------------------------------------- rotation
def frequencies(rot):
    """base^(-2i/dims), slowed down as rot["scaling"] says: all of them by a factor, or (with low / high / original) only
    those whose wavelength is long against the original context, with a ramp between."""
    out = []
    sc = rot.get("scaling")
    for i in range(rot["dims"] // 2):
        f = float(rot["base"]) ** (-2.0 * i / rot["dims"])
        if sc is None:
            out.append(f)
        elif "original" not in sc:
            out.append(f / sc["factor"])
        else:
            wave = 2.0 * math.pi / f
            if wave < sc["original"] / sc["high"]:
                out.append(f)
            elif wave > sc["original"] / sc["low"]:
                out.append(f / sc["factor"])
            else:
                s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                out.append((1.0 - s) * f / sc["factor"] + s * f)
    return out


def rotate(x, rot, interleaved):
    """x [T, ..., n]: pairs (2i, 2i + 1) when interleaved, else (i, i + dims/2), of the first `dims` features turned by
    position * frequency."""
    T, dims = x.shape[0], rot["dims"]
    pos = torch.arange(T, dtype=F)
    out = x.clone()
    shape = (T,) + (1,) * (x.dim() - 2)
    for i, f in enumerate(frequencies(rot)):
        a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + dims // 2)
        c, s = torch.cos(pos * f).reshape(shape), torch.sin(pos * f).reshape(shape)
        u, v = x[..., a], x[..., b]
        out[..., a] = u * c - v * s
        out[..., b] = v * c + u * s
    return out


# ---------------------------------------------------------------- masks and softmax
def visible(T, mask):
    """[T, T] booleans: which key j (column) query i (row) sees."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    if mask is not None:
        seen = seen & ((i - j < mask["size"]) | (j < mask.get("keep_first", 0)))
    return seen


def softmax_rows(s, seen, sink=None):
    """Softmax over the visible keys of every row; `sink` (a number): exp(sink) joins the denominator."""
    s = s.masked_fill(~seen, -math.inf)
    m = s.max(-1, keepdim=True).values
    if sink is not None:
        m = torch.clamp(m, min=float(sink))
    e = torch.exp(s - m)
    d = e.sum(-1, keepdim=True)
    if sink is not None:
        d = d + torch.exp(sink - m)
    return e / d


def capped(s, cap):
    return cap * torch.tanh(s / cap)


# ---------------------------------------------------------------- the three attentions
def head_norm_attention(h, w, m, eps):
    """Left side of 'parallel': biases, a norm per head, interleaved rotation, a factor per head, window, learned sink."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rotate(rms_norm(lin(w["q"], h, w["q.b"]).reshape(T, H, D), w["q.norm"], eps), m["rot"], True)
    k = rotate(rms_norm(lin(w["k"], h, w["k.b"]).reshape(T, G, D), w["k.norm"], eps), m["rot"], True)
    v = lin(w["v"], h, w["v.b"]).reshape(T, G, V)
    temp, sink, seen = w["temp"].to(F), w["sink"].to(F), visible(T, m.get("mask"))
    out = torch.zeros(T, H, V, dtype=F)
    for a in range(H):
        g = a // (H // G)
        out[:, a] = softmax_rows(q[:, a] @ k[:, g].t() * m["scale"] * temp[a], seen, sink[a]) @ v[:, g]
    return lin(w["o"], out.reshape(T, H * V), w["o.b"])


def row_norm_attention(h, w, m, eps):
    """Left side of 'parallel_2': a norm over the whole projection, interleaved rotation, capped scores, a window beside
    kept first tokens, a sigmoid gate on the heads."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rotate(rms_norm(lin(w["q"], h), w["q.norm"], eps).reshape(T, H, D), m["rot"], True)
    k = rotate(rms_norm(lin(w["k"], h), w["k.norm"], eps).reshape(T, G, D), m["rot"], True)
    v = lin(w["v"], h).reshape(T, G, V)
    seen = visible(T, m.get("mask"))
    out = torch.zeros(T, H, V, dtype=F)
    for a in range(H):
        g = a // (H // G)
        out[:, a] = softmax_rows(capped(q[:, a] @ k[:, g].t() * m["scale"], m["softcap"]), seen) @ v[:, g]
    return lin(w["o"], out.reshape(T, H * V) * torch.sigmoid(lin(w["g"], h)))


def difference_weight(w, diff):
    """lambda: exp(lq1 . lk1) - exp(lq2 . lk2) + diff, one number."""
    dot = lambda a, b: (w[a].to(F) * w[b].to(F)).sum()
    return torch.exp(dot("lq1", "lk1")) - torch.exp(dot("lq2", "lk2")) + diff


def combine_maps(a1, a2, lam, diff, eps):
    """(a1 - lambda a2) normed per head, no weight, times (1 - diff)."""
    return unit_rms(a1 - lam * a2, eps) * (1.0 - diff)


def differential_attention(h, w, m, eps, kv=None):
    """Returns (output, (k, v)); `kv`: keys and values of another layer, as that layer made them."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rotate(rms_norm(lin(w["q"], h, w["q.b"]).reshape(T, H, 2, D), w["q.norm"], eps), m["rot"], False)
    if kv is None:
        k = rotate(rms_norm(lin(w["k"], h, w["k.b"]).reshape(T, G, 2, D), w["k.norm"], eps), m["rot"], False)
        v = lin(w["v"], h, w["v.b"]).reshape(T, G, V)
        kv = (k, v)
    k, v = kv
    seen = visible(T, m.get("mask"))
    lam = difference_weight(w, m["diff"])
    out = torch.zeros(T, H, V, dtype=F)
    for a in range(H):
        g = a // (H // G)
        maps = [softmax_rows(q[:, a, i] @ k[:, g, i].t() * m["scale"], seen) @ v[:, g] for i in range(2)]
        out[:, a] = combine_maps(maps[0], maps[1], lam, m["diff"], eps)
    return lin(w["o"], out.reshape(T, H * V)), kv


# ---------------------------------------------------------------- the two recurrences
def causal_conv(x, taps, bias):
    """out[t, c] = bias[c] + sum_j taps[c, j] x[t - (n - 1) + j, c], zeros before the start."""
    T, C = x.shape
    n = taps.shape[1]
    padded = torch.cat([torch.zeros(n - 1, C, dtype=F), x], 0)
    out = bias.to(F).expand(T, C).clone()
    for j in range(n):
        out = out + taps.to(F)[:, j] * padded[j:j + T]
    return out


def linear_recurrence(a, b):
    """S_t = a_t S_(t-1) + b_t, element by element, from zero."""
    S, out = torch.zeros_like(a[0]), []
    for t in range(a.shape[0]):
        S = a[t] * S + b[t]
        out.append(S)
    return torch.stack(out)


def candidate(u):
    """u + 1/2 where u >= 0, sigmoid(u) where u < 0."""
    return torch.where(u >= 0, u + 0.5, torch.sigmoid(u))


def min_gru(h, w, m, eps):
    z = torch.sigmoid(lin(w["z"], h, w["z.b"]))
    S = linear_recurrence(1.0 - z, z * candidate(lin(w["x"], h, w["x.b"])))
    return lin(w["o"], S * torch.nn.functional.silu(lin(w["g"], h)))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def block_gates(u, w, b):
    """sigmoid of a product with one square matrix per block of channels."""
    T, C = u.shape
    nb = w.shape[0]
    z = torch.einsum("tbi,boi->tbo", u.reshape(T, nb, C // nb), w.to(F)) + b.to(F)
    return torch.sigmoid(z).reshape(T, C)


def gated_lru(h, w, m, eps):
    y = gelu_tanh(lin(w["y"], h, w["y.b"]))
    u = causal_conv(lin(w["x"], h, w["x.b"]), w["conv"], w["conv.b"])
    r, i = block_gates(u, w["ra"], w["ra.b"]), block_gates(u, w["ri"], w["ri.b"])
    log_a = -8.0 * r * torch.nn.functional.softplus(w["lam"].to(F))
    a = torch.exp(log_a)
    S = linear_recurrence(a, torch.sqrt(-torch.expm1(2.0 * log_a)) * i * u)
    return lin(w["o"], S * y)


# ---------------------------------------------------------------- two mixers side by side
def parallel(h, w, m, eps):
    return (m["left_scale"] * head_norm_attention(h, sub(w, "left."), m["left"], eps)
            + m["right_scale"] * min_gru(h, sub(w, "right."), m["right"], eps))


def parallel_2(h, w, m, eps):
    left = row_norm_attention(h, sub(w, "left."), m["left"], eps)
    right = gated_lru(h, sub(w, "right."), m["right"], eps)
    return 0.5 * (rms_norm(left, w["left.out"], eps) + rms_norm(right, w["right.out"], eps))


# ---------------------------------------------------------------- feed-forwards
def poly_norm(z, act, eps):
    a, b, c, e = [act.to(F)[i] for i in range(4)]
    return a * unit_rms(z, eps) + b * unit_rms(z ** 2, eps) + c * unit_rms(z ** 3, eps) + e


def dense_ff(h, w, eps):
    return lin(w["down"], poly_norm(lin(w["up"], h), w["act"], eps))


def capped_expert(h, gate, up, down, limit):
    g = torch.clamp(lin(gate, h), max=limit)
    u = torch.clamp(lin(up, h), min=-limit, max=limit)
    return lin(down, g * torch.sigmoid(1.702 * g) * (u + 1.0))


def route(h, router, correction, top):
    """Per token: the chosen experts (by softmax score + correction) and their weights (scores over their sum)."""
    s = torch.softmax(lin(router, h), -1)
    choice = s + correction.to(F)
    ids, weights = [], []
    for t in range(h.shape[0]):
        pick = sorted(range(s.shape[1]), key=lambda e: (-float(choice[t, e]), e))[:top]
        ids.append(pick)
        weights.append(s[t, pick] / (s[t, pick].sum() + 1e-20))
    return ids, weights


def expert_mixture(h, w, mlp):
    n, limit = mlp["router"]["experts"], mlp["expert"]["limit"]
    ids, weights = route(h, w["router"], w["correction"], mlp["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, p in zip(ids[t], weights[t]):
            row = h[t:t + 1]
            y = row if e >= n else capped_expert(row, w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"], limit)
            out[t] += p * y[0]
    if mlp.get("shared") is not None:
        y = capped_expert(h, w["shared.gate"], w["shared.up"], w["shared.down"], mlp["shared"]["limit"])
        out = out + torch.sigmoid(lin(w["shared.sg"], h)) * y
    return out


# ---------------------------------------------------------------- the model
def forward(config, weights, tokens):
    """logits [T, vocab] and the stream after every layer [layers, T, W]."""
    eps = config["norm"]["eps"]
    w = {k: v.to(F) for k, v in weights.items()}
    x = embedding(tokens, w, config)
    streams, cached = [], {}
    for i, layer in enumerate(config["layers"]):
        lw = sub(w, f"l{i}.")
        mw, m = sub(lw, "mix."), layer["mixer"]
        if layer["type"] == "attention":
            y, cached[i] = differential_attention(x, mw, m, eps, cached[m["kv_from"]] if m.get("kv_from") is not None else None)
        else:
            y = {"parallel": parallel, "parallel_2": parallel_2}[layer["type"]](x, mw, m, eps)
        x = x + rms_norm(y, lw["norm1"], eps)
        if layer.get("mlp") is not None:
            fw = sub(lw, "mlp.")
            y = dense_ff(x, fw, eps) if layer["mlp"]["kind"] == "dense" else expert_mixture(x, fw, layer["mlp"])
            x = x + rms_norm(y, lw["norm2"], eps)
        streams.append(x)
    logits = lin(w["head"], rms_norm(x, w["final.norm"], eps))
    if config.get("logit_softcap"):
        logits = capped(logits, config["logit_softcap"])
    return logits, torch.stack(streams)


def read_model_dir(folder):
    """(config.json as a dict, {name: tensor}) of a model folder; a reader of its own: 8 bytes of length, a JSON
    header name -> (dtype, shape, data_offsets), then the data."""
    import json
    import struct
    from pathlib import Path
    folder = Path(folder)
    config = json.loads((folder / "config.json").read_text())
    raw = (folder / "model.safetensors").read_bytes()
    n = struct.unpack("<Q", raw[:8])[0]
    header = json.loads(raw[8:8 + n])
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "I32": torch.int32}
    weights = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        lo, hi = info["data_offsets"]
        t = torch.frombuffer(bytearray(raw[8 + n + lo:8 + n + hi]), dtype=kinds[info["dtype"]])
        weights[name] = t.reshape(info["shape"]).clone()
    return config, weights
