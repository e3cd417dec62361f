"""A plain, slow statement of the Vekusun decoder, one function per mechanism, in float64 on the CPU.

It shares no code with the engine: every function takes plain tensors and the numbers of its own section of
config.json and works on ONE sequence from its first token.  `forward` returns the logits of every position and
the residual stream after every layer run (a layer inside the loop counts once per pass).

Notation: T tokens, W the model width, x [T, W] the residual stream, h [T, W] a layer's normed input.  Linear weights
are [out, in].
"""
from __future__ import annotations

import math

import torch

F = torch.float64


def lin(w, h):
    return h @ w.to(F).t()


def sub(w, prefix):
    return {k[len(prefix):]: t for k, t in w.items() if k.startswith(prefix)}


def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w.to(F)


def silu(z):
    return z / (1.0 + torch.exp(-z))


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def gelu(z):
    """z times the normal distribution function at z."""
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


# ---------------------------------------------------------------- rotation
def frequencies(rot):
    """base^(-2i/dims); with rot["scaling"] those that turn slowly against the original context are divided by the factor:
    c(t) is the (fractional) pair counted in features that turns t times in the original context, and between c(fast) and
    c(slow) a ramp leads from the plain to the divided frequency."""
    n, base, sc = rot["dims"], float(rot["base"]), rot.get("scaling")
    plain = [base ** (-2.0 * i / n) for i in range(n // 2)]
    if sc is None:
        return plain
    c = lambda turns: n * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(c(sc["fast"])), 0), min(math.ceil(c(sc["slow"])), n - 1)
    out = []
    for i, f in enumerate(plain):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / sc["factor"] * ramp + f * (1.0 - ramp))
    return out


def magnitude(rot):
    """The factor on sine and cosine that goes with the slowed frequencies."""
    return 1.0 if rot.get("scaling") is None else 0.1 * math.log(rot["scaling"]["factor"]) + 1.0


def rotate(x, rot):
    """x [T, ..., n]: pairs (2i, 2i + 1) of the first `dims` features turned by position * frequency."""
    T = x.shape[0]
    pos, amp = torch.arange(T, dtype=F), magnitude(rot)
    out = x.clone()
    shape = (T,) + (1,) * (x.dim() - 2)
    for i, f in enumerate(frequencies(rot)):
        c, s = (amp * torch.cos(pos * f)).reshape(shape), (amp * torch.sin(pos * f)).reshape(shape)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


# ---------------------------------------------------------------- the two attentions
def causal_weights(s, sink=None):
    """Softmax over the keys j <= i of every row i; `sink` (a number): exp(sink) joins the denominator."""
    T = s.shape[0]
    s = s.masked_fill(~torch.tril(torch.ones(T, T, dtype=torch.bool)), -math.inf)
    m = s.max(-1, keepdim=True).values
    if sink is not None:
        m = torch.clamp(m, min=float(sink))
    e = torch.exp(s - m)
    d = e.sum(-1, keepdim=True)
    return e / (d if sink is None else d + torch.exp(sink - m))


def sink_attention(h, w, m, eps):
    """Queries through a latent of their own, keys and values from one latent row, no positions, a sink per head."""
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = lin(w["uq"], rms_norm(lin(w["dq"], h), w["dq.norm"], eps)).reshape(T, H, D)
    c = rms_norm(lin(w["dkv"], h), w["dkv.norm"], eps)
    k, v = lin(w["uk"], c).reshape(T, H, D), lin(w["uv"], c).reshape(T, H, V)
    sink = w["sink"].to(F)
    out = torch.stack([causal_weights(q[:, a] @ k[:, a].t() * m["scale"], sink[a]) @ v[:, a] for a in range(H)], 1)
    return lin(w["o"], out.reshape(T, H * V))


def rotated_attention(h, w, m, eps):
    """Queries straight from the input, keys and values from one latent row beside one rotated key part for all heads,
    a sigmoid gate per head."""
    T, H, D, R, V = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    q = lin(w["q"], h).reshape(T, H, D + R)
    qr = rotate(q[..., D:], m["rot"])
    down = lin(w["dkv"], h)
    c, kr = rms_norm(down[:, :m["kv_rank"]], w["dkv.norm"], eps), rotate(down[:, m["kv_rank"]:], m["rot"])
    k, v = lin(w["uk"], c).reshape(T, H, D), lin(w["uv"], c).reshape(T, H, V)
    gate = sigmoid(lin(w["g"], h))
    out = torch.stack([gate[:, a:a + 1] * (causal_weights((q[:, a, :D] @ k[:, a].t() + qr[:, a] @ kr.t()) * m["scale"]) @ v[:, a])
                       for a in range(H)], 1)
    return lin(w["o"], out.reshape(T, H * V))


# ---------------------------------------------------------------- the recurrence
def causal_conv(x, taps):
    """out[t, c] = sum_j taps[c, j] x[t - (n - 1) + j, c], zeros before the start."""
    T, n = x.shape[0], taps.shape[1]
    padded = torch.cat([torch.zeros(n - 1, x.shape[1], dtype=F), x], 0)
    out = torch.zeros_like(x)
    for j in range(n):
        out = out + taps.to(F)[:, j] * padded[j:j + T]
    return out


def unit_vectors(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def head_decay(a, A_log, dt_bias):
    return torch.exp(-torch.exp(A_log.to(F)) * softplus(a + dt_bias.to(F)))


def delta_steps(q, k, v, beta, g):
    """q, k [T, H, D], v [T, H, P], beta, g [T, H]: decay, correct, write, then read; from a state of zeros."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=F)
    out = []
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdp,hd->hp", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hdp,hd->hp", S, q[t]))
    return torch.stack(out)


def delta(h, w, m, eps):
    T, H, G, D, P = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    mixed = lambda n: silu(causal_conv(lin(w[n], h), w[n + ".conv"]))
    per_head = lambda x: unit_vectors(x.reshape(T, G, D)).repeat_interleave(H // G, 1)
    q, k = per_head(mixed("q")) * D ** -0.5, per_head(mixed("k"))
    o = delta_steps(q, k, mixed("v").reshape(T, H, P), sigmoid(lin(w["b"], h)), head_decay(lin(w["a"], h), w["A_log"], w["dt_bias"]))
    y = rms_norm(o, w["norm"], eps) * silu(lin(w["g"], h)).reshape(T, H, P)
    return lin(w["o"], y.reshape(T, H * P))


MIXERS = {"latent_attention": sink_attention, "latent_attention_2": rotated_attention, "delta": delta}


# ---------------------------------------------------------------- feed-forwards
def dense_ff(h, w):
    return lin(w["down"], gelu(lin(w["up"], h)))


def route(h, router, correction, top):
    """Per token: the chosen experts (by softmax score + correction) and their weights (the scores as they are)."""
    s = torch.softmax(lin(router, h), -1)
    choice = s + correction.to(F)
    ids, weights = [], []
    for t in range(h.shape[0]):
        pick = sorted(range(s.shape[1]), key=lambda e: (-float(choice[t, e]), e))[:top]
        ids.append(pick)
        weights.append(s[t, pick])
    return ids, weights


def expert_mixture(h, w, mlp):
    ids, weights = route(h, w["router"], w["correction"], mlp["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        rows = [t for t in range(h.shape[0]) if e in ids[t]]
        if rows:
            x = h[rows]
            y = lin(w[f"e{e}.down"], silu(lin(w[f"e{e}.gate"], x)) * lin(w[f"e{e}.up"], x))
            p = torch.stack([weights[t][ids[t].index(e)] for t in rows])
            out[rows] += p[:, None] * y
    return out


# ---------------------------------------------------------------- the model
def run_order(config):
    """[(layer, pass or None)]: which layers run, and for a pass's first layer the number of the pass."""
    n, loop = len(config["layers"]), config.get("loop")
    if loop is None:
        return [(i, None) for i in range(n)]
    order = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        order += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return order + [(i, None) for i in range(loop["stop"], n)]


def layer_run(x, w, layer, m, eps):
    """One norm, mixer and feed-forward side by side on it, each scaled per channel, the sum times m added."""
    h = rms_norm(x, w["norm1"], eps)
    y = MIXERS[layer["type"]](h, sub(w, "mix."), layer["mixer"], eps) * w["ls1"].to(F)
    if layer.get("mlp") is not None:
        fw = sub(w, "mlp.")
        y = y + (dense_ff(h, fw) if layer["mlp"]["kind"] == "dense" else expert_mixture(h, fw, layer["mlp"])) * w["ls2"].to(F)
    return x + m * y


def capped(z, cap):
    return cap * torch.tanh(z / cap)


def forward(config, weights, tokens):
    """logits [T, vocab] and the stream after every layer run [runs, T, W]."""
    eps = config["norm"]["eps"]
    w = {k: v.to(F) for k, v in weights.items()}
    first = w["embed"][torch.as_tensor(list(tokens), dtype=torch.long)]
    x, streams = first, []
    for i, start_of in run_order(config):
        if start_of is not None:
            if start_of > 0:
                x = x + first
            x = x + w["loop.step"][start_of]
        x = layer_run(x, sub(w, f"l{i}."), config["layers"][i], config["residual_mult"], eps)
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
