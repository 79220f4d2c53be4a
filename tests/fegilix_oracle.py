"""Plain restatement of the Fegilix decoder in float64 torch, one function per mechanism, token loops where the
mathematics has a recurrence.  Independent of the package: it shares no code with it and keeps no cache.

``weights`` maps tensor names to torch tensors, ``config`` is the parsed config.json.
"""
import math

import torch

F64 = torch.float64


ROUND_16 = False     # round what enters and leaves every projection to bfloat16: shows how much a model amplifies rounding


def round_16(x):
    return x.to(torch.bfloat16).to(x.dtype) if ROUND_16 else x


def lin(x, w):
    return round_16(round_16(x) @ w.T)


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, weight, eps):
    return rms(x, eps) * weight


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


def rotary_frequencies(rot):
    """Inverse wavelengths f_i of the rotated pairs, after the three-band rescaling when the entry has one."""
    dims, base, sc = rot["dims"], float(rot["base"]), rot.get("scaling")
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if sc:
            wavelength = 2 * math.pi / f
            if wavelength > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif wavelength >= sc["original"] / sc["high"]:
                s = (sc["original"] / wavelength - sc["low"]) / (sc["high"] - sc["low"])
                f = (1 - s) * f / sc["factor"] + s * f
        out.append(f)
    return torch.tensor(out, dtype=F64)


def rotate(x, positions, rot):
    """x [T, heads, dim]: rotate-half layout on the first ``dims`` entries of each head."""
    half = rot["dims"] // 2
    a = positions.to(F64)[:, None, None] * rotary_frequencies(rot)
    u, v, rest = x[..., :half], x[..., half:2 * half], x[..., 2 * half:]
    return torch.cat([u * a.cos() - v * a.sin(), v * a.cos() + u * a.sin(), rest], -1)


def causal_conv_silu(x, taps):
    """x [T, C], taps [C, K] with the newest token's coefficient last; zeros in front of the sequence."""
    T, K = x.shape[0], taps.shape[1]
    padded = torch.cat([torch.zeros(K - 1, x.shape[1], dtype=x.dtype), x])
    out = torch.zeros_like(x)
    for j in range(K):
        out = out + padded[j:j + T] * taps[:, j]
    return silu(out)


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def gated_delta_scan(q, k, v, beta, decay):
    """q, k, decay [T, H, dk], v [T, H, dv], beta [T, H]; returns [T, H, dv]."""
    T, H, dk = q.shape
    S = torch.zeros(H, dk, v.shape[-1], dtype=q.dtype)
    out = []
    for t in range(T):
        S = decay[t][:, :, None] * S
        read = (S * k[t][:, :, None]).sum(1)
        u = beta[t][:, None] * (v[t] - read)
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out)


def mlstm_scan(q, k, v, i_gate, f_gate, floor=True):
    """``floor=False`` plants a mistake: the denominator is |n . q| alone.  q, k [T, H, dk], v [T, H, dv], log gates [T, H]; returns [T, H, dv]."""
    T, H, dk = q.shape
    S = torch.zeros(H, dk, v.shape[-1], dtype=q.dtype)
    n = torch.zeros(H, dk, dtype=q.dtype)
    m = torch.zeros(H, dtype=q.dtype)
    out = []
    for t in range(T):
        m_new = torch.maximum(f_gate[t] + m, i_gate[t])
        keep, add = torch.exp(f_gate[t] + m - m_new), torch.exp(i_gate[t] - m_new)
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[t]
        m = m_new
        num = (S * q[t][:, :, None]).sum(1)
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m) * float(floor)) + 1e-6
        out.append(num / den[:, None])
    return torch.stack(out)


def softmax_with_sink(scores, sink):
    """scores [H, T, L] (masked entries -inf), sink [H]: one more term in every denominator."""
    top = torch.maximum(scores.max(-1, keepdim=True).values, sink[:, None, None])
    e = torch.exp(scores - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink[:, None, None] - top))


def causal_attention(q, k, v, scale, sink):
    """q [T, H, d], k [T, G, d], v [T, G, dv]: query head h reads key / value head h // (H / G)."""
    rep = q.shape[1] // k.shape[1]
    k, v = k.repeat_interleave(rep, 1), v.repeat_interleave(rep, 1)
    s = torch.einsum("thd,lhd->htl", q, k) * scale
    pos = torch.arange(q.shape[0])
    s = s.masked_fill(pos[None, None, :] > pos[None, :, None], float("-inf"))
    return torch.einsum("htl,lhv->thv", softmax_with_sink(s, sink), v)


def channel_delta(h, w, p, m, eps):
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = causal_conv_silu(lin(h, w[p + "q"]), w[p + "q.conv"]).view(T, G, dk)
    k = causal_conv_silu(lin(h, w[p + "k"]), w[p + "k.conv"]).view(T, G, dk)
    v = causal_conv_silu(lin(h, w[p + "v"]), w[p + "v.conv"]).view(T, H, dv)
    q, k = unit(q) * dk ** -0.5, unit(k)
    q, k = q.repeat_interleave(H // G, 1), k.repeat_interleave(H // G, 1)
    beta = torch.sigmoid(lin(h, w[p + "b"]))
    rate = torch.nn.functional.softplus(lin(lin(h, w[p + "a1"]), w[p + "a2"]) + w[p + "dt_bias"], threshold=1e9).view(T, H, dk)
    decay = torch.exp(-torch.exp(w[p + "A_log"])[None, :, None] * rate)
    o = rms_norm(gated_delta_scan(q, k, v, beta, decay), w[p + "norm"], eps)
    gate = torch.sigmoid(lin(lin(h, w[p + "g1"]), w[p + "g2"])).view(T, H, dv)
    return lin((o * gate).reshape(T, H * dv), w[p + "o"])


def mlstm(h, w, p, m, eps):
    T = h.shape[0]
    H, dk, dv, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (lin(h, w[p + "q"]) * dk ** -0.5).view(T, H, dk)
    k = (lin(h, w[p + "k"])).view(T, H, dk)
    v = (lin(h, w[p + "v"])).view(T, H, dv)
    i_gate = cap * torch.tanh((lin(h, w[p + "i"]) + w[p + "i.b"]) / cap)
    f_gate = torch.nn.functional.logsigmoid(cap * torch.tanh((lin(h, w[p + "f"]) + w[p + "f.b"]) / cap))
    o = rms(mlstm_scan(q, k, v, i_gate, f_gate), eps).reshape(T, H * dv)
    return lin(o * w[p + "norm"] * torch.sigmoid(lin(h, w[p + "g"])), w[p + "o"])


def attention(h, w, p, m, eps, kv=None):
    """Returns (output, (keys, values)); ``kv`` = another layer's keys and values."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    turn = (lambda x: rotate(x, pos, m["rot"])) if m.get("rot") else (lambda x: x)
    q = turn(rms_norm((lin(h, w[p + "q"])).view(T, H, d), w[p + "q.norm"], eps))
    if kv is None:
        k = turn(rms_norm((lin(h, w[p + "k"])).view(T, G, d), w[p + "k.norm"], eps))
        v = (lin(h, w[p + "v"])).view(T, G, dv)
        kv = (k, v)
    o = causal_attention(q, kv[0], kv[1], m["scale"], w[p + "sink"]).reshape(T, H * dv)
    return lin(o * torch.sigmoid(lin(h, w[p + "g"])), w[p + "o"]), kv


def dense_ff(h, w, p):
    return lin(gelu_tanh(lin(h, w[p + "gate"])) * lin(h, w[p + "up"]), w[p + "down"])


def hyper_read(streams, w_in):
    return torch.einsum("s,tsw->tw", w_in, streams)


def hyper_write(streams, mix, w_out, y):
    return torch.einsum("st,nsw->ntw", mix, streams) + w_out[None, :, None] * y[:, None, :]


class PlainStream(dict):
    """Weights of a model without hyper-connections: every read, write and mix factor is 1."""

    def __missing__(self, name):
        assert ".hc" in name, name
        return torch.ones((1, 1) if name.endswith("mix") else 1, dtype=F64)


def forward(config, weights, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence; ``layers_out`` (a list) receives the stream sum after every layer."""
    w = {k: v.to(F64) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)]
    plain = config.get("streams") is None       # one residual stream, x <- x + y
    n = 1 if plain else config["streams"]
    if plain:
        w = PlainStream(w)
    streams = x[:, None, :].repeat(1, n, 1)
    caches = {}
    for i, layer in enumerate(config["layers"]):
        L, m = f"l{i}.", layer["mixer"]
        h = rms_norm(hyper_read(streams, w[L + "hc1.in"]), w[L + "norm1"], eps)
        if layer["type"] == "attention":
            y, caches[i] = attention(h, w, L + "mix.", m, eps, caches[m["kv_from"]] if m.get("kv_from") is not None else None)
        elif layer["type"] == "channel_delta":
            y = channel_delta(h, w, L + "mix.", m, eps)
        else:
            y = mlstm(h, w, L + "mix.", m, eps)
        streams = hyper_write(streams, w[L + "hc1.mix"], w[L + "hc1.out"], y)
        if layer["mlp"] is not None:
            h = rms_norm(hyper_read(streams, w[L + "hc2.in"]), w[L + "norm2"], eps)
            streams = hyper_write(streams, w[L + "hc2.mix"], w[L + "hc2.out"], dense_ff(h, w, L + "mlp."))
        if layers_out is not None:
            layers_out.append(streams.sum(1))
    logits = rms_norm(streams.sum(1), w["final.norm"], eps) @ w["head"].T
    cap = config.get("logit_softcap")
    return cap * torch.tanh(logits / cap) if cap else logits


def rounding_noise(config, weights, tokens):
    """Difference of the logits that 16-bit projections alone make, [T, vocab]."""
    global ROUND_16
    exact = forward(config, weights, tokens)
    ROUND_16 = True
    try:
        return forward(config, weights, tokens) - exact
    finally:
        ROUND_16 = False
