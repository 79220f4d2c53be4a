"""Plain restatement of the Rovurax decoder in float64 torch, one function per mechanism.  Independent of the package: it
shares no code with it and keeps no cache.

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


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def yarn_frequencies(rot):
    """(f_i of the rotated pairs, factor on cos and sin)."""
    dims, base, sc = rot["dims"], float(rot["base"]), rot.get("scaling")
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not sc:
        return torch.tensor(f, dtype=F64), 1.0

    def pair_that_turns(t):          # index of the pair that turns t times within the original length
        return dims * math.log(sc["original"] / (2 * math.pi * t)) / (2 * math.log(base))
    lo = max(math.floor(pair_that_turns(sc["fast"])), 0)
    hi = min(math.ceil(pair_that_turns(sc["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / sc["factor"] * ramp + fi * (1 - ramp))
    return torch.tensor(out, dtype=F64), 0.1 * math.log(sc["factor"]) + 1


def rotate_interleaved(x, positions, rot):
    """x [T, heads, dim]: neighbours (2 i, 2 i + 1) of the first ``dims`` entries turn together."""
    f, gain = yarn_frequencies(rot)
    a = positions.to(F64)[:, None, None] * f
    c, s = gain * a.cos(), gain * a.sin()
    out = x.clone()
    u, v = x[..., 0:rot["dims"]:2], x[..., 1:rot["dims"]:2]
    out[..., 0:rot["dims"]:2] = u * c - v * s
    out[..., 1:rot["dims"]:2] = v * c + u * s
    return out


def causal_mask(T):
    """[T, T], True where row i sees column j."""
    pos = torch.arange(T)
    return pos[None, :] <= pos[:, None]


def chunk_mask(T, size):
    pos = torch.arange(T)
    return causal_mask(T) & (pos[None, :] // size == pos[:, None] // size)


def visible_softmax(scores, mask, sink=None):
    """scores [H, T, L]; ``sink`` [H]: one more term in every denominator."""
    s = scores.masked_fill(~mask, float("-inf"))
    top = s.max(-1, keepdim=True).values
    if sink is not None:
        top = torch.maximum(top, sink[:, None, None])
    e = torch.exp(s - top)
    total = e.sum(-1, keepdim=True)
    if sink is not None:
        total = total + torch.exp(sink[:, None, None] - top)
    return e / total


def attend(q, k, v, scale, mask, sink=None):
    """q [T, H, d], k [T, G, d], v [T, G, dv]: query head h reads key / value head h // (H / G)."""
    rep = q.shape[1] // k.shape[1]
    k, v = k.repeat_interleave(rep, 1), v.repeat_interleave(rep, 1)
    s = torch.einsum("thd,lhd->htl", q, k) * scale
    return torch.einsum("htl,lhv->thv", visible_softmax(s, mask, sink), v)


def mix_values(v, first, weight):
    return (1 - weight) * v + weight * first


def latent_attention(h, w, p, m, eps):
    T = h.shape[0]
    H, d, r, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    q = lin(h, w[p + "q"]).view(T, H, d + r)
    down = lin(h, w[p + "dkv"])
    c, turned = round_16(rms_norm(down[:, :rank], w[p + "dkv.norm"], eps)), down[:, None, rank:]
    plain, q_turned = q[..., :d], q[..., d:]
    if m.get("rot"):
        turned, q_turned = rotate_interleaved(turned, pos, m["rot"]), rotate_interleaved(q_turned, pos, m["rot"])
    k = torch.cat([lin(c, w[p + "uk"]).view(T, H, d), round_16(turned).expand(T, H, r)], -1)
    v = lin(c, w[p + "uv"]).view(T, H, dv)
    o = attend(torch.cat([plain, round_16(q_turned)], -1), k, v, m["scale"], causal_mask(T), w[p + "sink"])
    o = o * torch.sigmoid(lin(h, w[p + "g"]))[:, :, None]
    return lin(o.reshape(T, H * dv), w[p + "o"])


def attention(h, w, p, m, first=None):
    """Returns (output, values before mixing); ``first`` = the values to mix in, None when there is nothing to mix."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, own = lin(h, w[p + "q"]).view(T, H, d), lin(h, w[p + "k"]).view(T, G, d), lin(h, w[p + "v"]).view(T, G, dv)
    v = own if first is None else round_16(mix_values(own, first, w[p + "vmix"]))
    mask = chunk_mask(T, m["mask"]["size"]) if m.get("mask") else causal_mask(T)
    o = attend(q, k, v, m["scale"], mask)
    return lin(o.reshape(T, H * dv), w[p + "o"]), own


def clamped_gate(g, u, limit):
    g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


def dense_ff(h, w, p, limit):
    return lin(clamped_gate(lin(h, w[p + "gate"]), lin(h, w[p + "up"]), limit), w[p + "down"])


def forward(config, weights, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence; ``layers_out`` (a list) receives the residual after every layer."""
    w = {k: v.to(F64) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)]
    first = None
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = rms_norm(x, w[p + "norm1"], eps)
        if layer["type"] == "latent_attention":
            y = latent_attention(h, w, p + "mix.", m, eps)
        else:
            mixes = bool(m.get("v_mix"))
            y, own = attention(h, w, p + "mix.", m, first if mixes else None)
            if mixes and first is None:
                first = own
        if layer["mlp"] is not None:
            y = y + dense_ff(h, w, p + "mlp.", layer["mlp"]["limit"])
        x = x + y
        if layers_out is not None:
            layers_out.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T


def rounding_noise(config, weights, tokens):
    """Difference of the logits that 16-bit projections alone make, [T, vocab]."""
    global ROUND_16
    exact = forward(config, weights, tokens)
    ROUND_16 = True
    try:
        return forward(config, weights, tokens) - exact
    finally:
        ROUND_16 = False
