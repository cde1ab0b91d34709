"""The Zegorax design restated in plain torch, slowly, one function per mechanism: the oracle of the tests.

Everything is float64 and works on ONE whole sequence (tokens 0 .. T-1 from empty memory); the recurrence is a loop over
tokens with the state written out, attention a loop over queries with an explicit list of the keys each one sees, latent
attention expands every key and value, the two maps of differential attention are two attentions.  Nothing here is shared
with the package: weights come as a dictionary from tensor name to tensor, the configuration as the dictionary config.json
holds.
"""
import math

import torch

F64 = torch.float64


def lin(w, x):
    return x @ w.T


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return torch.where(z > 30.0, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


def rms_unit(x, eps):
    """x divided by its root mean square over the last dimension (eps inside the root)."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def tanh_norm(x, alpha, w, b):
    """A squashing in the place of a norm: no statistics of the vector enter."""
    return torch.tanh(alpha * x) * w + b


# ----------------------------------------------------------------------------------------- rotation
def scaled_frequencies(rot):
    """The angle a position adds for each rotated pair.  With ``scaling`` slow pairs (long wavelengths) turn ``factor`` times
    slower, fast ones as they are, and between the two wavelengths the two frequencies are blended."""
    n, base = rot["dims"], rot["base"]
    out = []
    for i in range(n // 2):
        f = base ** (-2.0 * i / n)
        sc = rot.get("scaling")
        if sc:
            length = 2.0 * math.pi / f
            if length > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif length >= sc["original"] / sc["high"]:
                s = (sc["original"] / length - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return out


def turn(x, pairs, freqs):
    """x [T, heads, n]: each (a, b) of ``pairs`` turns by position * its frequency; all other dimensions pass."""
    pos = torch.arange(x.shape[0], dtype=F64)
    out = x.clone()
    for (a, b), f in zip(pairs, freqs):
        c, s = torch.cos(pos * f)[:, None], torch.sin(pos * f)[:, None]
        u, v = x[..., a], x[..., b]
        out[..., a] = u * c - v * s
        out[..., b] = v * c + u * s
    return out


def rotate_halves(x, rot):
    n = rot["dims"]
    return turn(x, [(i, i + n // 2) for i in range(n // 2)], scaled_frequencies(rot))


def rotate_neighbours(x, rot):
    return turn(x, [(2 * i, 2 * i + 1) for i in range(rot["dims"] // 2)], scaled_frequencies(rot))


def visible(i, window):
    """The positions query i sees: all up to itself, or with a window the last ``window`` of them."""
    return (0 if window is None else max(0, i - window + 1)), i + 1


# ----------------------------------------------------------------------------------------- mixers
def one_map(q, k, v, scale):
    """Ordinary causal attention of one head: q, k [T, d], v [T, dv]."""
    out = torch.zeros(q.shape[0], v.shape[1], dtype=F64)
    for i in range(q.shape[0]):
        lo, hi = visible(i, None)
        out[i] = torch.softmax((k[lo:hi] @ q[i]) * scale, 0) @ v[lo:hi]
    return out


def map_weight(w, diff):
    """How much of the second map is taken off the first: one number for the layer."""
    return torch.exp((w["lq1"] * w["lk1"]).sum()) - torch.exp((w["lq2"] * w["lk2"]).sum()) + diff


def differential_attention(h, w, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rotate_halves(lin(w["q"], h).view(T, H * 2, d), m["rot"]).view(T, H, 2, d)
    k = rotate_halves(lin(w["k"], h).view(T, G * 2, d), m["rot"]).view(T, G, 2, d)
    v = lin(w["v"], h).view(T, G, dv)
    lam = map_weight(w, m["diff"])
    gate = torch.sigmoid(lin(w["g"], h))
    o = torch.zeros(T, H, dv, dtype=F64)
    for a in range(H):
        g = a // (H // G)
        first = one_map(q[:, a, 0], k[:, g, 0], v[:, g], m["scale"])
        second = one_map(q[:, a, 1], k[:, g, 1], v[:, g], m["scale"])
        o[:, a] = rms_unit(first - lam * second, eps) * (1.0 - m["diff"]) * gate[:, a:a + 1]
    return lin(w["o"], o.reshape(T, H * dv))


def latent_attention(h, w, m, eps):
    """Keys and values of every head made from one normed vector per token, beside one rotated key part all heads share;
    queries made from a vector of their own; a window; a gate on every number of the output."""
    T = h.shape[0]
    H, d, dr, dv, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = lin(w["uq"], rms_unit(lin(w["dq"], h), eps) * w["dq.norm"]).view(T, H, d + dr)
    down = lin(w["dkv"], h)
    c = rms_unit(down[:, :r], eps) * w["dkv.norm"]
    q_rot = rotate_neighbours(q[..., d:], m["rot"])
    k_rot = rotate_neighbours(down[:, None, r:], m["rot"])[:, 0]
    k = lin(w["uk"], c).view(T, H, d)
    v = lin(w["uv"], c).view(T, H, dv)
    window = (m.get("mask") or {}).get("size")
    o = torch.zeros(T, H, dv, dtype=F64)
    for a in range(H):
        for i in range(T):
            lo, hi = visible(i, window)
            s = (k[lo:hi, a] @ q[i, a, :d] + k_rot[lo:hi] @ q_rot[i, a]) * m["scale"]
            o[i, a] = torch.softmax(s, 0) @ v[lo:hi, a]
    return lin(w["o"], o.reshape(T, H * dv) * torch.sigmoid(lin(w["g"], h)))


def short_conv(u, w):
    """Causal convolution per channel: u [T, C], w [C, taps]; the last tap multiplies the token itself and what lies
    before the sequence is zero."""
    T, taps = u.shape[0], w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=u.dtype), u])
    out = torch.zeros_like(u)
    for t in range(T):
        out[t] = (padded[t:t + taps] * w.T).sum(0)
    return out


def delta_rule(q, k, v, beta, keep):
    """One head: q, k [T, d], v [T, dv], beta, keep [T].  S [d, dv] from zero: it decays as a whole, what it holds under k is
    taken off what is written, and the read sees the write."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=F64)
    out = torch.zeros(q.shape[0], v.shape[1], dtype=F64)
    for t in range(q.shape[0]):
        S = keep[t] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + torch.outer(k[t], u)
        out[t] = S.T @ q[t]
    return out


def delta_mixer(h, w, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = silu(short_conv(lin(w["q"], h), w["q.conv"])).view(T, G, d)
    k = silu(short_conv(lin(w["k"], h), w["k.conv"])).view(T, G, d)
    v = silu(short_conv(lin(w["v"], h), w["v.conv"])).view(T, H, dv)

    def unit(x):
        return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)
    q, k = unit(q) * d ** -0.5, unit(k)
    beta = torch.sigmoid(lin(w["b"], h))
    keep = torch.exp(-torch.exp(w["A_log"]) * softplus(lin(w["a"], h) + w["dt_bias"]))
    out = torch.zeros(T, H, dv, dtype=F64)
    for a in range(H):
        g = a // (H // G)
        out[:, a] = delta_rule(q[:, g], k[:, g], v[:, a], beta[:, a], keep[:, a])
    y = rms_unit(out, eps) * w["norm"] * silu(lin(w["g"], h)).view(T, H, dv)
    return lin(w["o"], y.reshape(T, H * dv))


# ----------------------------------------------------------------------------------------- feed-forward
def dense_feed_forward(h, w):
    a = gelu_tanh(lin(w["gate"], h) + w["gate.b"]) * (lin(w["up"], h) + w["up.b"])
    return lin(w["down"], a) + w["down.b"]


def routed_feed_forward(h, w, f):
    z = lin(w["router"], h) + w["router.b"]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        chosen = torch.topk(z[t], f["router"]["top"]).indices
        share = torch.softmax(z[t][chosen], 0)
        for e, s in zip(chosen.tolist(), share):
            out[t] += s * lin(w[f"e{e}.down"], silu(lin(w[f"e{e}.gate"], h[t])) * lin(w[f"e{e}.up"], h[t]))
    return out


# ----------------------------------------------------------------------------------------- the model
MIXERS = {"attention": differential_attention, "latent_attention": latent_attention, "delta": delta_mixer}


def layer_runs(config):
    """The layers in the order they run."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


def sub(weights, prefix):
    return {k[len(prefix):]: t.to(F64) for k, t in weights.items() if k.startswith(prefix)}


def forward(config, weights, tokens, return_layers=False):
    """Logits [T, vocab] of one sequence (float64); with ``return_layers`` also the residual stream after every layer run."""
    eps = config["norm"]["eps"]
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    x = weights["embed"].to(F64)[tokens] + weights["pos"].to(F64)[:len(tokens)]

    def normed(y, name):
        return tanh_norm(y, *(weights[name + s].to(F64) for s in (".alpha", "", ".b")))
    layers = []
    for i in layer_runs(config):
        layer = config["layers"][i]
        h = normed(x, f"l{i}.norm1")
        y = MIXERS[layer["type"]](h, sub(weights, f"l{i}.mix."), layer["mixer"], eps)
        f = layer.get("mlp")
        if f is not None:
            w = sub(weights, f"l{i}.mlp.")
            y = y + (dense_feed_forward(h, w) if f["kind"] == "dense" else routed_feed_forward(h, w, f))
        x = x + y
        layers.append(x)
    logits = lin(weights["embed"].to(F64), normed(x, "final.norm"))
    return (logits, torch.stack(layers)) if return_layers else logits
