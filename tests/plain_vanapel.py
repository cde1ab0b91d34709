"""The Vanapel design restated in plain torch, slowly, one function per mechanism: the oracle of the tests.

Everything is float64 and works on ONE whole sequence (tokens 0 .. T-1); attention is a loop over queries with an explicit
list of the keys each one sees, and latent attention expands every key and value.  Nothing here is shared with the package:
weights come as a dictionary from tensor name to tensor, the configuration as the dictionary config.json holds.
"""
import math

import torch

F64 = torch.float64


def lin(w, x):
    return x @ w.T


def rms_unit(x, eps):
    """x divided by its root mean square over the last dimension (eps inside the root)."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def grouped_norm(x, w, groups, eps):
    """The vector in ``groups`` runs of neighbours, each divided by its own root mean square; the whole times w."""
    n = x.shape[-1] // groups
    out = torch.empty_like(x)
    for g in range(groups):
        out[..., g * n:(g + 1) * n] = rms_unit(x[..., g * n:(g + 1) * n], eps)
    return out * w


def distance_penalty(r1, r2, distance):
    """What is taken off the score of a key ``distance`` positions back."""
    return r1 * torch.log(1.0 + r2 * distance)


def weights_with_sink(scores, sink):
    """Softmax over the scores and one more number that stands for no key: what is left for the keys."""
    all_of_them = torch.cat([scores, sink.reshape(1)])
    return torch.softmax(all_of_them, 0)[:-1]


def visible(i, window):
    """The positions query i sees: all up to itself, or with a window the last ``window`` of them."""
    return (0 if window is None else max(0, i - window + 1)), i + 1


def mixed_values(v, v_first, lam):
    """Each token's values moved towards the values of the same token in an earlier layer."""
    return (1.0 - lam) * v + lam * v_first


def window_attention(h, w, m, eps, v_first=None):
    """Grouped-query attention without rotation: unit queries and keys, a logarithmic distance penalty, a window, a sink.
    Returns (output, the values as projected)."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_unit(lin(w["q"], h).view(T, H, d), eps)
    k = rms_unit(lin(w["k"], h).view(T, G, d), eps)
    own = lin(w["v"], h).view(T, G, dv)
    v = own if v_first is None else mixed_values(own, v_first, w["vmix"])
    window = (m.get("mask") or {}).get("size")
    o = torch.zeros(T, H, dv, dtype=F64)
    for a in range(H):
        g = a // (H // G)
        for i in range(T):
            lo, hi = visible(i, window)
            s = (k[lo:hi, g] @ q[i, a]) * m["scale"]
            s = s - distance_penalty(w["r1"][a], w["r2"][a], i - torch.arange(lo, hi, dtype=F64))
            o[i, a] = weights_with_sink(s, w["sink"][a]) @ v[lo:hi, g]
    return lin(w["o"], o.reshape(T, H * dv)), own


def stretched_frequencies(rot):
    """The angle a position adds for each pair of rotated dimensions, and the factor on cos and sin."""
    n, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0

    def dim_of(turns):
        return n * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(dim_of(sc["fast"])), 0), min(math.ceil(dim_of(sc["slow"])), n - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / sc["factor"] * ramp + fi * (1.0 - ramp))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate_halves(x, rot):
    """x [T, heads, n]: dimension i turns with i + dims/2 by position * frequency i; what lies beyond dims passes."""
    f, mult = stretched_frequencies(rot)
    half = rot["dims"] // 2
    pos = torch.arange(x.shape[0], dtype=F64)
    out = x.clone()
    for i in range(half):
        c, s = mult * torch.cos(pos * f[i])[:, None], mult * torch.sin(pos * f[i])[:, None]
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * c - v * s
        out[..., i + half] = v * c + u * s
    return out


def latent_attention(h, w, m, eps):
    """Keys and values of every head made from one normed vector per token, beside one rotated key part all heads share;
    queries made from a vector of their own; a sink."""
    T = h.shape[0]
    H, d, dr, dv, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = lin(w["uq"], rms_unit(lin(w["dq"], h), eps) * w["dq.norm"]).view(T, H, d + dr)
    down = lin(w["dkv"], h)
    c = rms_unit(down[:, :r], eps) * w["dkv.norm"]
    q_rot = rotate_halves(q[..., d:], m["rot"])
    k_rot = rotate_halves(down[:, None, r:], m["rot"])[:, 0]
    k = lin(w["uk"], c).view(T, H, d)
    v = lin(w["uv"], c).view(T, H, dv)
    o = torch.zeros(T, H, dv, dtype=F64)
    for a in range(H):
        for i in range(T):
            s = (k[:i + 1, a] @ q[i, a, :d] + k_rot[:i + 1] @ q_rot[i, a]) * m["scale"]
            o[i, a] = weights_with_sink(s, w["sink"][a]) @ v[:i + 1, a]
    return lin(w["o"], o.reshape(T, H * dv))


def capped_feed_forward(h, w, limit):
    g = torch.clamp(lin(w["gate"], h), max=limit)
    u = torch.clamp(lin(w["up"], h), -limit, limit)
    return lin(w["down"], g * torch.sigmoid(1.702 * g) * (u + 1.0))


def sub(weights, prefix):
    return {k[len(prefix):]: t.to(F64) for k, t in weights.items() if k.startswith(prefix)}


def forward(config, weights, tokens, return_layers=False):
    """Logits [T, vocab] of one sequence (float64); with ``return_layers`` also the residual stream after every layer."""
    eps, groups = config["norm"]["eps"], config["norm"]["groups"]
    x = weights["embed"].to(F64)[torch.as_tensor(tokens, dtype=torch.long)]
    v_first, layers = None, []

    def normed(y, name):
        return grouped_norm(y, weights[name].to(F64), groups, eps)
    for i, layer in enumerate(config["layers"]):
        w, m = sub(weights, f"l{i}.mix."), layer["mixer"]
        h = normed(x, f"l{i}.norm1")
        if layer["type"] == "attention":
            mixes = bool(m.get("v_mix"))
            y, own = window_attention(h, w, m, eps, v_first if mixes else None)
            if mixes and v_first is None:
                v_first = own
        else:
            y = latent_attention(h, w, m, eps)
        x = x + normed(y, f"l{i}.norm1b")
        if layer.get("mlp") is not None:
            y = capped_feed_forward(normed(x, f"l{i}.norm2"), sub(weights, f"l{i}.mlp."), layer["mlp"]["limit"])
            x = x + normed(y, f"l{i}.norm2b")
        layers.append(x)
    logits = lin(weights["head"].to(F64), normed(x, "final.norm"))
    return (logits, torch.stack(layers)) if return_layers else logits
