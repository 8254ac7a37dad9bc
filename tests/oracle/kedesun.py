"""A slow, literal implementation of the Kedesun decoder for the tests: one function per mechanism, one token or one
score at a time where that is the clearest form, float64 by default.  It works on the checkpoint's own tensors (a plain
dict of name -> tensor) and on the configuration dict, and shares no code with ``gcore_b200``."""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


# ------------------------------------------------------------------------------------------------ rotation
def frequencies(rot):
    """Angle per position of every rotated pair, and the factor both cosine and sine carry."""
    n, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0

    def place(turns):   # (fractional) pair index whose wavelength makes ``turns`` turns over the original length
        return n * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(place(sc["fast"])), 0)
    hi = min(math.ceil(place(sc["slow"])), n - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / sc["factor"] * r + fi * (1 - r))
    return out, 0.1 * math.log(sc["factor"]) + 1


def rotate(x, rot, positions):
    """Rotates neighbouring pairs of the last axis of ``x`` [T, ..., n]."""
    f, m = frequencies(rot)
    y = x.clone()
    for t, p in enumerate(positions):
        for i, fi in enumerate(f):
            c, s = m * math.cos(p * fi), m * math.sin(p * fi)
            u, v = x[t, ..., 2 * i], x[t, ..., 2 * i + 1]
            y[t, ..., 2 * i] = u * c - v * s
            y[t, ..., 2 * i + 1] = v * c + u * s
    return y


# ------------------------------------------------------------------------------------------------ mixers
def latent_attention(W, name, m, h, eps):
    T, H, d, r, dv, C = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ W[name + ".q"].T).view(T, H, d + r)
    down = h @ W[name + ".dkv"].T
    c = rms(down[:, :C], eps) * W[name + ".dkv.norm"]
    kr = rotate(down[:, C:], m["rot"], range(T))
    qr = rotate(q[:, :, d:], m["rot"], range(T))
    k = (c @ W[name + ".uk"].T).view(T, H, d)
    v = (c @ W[name + ".uv"].T).view(T, H, dv)
    gate = torch.sigmoid(h @ W[name + ".g"].T)
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for t in range(T):
        for a in range(H):
            s = (k[:t + 1, a] @ q[t, a, :d] + kr[:t + 1] @ qr[t, a]) * m["scale"]
            out[t, a] = torch.softmax(s, 0) @ v[:t + 1, a] * gate[t, a]
    return out.reshape(T, H * dv) @ W[name + ".o"].T


def retention_core(q, k, v, decay, state=None):
    """q, k [T, H, d], v [T, H, dv]; ``state`` [H, d, dv] is updated in place when given."""
    T, H, d = q.shape
    S = state if state is not None else torch.zeros(H, d, v.shape[-1], dtype=q.dtype)
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for t in range(T):
        for a in range(H):
            S[a] = decay[a] * S[a] + torch.outer(k[t, a] * d ** -0.5, v[t, a])
            out[t, a] = S[a].T @ q[t, a]
    return out


def retention(W, name, m, h, eps, state=None):
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    o = retention_core((h @ W[name + ".q"].T).view(T, H, d), (h @ W[name + ".k"].T).view(T, H, d),
                       (h @ W[name + ".v"].T).view(T, H, dv), m["decay"], state)
    return (rms(o, eps).reshape(T, H * dv) * silu(h @ W[name + ".g"].T)) @ W[name + ".o"].T


# ------------------------------------------------------------------------------------------------ feed-forward
def gated_ffn(W, name, h):
    return (silu(h @ W[name + ".gate"].T) * (h @ W[name + ".up"].T)) @ W[name + ".down"].T


def squared_relu_ffn(W, name, h):
    return torch.relu(h @ W[name + ".up"].T) ** 2 @ W[name + ".down"].T


def choose_experts(z, correction, top):
    """[(expert, weight)] of one token's router logits."""
    s = torch.softmax(z, 0)
    order = sorted(range(len(z)), key=lambda e: -float(s[e] + correction[e]))[:top]
    total = sum(float(s[e]) for e in order) + 1e-20
    return [(e, float(s[e]) / total) for e in order]


def mixture(W, name, m, h):
    out = torch.zeros_like(h)
    z = h @ W[name + ".router"].T
    for t in range(h.shape[0]):
        for e, w in choose_experts(z[t], W[name + ".correction"], m["router"]["top"]):
            out[t] += w * squared_relu_ffn(W, f"{name}.e{e}", h[t])
    if m.get("shared"):
        out = out + torch.sigmoid(h @ W[name + ".shared.sg"].T) * squared_relu_ffn(W, name + ".shared", h)
    return out


# ------------------------------------------------------------------------------------------------ decoder
MIXERS = {"latent_attention": latent_attention, "retention": retention}


def layer(W, i, spec, x, eps):
    """Mixer and feed-forward read the same normed input; the result in front of the depth average."""
    n = f"l{i}"
    h = rms(x, eps) * W[n + ".norm1"]
    y = x + MIXERS[spec["type"]](W, n + ".mix", spec["mixer"], h, eps)
    mlp = spec.get("mlp")
    if mlp is not None:
        y = y + (gated_ffn(W, n + ".mlp", h) if mlp["kind"] == "dense" else mixture(W, n + ".mlp", mlp, h))
    return y


def depth_average(weights, results):
    return sum(w * x for w, x in zip(weights, results))


def forward(W, config, tokens, dtype=torch.float64, collect=None):
    """Logits [T, vocab] of one whole sequence; ``collect`` (a list) receives what every layer hands on."""
    W = {k: v.to(dtype) for k, v in W.items()}
    eps = config["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    results = [x]
    for i, spec in enumerate(config["layers"]):
        results.append(layer(W, i, spec, x, eps))
        x = depth_average(W[f"l{i}.dwa"], results)
        if collect is not None:
            collect.append(x.clone())
    return (rms(x, eps) * W["final.norm"]) @ W["embed"].T


# ------------------------------------------------------------------------------------------------ random weights
def random_weights(config, seed=0, scale=1.0):
    """Small random weights for a configuration, in the checkpoint's layout and precision."""
    g = torch.Generator().manual_seed(seed)

    def r(*shape, std=1.0):
        return (torch.randn(*shape, generator=g) * std).to(torch.bfloat16)

    w, V = config["width"], config["vocab"]
    s = scale / math.sqrt(w)
    W = {"embed": r(V, w), "final.norm": 1 + r(w, std=0.1)}
    for i, sp in enumerate(config["layers"]):
        n, m, f = f"l{i}", sp["mixer"], sp.get("mlp")
        W[n + ".norm1"] = 1 + r(w, std=0.1)
        W[n + ".dwa"] = r(i + 2, std=0.3) + torch.tensor([0.0] * (i + 1) + [1.0]).to(torch.bfloat16)
        H, vd = m["heads"], m["heads"] * m["vdim"]
        mix = n + ".mix."
        if sp["type"] == "retention":
            W[mix + "q"], W[mix + "k"] = r(H * m["dim"], w, std=s), r(H * m["dim"], w, std=s)
            W[mix + "v"], W[mix + "g"] = r(vd, w, std=s), r(vd, w, std=s)
        else:
            C = m["kv_rank"]
            W[mix + "q"] = r(H * (m["dim"] + m["rot_dim"]), w, std=2 * s)
            W[mix + "dkv"] = r(C + m["rot_dim"], w, std=s)
            W[mix + "dkv.norm"] = 1 + r(C, std=0.1)
            W[mix + "uk"], W[mix + "uv"] = r(H * m["dim"], C, std=C ** -0.5), r(vd, C, std=C ** -0.5)
            W[mix + "g"] = r(H, w, std=s)
        W[mix + "o"] = r(w, vd, std=vd ** -0.5)
        if f is None:
            continue
        mlp = n + ".mlp."
        if f["kind"] == "dense":
            W[mlp + "gate"], W[mlp + "up"] = r(f["ff"], w, std=s), r(f["ff"], w, std=s)
            W[mlp + "down"] = r(w, f["ff"], std=f["ff"] ** -0.5)
            continue
        E = f["router"]["experts"]
        for nm, ff in [(f"e{e}.", f["expert"]["ff"]) for e in range(E)] + [("shared.", f["shared"]["ff"])]:
            W[mlp + nm + "up"], W[mlp + nm + "down"] = r(ff, w, std=s), r(w, ff, std=ff ** -0.5)
        W[mlp + "router"], W[mlp + "correction"] = r(E, w, std=2 * s), r(E, std=0.1)
        W[mlp + "shared.sg"] = r(1, w, std=s)
    return W
