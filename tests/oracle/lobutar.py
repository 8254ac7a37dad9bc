"""A slow, literal implementation of the Lobutar decoder for the tests: one function per mechanism, one token or one
score at a time where that is the clearest form, float64 by default.  It works on the checkpoint's own tensors (a plain
dict of name -> tensor) and on the configuration dict, and shares no code with ``gcore_b200``."""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def project(W, name, h):
    y = h @ W[name].T
    return y + W[name + ".b"] if name + ".b" in W else y


# ------------------------------------------------------------------------------------------------ rotation
def rotate(x, rot, positions):
    """Rotates the first ``rot['dims']`` dimensions of the last axis of ``x`` [T, ..., n], neighbours paired."""
    y = x.clone()
    for i in range(rot["dims"] // 2):
        a = torch.tensor([p * rot["base"] ** (-2.0 * i / rot["dims"]) for p in positions], dtype=torch.float64)
        c, s = (f(a).to(x.dtype).view(-1, *[1] * (x.dim() - 2)) for f in (torch.cos, torch.sin))
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i] = u * c - v * s
        y[..., 2 * i + 1] = v * c + u * s
    return y


# ------------------------------------------------------------------------------------------------ attention
def visible(i, window=0):
    """Keys that position i sees: all up to itself, or the last ``window`` of them."""
    return range(max(0, i - window + 1) if window else 0, i + 1)


def softmax_with_sink(s, sink=None):
    """Weights of scores ``s``; a sink takes its share of the denominator and nothing else."""
    m = s.max() if sink is None else torch.maximum(s.max(), sink)
    e = torch.exp(s - m)
    return e / (e.sum() + (torch.exp(sink - m) if sink is not None else 0.0))


def attend(q, k, v, scale, window=0, sink=None):
    """One head over one sequence: q, k [T, d], v [T, dv]."""
    out = torch.zeros(q.shape[0], v.shape[1], dtype=q.dtype)
    for i in range(q.shape[0]):
        j = list(visible(i, window))
        out[i] = softmax_with_sink(k[j] @ q[i] * scale, sink) @ v[j]
    return out


def difference_weight(lq1, lk1, lq2, lk2, diff):
    return math.exp(float(lq1 @ lk1)) - math.exp(float(lq2 @ lk2)) + diff


def combine_maps(a1, a2, lam, diff, eps):
    return rms(a1 - lam * a2, eps) * (1 - diff)


def differential_attention(W, name, m, h, eps):
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rotate(project(W, name + ".q", h).view(T, H, 2, d), m["rot"], range(T))
    k = rotate(project(W, name + ".k", h).view(T, G, 2, d), m["rot"], range(T))
    v = project(W, name + ".v", h).view(T, G, dv)
    gate = torch.sigmoid(h @ W[name + ".g"].T)
    lam = difference_weight(*(W[f"{name}.{n}"] for n in ("lq1", "lk1", "lq2", "lk2")), m["diff"])
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for a in range(H):
        g = a // (H // G)
        a1, a2 = (attend(q[:, a, i], k[:, g, i], v[:, g], m["scale"]) for i in range(2))
        out[:, a] = combine_maps(a1, a2, lam, m["diff"], eps) * gate[:, a:a + 1]
    return project(W, name + ".o", out.reshape(T, H * dv))


def latent_attention(W, name, m, h, eps):
    T, H, d, r, dv, C = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = project(W, name + ".q", h).view(T, H, d + r)
    down = h @ W[name + ".dkv"].T
    c = rms(down[:, :C], eps) * W[name + ".dkv.norm"]
    kr = rotate(down[:, C:], m["rot"], range(T))
    qr = rotate(q[:, :, d:], m["rot"], range(T))
    k = (c @ W[name + ".uk"].T).view(T, H, d)
    v = (c @ W[name + ".uv"].T).view(T, H, dv)
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for a in range(H):
        out[:, a] = attend(torch.cat([q[:, a, :d], qr[:, a]], -1), torch.cat([k[:, a], kr], -1), v[:, a], m["scale"],
                           m["mask"]["size"], W[name + ".sink"][a])
    return (out.reshape(T, H * dv) * torch.sigmoid(h @ W[name + ".g"].T)) @ W[name + ".o"].T


# ------------------------------------------------------------------------------------------------ feed-forward
def gated_ffn(W, name, h):
    return (silu(h @ W[name + ".gate"].T) * (h @ W[name + ".up"].T)) @ W[name + ".down"].T


def choose_experts(z, correction, router):
    """[(expert, weight)] of one token's router logits."""
    E, groups = len(z), router.get("groups")
    s = torch.sigmoid(z)
    choice = [float(s[e] + correction[e]) for e in range(E)]
    allowed = list(range(E))
    if groups:
        n = E // groups["count"]
        score = {g: sum(sorted(choice[g * n:(g + 1) * n])[-2:]) for g in range(groups["count"])}
        kept = sorted(score, key=lambda g: -score[g])[:groups["keep"]]
        allowed = [e for e in allowed if e // n in kept]
    best = sorted(allowed, key=lambda e: -choice[e])[:router["top"]]
    return [(e, float(s[e]) * router.get("scale", 1.0)) for e in best]


def mixture(W, name, m, h):
    out = torch.zeros_like(h)
    z = h @ W[name + ".router"].T
    for t in range(h.shape[0]):
        for e, w in choose_experts(z[t], W[name + ".correction"], m["router"]):
            out[t] += w * gated_ffn(W, f"{name}.e{e}", h[t])
    return out + gated_ffn(W, name + ".shared", h) if m.get("shared") else out


# ------------------------------------------------------------------------------------------------ decoder
MIXERS = {"attention": differential_attention, "latent_attention": latent_attention}


def read_streams(weights, streams):
    """Weighted sum of the streams [S, T, w]."""
    return sum(weights[s] * streams[s] for s in range(len(streams)))


def write_streams(mix, out, streams, y):
    """Every stream from all the old ones (``mix`` is indexed [from, to]) and the sublayer's output."""
    S = len(streams)
    return torch.stack([sum(mix[s, t] * streams[s] for s in range(S)) + out[t] * y for t in range(S)])


def owner(config, i):
    """The layer whose tensors layer i uses."""
    while "weights_of" in config["layers"][i]:
        i = config["layers"][i]["weights_of"]
    return i


def sublayer(W, name, which, streams, eps, run):
    hc = f"{name}.hc{which}."
    u = read_streams(W[hc + "in"], streams)
    return write_streams(W[hc + "mix"], W[hc + "out"], streams, run(rms(u, eps) * W[f"{name}.norm{which}"]))


def layer(W, name, spec, streams, eps):
    streams = sublayer(W, name, 1, streams, eps,
                       lambda h: MIXERS[spec["type"]](W, name + ".mix", spec["mixer"], h, eps))
    mlp = spec.get("mlp")
    if mlp is None:
        return streams
    ff = (lambda h: gated_ffn(W, name + ".mlp", h)) if mlp["kind"] == "dense" else \
        (lambda h: mixture(W, name + ".mlp", mlp, h))
    return sublayer(W, name, 2, streams, eps, ff)


def forward(W, config, tokens, dtype=torch.float64, collect=None):
    """Logits [T, vocab] of one whole sequence; ``collect`` (a list) receives the streams' sum after every layer."""
    W = {k: v.to(dtype) for k, v in W.items()}
    eps = config["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    streams = torch.stack([x] * config["streams"])
    for i, spec in enumerate(config["layers"]):
        streams = layer(W, f"l{owner(config, i)}", spec, streams, eps)
        if collect is not None:
            collect.append(streams.sum(0))
    return (rms(streams.sum(0), eps) * W["final.norm"]) @ W["head"].T


# ------------------------------------------------------------------------------------------------ random weights
def random_weights(config, seed=0, scale=1.0):
    """Small random weights for a configuration, in the checkpoint's layout and precision."""
    g = torch.Generator().manual_seed(seed)

    def r(*shape, std=1.0):
        return (torch.randn(*shape, generator=g) * std).to(torch.bfloat16)

    w, V, S = config["width"], config["vocab"], config["streams"]
    s = scale / math.sqrt(w)
    W = {"embed": r(V, w), "final.norm": 1 + r(w, std=0.1), "head": r(V, w, std=w ** -0.5)}
    for i, sp in enumerate(config["layers"]):
        if "weights_of" in sp:
            continue
        n, m, f = f"l{i}", sp["mixer"], sp.get("mlp")
        for q in (1,) if f is None else (1, 2):
            W[f"{n}.norm{q}"] = 1 + r(w, std=0.1)
            W[f"{n}.hc{q}.in"] = 1 / S + r(S, std=0.3)
            W[f"{n}.hc{q}.out"] = 1 + r(S, std=0.3)
            W[f"{n}.hc{q}.mix"] = torch.eye(S).to(torch.bfloat16) + r(S, S, std=0.2)
        H, mix = m["heads"], n + ".mix."
        if sp["type"] == "attention":
            G, d, dv = m["kv_heads"], m["dim"], m["vdim"]
            for nm, rows, std in (("q", H * 2 * d, 2 * s), ("k", G * 2 * d, 2 * s), ("v", G * dv, s)):
                W[mix + nm], W[mix + nm + ".b"] = r(rows, w, std=std), r(rows, std=0.3)
            for nm in ("lq1", "lk1", "lq2", "lk2"):
                W[mix + nm] = r(d, std=0.6 * d ** -0.5)
            W[mix + "g"] = r(H, w, std=s)
            W[mix + "o.b"] = r(w, std=0.1)
        else:
            C, dv = m["kv_rank"], m["vdim"]
            W[mix + "q"] = r(H * (m["dim"] + m["rot_dim"]), w, std=2 * s)
            W[mix + "dkv"] = r(C + m["rot_dim"], w, std=s)
            W[mix + "dkv.norm"] = 1 + r(C, std=0.1)
            W[mix + "uk"], W[mix + "uv"] = r(H * m["dim"], C, std=C ** -0.5), r(H * dv, C, std=C ** -0.5)
            W[mix + "sink"] = r(H)
            W[mix + "g"] = r(H * dv, w, std=s)
        W[mix + "o"] = r(w, H * dv, std=(H * dv) ** -0.5)
        if f is None:
            continue
        mlp = n + ".mlp."
        if f["kind"] == "dense":
            parts = [("", f["ff"])]
        else:
            E = f["router"]["experts"]
            parts = [(f"e{e}.", f["expert"]["ff"]) for e in range(E)] + \
                ([("shared.", f["shared"]["ff"])] if f.get("shared") else [])
            W[mlp + "router"], W[mlp + "correction"] = r(E, w, std=2 * s), r(E, std=0.2)
        for nm, ff in parts:
            W[mlp + nm + "gate"], W[mlp + nm + "up"] = r(ff, w, std=s), r(ff, w, std=s)
            W[mlp + nm + "down"] = r(w, ff, std=ff ** -0.5)
    return W
