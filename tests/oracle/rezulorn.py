"""A slow, literal implementation of the Rezulorn decoder for the tests: one function per mechanism, one token or one
score at a time where that is the clearest form, float64 by default.  It works on the checkpoint's own tensors (a plain
dict of name -> tensor) and on the configuration dict, and shares no code with ``gcore_b200``."""
import math

import torch


def silu(z):
    return z * torch.sigmoid(z)


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, w, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def input_conv(h, w):
    """``h`` [T, width] plus a causal convolution over time of each channel; the last tap is the present."""
    T, n = h.shape[0], w.shape[1]
    out = h.clone()
    for t in range(T):
        for j in range(n):
            s = t - n + 1 + j
            if s >= 0:
                out[t] = out[t] + w[:, j] * h[s]
    return out


# ------------------------------------------------------------------------------------------------ positions
def rotate(x, rot, positions):
    """Rotates the first ``rot['dims']`` dimensions of the last axis of ``x`` [T, heads, n]: dimension i turns together with
    dimension i + dims / 2."""
    y, half = x.clone(), rot["dims"] // 2
    slow = rot["scaling"]["factor"] if rot.get("scaling") else 1.0
    for i in range(half):
        a = torch.tensor([p * rot["base"] ** (-2.0 * i / rot["dims"]) / slow for p in positions], dtype=torch.float64)
        c, s = (f(a).to(x.dtype)[:, None] for f in (torch.cos, torch.sin))
        u, v = x[..., i], x[..., i + half]
        y[..., i] = u * c - v * s
        y[..., i + half] = v * c + u * s
    return y


def distance_penalty(d, r1, r2):
    return r1 * torch.log(1 + r2 * d)


def visible(i, mask=None):
    """Keys that position i sees: all up to itself, or those inside the window and the first ones."""
    return [j for j in range(i + 1) if mask is None or i - j < mask["size"] or j < mask["keep_first"]]


# ------------------------------------------------------------------------------------------------ mixers
def softmax_attention(q, k, v, scale, mask, r1, r2):
    """One head over one sequence: q, k [T, d], v [T, dv]."""
    out = torch.zeros(q.shape[0], v.shape[1], dtype=q.dtype)
    for i in range(q.shape[0]):
        j = visible(i, mask)
        d = torch.tensor([i - x for x in j], dtype=q.dtype)
        out[i] = torch.softmax(k[j] @ q[i] * scale - distance_penalty(d, r1, r2), -1) @ v[j]
    return out


def sigmoid_attention(q, k, v, scale, bias):
    out = torch.zeros(q.shape[0], v.shape[1], dtype=q.dtype)
    for i in range(q.shape[0]):
        j = visible(i)
        out[i] = torch.sigmoid(k[j] @ q[i] * scale + bias) @ v[j]
    return out


def fading_memory(q, k, v, decay):
    """One head of linear attention with a fixed decay, token by token: q, k [T, d], v [T, dv]."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype)
    out = torch.zeros(q.shape[0], v.shape[1], dtype=q.dtype)
    for t in range(q.shape[0]):
        S = decay * S + torch.outer(k[t], v[t])
        out[t] = S.T @ q[t]
    return out


def heads_of(W, name, h, n):
    return (h @ W[name].T).view(h.shape[0], n, -1)


def attention(W, p, m, h, eps):
    H, G = m["heads"], m["kv_heads"]
    q, k, v = heads_of(W, p + "q", h, H), heads_of(W, p + "k", h, G), heads_of(W, p + "v", h, G)
    out = [softmax_attention(q[:, a], k[:, a // (H // G)], v[:, a // (H // G)], m["scale"], m["mask"], W[p + "r1"][a],
                             W[p + "r2"][a]) for a in range(H)]
    return torch.cat(out, -1) @ W[p + "o"].T


def gate_attention(W, p, m, h, eps):
    H, G, at = m["heads"], m["kv_heads"], range(h.shape[0])
    q, k = (rms(rotate(heads_of(W, p + n, h, c), m["rot"], at), eps) for n, c in (("q", H), ("k", G)))
    v = heads_of(W, p + "v", h, G)
    out = [sigmoid_attention(q[:, a], k[:, a // (H // G)], v[:, a // (H // G)], m["scale"], W[p + "pb"][a]) for a in range(H)]
    return torch.cat(out, -1) @ W[p + "o"].T


def retention(W, p, m, h, eps):
    H, at = m["heads"], range(h.shape[0])
    q, k = (rotate(heads_of(W, p + n, h, H), m["rot"], at) for n in "qk")
    v = heads_of(W, p + "v", h, H)
    out = [rms(fading_memory(q[:, a], k[:, a] * m["dim"] ** -0.5, v[:, a], m["decay"][a]), eps) for a in range(H)]
    return (torch.cat(out, -1) * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


def lightning(W, p, m, h, eps):
    H = m["heads"]
    q, k, v = (silu(heads_of(W, p + n, h, H)) for n in "qkv")
    o = torch.cat([fading_memory(q[:, a], k[:, a], v[:, a], m["decay"][a]) for a in range(H)], -1)
    return (rms(o, eps) * W[p + "norm"] * torch.sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def parallel(W, p, m, h, eps):
    return m["left_scale"] * gate_attention(W, p + "left.", m["left"], h, eps) + \
        m["right_scale"] * retention(W, p + "right.", m["right"], h, eps)


MIXERS = {"attention": attention, "lightning": lightning, "parallel": parallel}


def feed_forward(W, p, h):
    return torch.relu(h @ W[p + "up"].T) ** 2 @ W[p + "down"].T


# ------------------------------------------------------------------------------------------------ model
def forward(W, c, tokens, dtype=torch.float64):
    """Logits [T, vocab] of one sequence and the residual behind every layer."""
    W = {k: v.to(dtype) for k, v in W.items()}
    eps, mult = c["norm"]["eps"], c["residual_mult"]
    x, kept = W["embed"][torch.tensor(tokens)], []
    for i, ly in enumerate(c["layers"]):
        p = f"l{i}."
        h = input_conv(layer_norm(x, W[p + "norm1"], eps), W[p + "canon1"])
        x = x + mult * MIXERS[ly["type"]](W, p + "mix.", ly["mixer"], h, eps)
        if ly.get("mlp"):
            h = input_conv(layer_norm(x, W[p + "norm2"], eps), W[p + "canon2"])
            x = x + mult * feed_forward(W, p + "mlp.", h)
        kept.append(x)
    return layer_norm(x, W["final.norm"], eps) @ W["head"].T * c["logit_scale"], kept


def greedy(W, c, prompt, n):
    out = list(prompt)
    for _ in range(n):
        out.append(int(forward(W, c, out)[0][-1].argmax()))
    return out[len(prompt):]


# ------------------------------------------------------------------------------------------------ weights
def shapes(c):
    """name -> shape of every tensor of a checkpoint."""
    E, V = c["width"], c["vocab"]
    out = {"embed": (V, E), "final.norm": (E,), "head": (V, E)}

    def projections(p, **rows):
        for n, r in rows.items():
            out[p + n] = (r, E)

    for i, ly in enumerate(c["layers"]):
        p, m = f"l{i}.", ly["mixer"]
        for s in (1, 2):
            out[p + f"norm{s}"] = (E,)
            out[p + f"canon{s}"] = (E, c["canon"]["taps"])
        at = p + "mix."
        if ly["type"] == "lightning":
            n, k = m["heads"] * m["vdim"], m["heads"] * m["dim"]
            projections(at, q=k, k=k, v=n, g=n)
            out.update({at + "norm": (n,), at + "o": (E, n)})
        else:
            a = m if ly["type"] == "attention" else m["left"]
            left = at if ly["type"] == "attention" else at + "left."
            projections(left, q=a["heads"] * a["dim"], k=a["kv_heads"] * a["dim"], v=a["kv_heads"] * a["vdim"])
            out[left + "o"] = (E, a["heads"] * a["vdim"])
            for n in (("r1", "r2") if ly["type"] == "attention" else ("pb",)):
                out[left + n] = (a["heads"],)
            if ly["type"] == "parallel":
                r = m["right"]
                n, k = r["heads"] * r["vdim"], r["heads"] * r["dim"]
                projections(at + "right.", q=k, k=k, v=n, g=n)
                out[at + "right.o"] = (E, n)
        if ly.get("mlp"):
            out.update({p + "mlp.up": (ly["mlp"]["ff"], E), p + "mlp.down": (E, ly["mlp"]["ff"])})
    return out


def random_weights(c, seed=0):
    """Weights every mechanism shows in: convolutions as large as their input, penalties and biases of order one."""
    g = torch.Generator().manual_seed(seed)
    W = {}
    for name, shape in shapes(c).items():
        leaf, w = name.rsplit(".", 1)[-1], torch.randn(*shape, generator=g)
        if "norm" in leaf:
            w = 1 + 0.2 * w
        elif leaf.startswith("canon"):
            w = w * 0.4
        elif leaf in ("r1", "r2"):
            w = 0.3 + 0.7 * torch.rand(*shape, generator=g) if leaf == "r1" else 0.05 + torch.rand(*shape, generator=g)
        elif leaf == "pb":
            w = w * 0.5 - 2.0
        elif len(shape) == 2 and name != "embed":
            w = w / math.sqrt(shape[1])
        W[name] = w.to(torch.bfloat16)
    return W
