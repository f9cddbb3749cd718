"""Plain double-precision Vogunex model over checkpoint tensors by name, one function per mechanism, one sequence at a time
and without any cache: every function sees the whole sequence.  Works on the `config.json` object; shares no code with the
package."""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def token_shift(h, s):
    """Every row moves towards the row before it (zeros before the first)."""
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * s


def angles(n, base, dims):
    return torch.arange(n, dtype=torch.float64)[:, None] * base ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / max(dims, 1))


def rotate_halves(x, base, dims):
    """x [n, heads, d]: dimension i turns with i + dims / 2."""
    a = angles(x.shape[0], base, dims)[:, None]
    u, v = x[..., :dims // 2], x[..., dims // 2:dims]
    return torch.cat([u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a), x[..., dims:]], -1)


def rotate_pairs(x, base, dims):
    """x [n, heads, d]: dimension 2 i turns with 2 i + 1."""
    a = angles(x.shape[0], base, dims)[:, None]
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * torch.cos(a) - v * torch.sin(a)
    out[..., 1:dims:2] = v * torch.cos(a) + u * torch.sin(a)
    return out


def window(n, size):
    """[n, n] visibility of the key at j for the query at i."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None]
    return (j <= i) & (i - j < size)


def pooled_visible(n, size, pool):
    """[n, blocks]: a block of `pool` tokens is seen once it lies wholly before the window."""
    i, b = torch.arange(n)[:, None], torch.arange(n // pool)[None]
    return b * pool + pool - 1 <= i - size


def block_means(x, pool):
    """[n, ...] -> [n // pool, ...]"""
    m = x.shape[0] // pool
    return x[:m * pool].reshape(m, pool, *x.shape[1:]).mean(1)


def softcap(s, cap):
    return cap * torch.tanh(s / cap) if cap else s


def mixed_weights(w, T):
    """weight_h <- sum_g T[h, g] weight_g, w [H, ...]."""
    out = torch.zeros_like(w)
    for h in range(w.shape[0]):
        for g in range(w.shape[0]):
            out[h] += T[h, g] * w[g]
    return out


def pooled_attention(h, T, p, m, eps):
    n, H, G, dim, vdim = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    proj = lambda name: h @ T(p + name).T + T(p + name + ".b")
    base, dims = m["rot"]["base"], m["rot"]["dims"]
    q = rms(rotate_halves(proj("q").view(n, H, dim), base, dims), eps)
    k = rms(rotate_halves(proj("k").view(n, G, dim), base, dims), eps)
    v = proj("v").view(n, G, vdim)
    P, size = m["mask"]["pool"], m["mask"]["size"]
    keys, values = torch.cat([block_means(k, P), k]), torch.cat([block_means(v, P), v])
    seen = torch.cat([pooled_visible(n, size, P), window(n, size)], 1)
    weights = []
    for head in range(H):
        s = softcap(q[:, head] @ keys[:, head // (H // G)].T * m["scale"], m.get("softcap"))
        weights.append(torch.softmax(s.masked_fill(~seen, -math.inf), -1))
    weights = mixed_weights(torch.stack(weights), T(p + "talk"))
    o = torch.cat([weights[head] @ values[:, head // (H // G)] for head in range(H)], -1)
    return o @ T(p + "o").T


def latent_attention(h, T, p, m, eps):
    n, H, dim, R, vdim, C = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    base = m["rot"]["base"]
    q = ((rms(h @ T(p + "dq").T, eps) * T(p + "dq.norm")) @ T(p + "uq").T).view(n, H, dim + R)
    down = h @ T(p + "dkv").T
    c = rms(down[:, :C], eps) * T(p + "dkv.norm")
    k_rot = rotate_pairs(down[:, None, C:], base, R)[:, 0]
    q_rot = rotate_pairs(q[..., dim:], base, R)
    k = (c @ T(p + "uk").T).view(n, H, dim)
    v = (c @ T(p + "uv").T).view(n, H, vdim)
    seen = window(n, m["mask"]["size"])
    gate = torch.sigmoid(h @ T(p + "g").T)
    o = []
    for head in range(H):
        s = (q[:, head, :dim] @ k[:, head].T + q_rot[:, head] @ k_rot.T) * m["scale"]
        o.append(torch.softmax(s.masked_fill(~seen, -math.inf), -1) @ v[:, head] * gate[:, head:head + 1])
    return torch.cat(o, -1) @ T(p + "o").T


def causal_conv(x, w, b):
    """x [n, channels], w [channels, taps]: the last tap is the row's own."""
    taps, n = w.shape[1], x.shape[0]
    xs = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x])
    return sum(xs[t:t + n] * w[:, t] for t in range(taps)) + b


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    return torch.log1p(torch.exp(-x.abs())) + x.clamp(min=0)


def scalar_decay_scan(x, B, C, dt, A, D):
    """x [n, H, V], B / C [n, G, N], dt [n, H]: the state of head h is [N, V]."""
    n, H, V = x.shape
    G, N = B.shape[1:]
    S, out = torch.zeros(H, N, V, dtype=x.dtype), torch.zeros_like(x)
    for t in range(n):
        for h in range(H):
            g = h // (H // G)
            S[h] = torch.exp(A[h] * dt[t, h]) * S[h] + dt[t, h] * torch.outer(B[t, g], x[t, h])
            out[t, h] = S[h].T @ C[t, g] + D[h] * x[t, h]
    return out


def part_norm(y, parts, eps):
    return torch.cat([rms(c, eps) for c in y.chunk(parts, -1)], -1)


def mamba2(h, T, p, m, eps):
    n, H, V, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * V
    z, xbc, dt = (h @ T(p + "in").T).split([inner, inner + 2 * G * N, H], -1)
    xbc = silu(causal_conv(xbc, T(p + "conv"), T(p + "conv.b")))
    x, B, C = xbc.split([inner, G * N, G * N], -1)
    y = scalar_decay_scan(x.reshape(n, H, V), B.reshape(n, G, N), C.reshape(n, G, N), softplus(dt + T(p + "dt_bias")),
                          -torch.exp(T(p + "A_log")), T(p + "D")).reshape(n, inner)
    return (part_norm(y * silu(z), m["norm_groups"], eps) * T(p + "norm")) @ T(p + "o").T


def gelu(z):
    return 0.5 * z * (1 + torch.erf(z / math.sqrt(2)))


def dense_ff(x, T, p):
    return gelu(x @ T(p + "up").T + T(p + "up.b")) @ T(p + "down").T + T(p + "down.b")


def expert(x, T, p, limit):
    g, u = (x @ T(p + "gate").T).clamp(max=limit), (x @ T(p + "up").T).clamp(-limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ T(p + "down").T


def route(z, top):
    """Weights of the experts [n, experts]: softmax over the `top` largest logits of a row, zero elsewhere."""
    val, idx = z.topk(top, -1)
    return torch.zeros_like(z).scatter(-1, idx, torch.softmax(val, -1))


def moe_ff(x, T, p, m):
    w = route(x @ T(p + "router").T + T(p + "router.b"), m["router"]["top"])
    out = torch.zeros_like(x)
    for e in range(m["router"]["experts"]):
        rows = w[:, e] > 0
        out[rows] += w[rows, e:e + 1] * expert(x[rows], T, f"{p}e{e}.", m["expert"]["limit"])
    if m.get("shared"):
        out = out + torch.sigmoid(x @ T(p + "shared.sg").T) * expert(x, T, p + "shared.", m["shared"]["limit"])
    return out


MIXERS = {"attention": pooled_attention, "latent_attention": latent_attention, "mamba2": mamba2}


def owner(layers, i):
    """The layer whose tensors layer i uses."""
    while layers[i].get("weights_of") is not None:
        i = layers[i]["weights_of"]
    return i


class Oracle:
    def __init__(self, config, tensors):
        self.c, self.cache, self.tensors = config, {}, tensors

    def T(self, name):
        if name not in self.cache:
            self.cache[name] = self.tensors(name).double().cpu()
        return self.cache[name]

    def layers(self, tokens):
        """Residual stream after every layer."""
        c, T, eps = self.c, self.T, self.c["norm"]["eps"]
        x = T("embed")[torch.tensor(tokens)] * c["embedding"]["scale"]
        out = []
        for i, l in enumerate(c["layers"]):
            p = f"l{owner(c['layers'], i)}."
            h = token_shift(rms(x, eps) * T(p + "norm1"), T(p + "shift"))
            x = x + MIXERS[l["type"]](h, T, p + "mix.", l["mixer"], eps)
            if l["mlp"]:
                h = rms(x, eps) * T(p + "norm2")
                x = x + (dense_ff(h, T, p + "mlp.") if l["mlp"]["kind"] == "dense" else moe_ff(h, T, p + "mlp.", l["mlp"]))
            out.append(x)
        return out

    def logits(self, tokens):
        key = tuple(tokens)
        if key not in self.cache:
            x = self.layers(tokens)[-1]
            self.cache[key] = (rms(x, self.c["norm"]["eps"]) * self.T("final.norm")) @ self.T("head").T
        return self.cache[key]

    def greedy(self, prompt, n):
        seq = list(prompt)
        for _ in range(n):
            seq.append(int(self.logits(seq)[-1].argmax()))
        return seq[len(prompt):]
