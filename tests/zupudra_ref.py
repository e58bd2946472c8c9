"""Plain evaluation of the Zupudra decoder in numpy, one function per mechanism.

Everything is token by token and head by head in the order of the equations, in the float type of
the inputs (the tests use float64), with no code shared with the package under test.
"""
import numpy as np


def rms(x, eps):
    return x / np.sqrt(np.mean(x * x) + eps)


def rms_norm(x, w, eps):
    return rms(x, eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.log1p(np.exp(-np.abs(z))) + np.maximum(z, 0.0)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def rotate_half(v, position, dims, base):
    """Rotates (v[i], v[i + dims/2]) by position * base^(-2i/dims) for i < dims/2; v[dims:] stays."""
    out = v.copy()
    half = dims // 2
    for i in range(half):
        a = position * base ** (-2.0 * i / dims)
        c, s = np.cos(a), np.sin(a)
        out[i] = v[i] * c - v[i + half] * s
        out[i + half] = v[i + half] * c + v[i] * s
    return out


def retention_state(S, k, v, decay):
    return decay * S + np.outer(k, v)


def retention(h, w, m, eps, state, position):
    """One token of the fixed-decay linear attention. state: [heads, dim, vdim], updated in place."""
    H, D, E = m["heads"], m["dim"], m["vdim"]
    q, k, v = w["q"] @ h, w["k"] @ h, w["v"] @ h
    out = []
    for n in range(H):
        qn = rotate_half(q[n * D:(n + 1) * D], position, m["rot"]["dims"], m["rot"]["base"])
        kn = rotate_half(k[n * D:(n + 1) * D], position, m["rot"]["dims"], m["rot"]["base"]) * D ** -0.5
        state[n] = retention_state(state[n], kn, v[n * E:(n + 1) * E], m["decay"][n])
        out.append(rms(state[n].T @ qn, eps))
    return w["o"] @ (np.concatenate(out) * silu(w["g"] @ h))


def causal_conv(x, tail, w, b):
    """One token of a per-channel causal convolution. tail: [taps - 1, channels], oldest first, updated."""
    taps = np.concatenate([tail, x[None]], 0)
    if len(tail):
        tail[:] = taps[1:]
    return (taps * w.T).sum(0) + b


def rglru_gates(u, w, blocks):
    n = len(u) // blocks
    r, i = np.empty_like(u), np.empty_like(u)
    for b in range(blocks):
        s = slice(b * n, (b + 1) * n)
        r[s] = sigmoid(w["ra"][b] @ u[s] + w["ra.b"][b])
        i[s] = sigmoid(w["ri"][b] @ u[s] + w["ri.b"][b])
    return r, i


def rglru_state(S, u, r, i, lam):
    a = np.exp(-8.0 * r * softplus(lam))
    return a * S + np.sqrt(1.0 - a * a) * i * u


def rglru(h, w, m, state, tail):
    """One token of the gated recurrent block. state: [width], tail: [conv - 1, width], updated in place."""
    y = gelu_tanh(w["y"] @ h + w["y.b"])
    u = causal_conv(w["x"] @ h + w["x.b"], tail, w["conv"], w["conv.b"])
    r, i = rglru_gates(u, w, m["blocks"])
    state[:] = rglru_state(state, u, r, i, w["lam"])
    return w["o"] @ (state * y)


def softmax(s):
    e = np.exp(s - s.max())
    return e / e.sum()


def latent_attention(h, w, m, eps, latents):
    """One token of the attention over cached latents; `latents` (a list) grows by this token's."""
    H, D, E = m["heads"], m["dim"], m["vdim"]
    latents.append(rms_norm(w["dkv"] @ h, w["dkv.norm"], eps))
    q = w["q"] @ h
    c = np.stack(latents)
    out = []
    for n in range(H):
        k = c @ w["uk"][n * D:(n + 1) * D].T
        v = c @ w["uv"][n * E:(n + 1) * E].T
        p = softmax((k @ q[n * D:(n + 1) * D]) * m["scale"])
        out.append(p @ v)
    return w["o"] @ (np.concatenate(out) * sigmoid(w["g"] @ h))


def gated_ff(x, w):
    return w["down"] @ (silu(w["gate"] @ x) * (w["up"] @ x))


def new_state(layer, dtype=np.float64):
    m = layer["mixer"]
    if layer["type"] == "retention":
        return {"S": np.zeros((m["heads"], m["dim"], m["vdim"]), dtype)}
    if layer["type"] == "rglru":
        return {"S": np.zeros(m["width"], dtype), "tail": np.zeros((m["conv"] - 1, m["width"]), dtype)}
    return {"latents": []}


class Model:
    """config: the parsed config.json; tensors: name -> array. `forward` continues where it stopped."""

    def __init__(self, config, tensors, dtype=np.float64):
        self.config = config
        self.t = {k: np.asarray(v, dtype) for k, v in tensors.items()}
        self.dtype = dtype
        self.eps = config["norm"]["eps"]
        self.owner = []
        for i, layer in enumerate(config["layers"]):
            self.owner.append(i)
            while "weights_of" in config["layers"][self.owner[i]]:
                self.owner[i] = config["layers"][self.owner[i]]["weights_of"]
        self.reset()

    def reset(self):
        self.position = 0
        self.state = [new_state(layer, self.dtype) for layer in self.config["layers"]]

    def part(self, i, kind):
        p = f"l{self.owner[i]}.{kind}."
        return {k[len(p):]: v for k, v in self.t.items() if k.startswith(p)}

    def layer(self, i, x):
        layer, st, l = self.config["layers"][i], self.state[i], f"l{self.owner[i]}."
        h = rms_norm(x, self.t[l + "norm1"], self.eps)
        w = self.part(i, "mix")
        if layer["type"] == "retention":
            x = x + retention(h, w, layer["mixer"], self.eps, st["S"], self.position)
        elif layer["type"] == "rglru":
            x = x + rglru(h, w, layer["mixer"], st["S"], st["tail"])
        else:
            x = x + latent_attention(h, w, layer["mixer"], self.eps, st["latents"])
        if layer.get("mlp"):
            x = x + gated_ff(rms_norm(x, self.t[l + "norm2"], self.eps), self.part(i, "mlp"))
        return x

    def forward(self, tokens, trace=None):
        """Logits of every token, [tokens, vocab]; trace (a list) receives [layers, width] per token."""
        out = []
        for tok in tokens:
            x = self.t["embed"][tok]
            rows = []
            for i in range(len(self.config["layers"])):
                x = self.layer(i, x)
                rows.append(x)
            if trace is not None:
                trace.append(np.stack(rows))
            out.append(self.t["embed"] @ rms_norm(x, self.t["final.norm"], self.eps))
            self.position += 1
        return np.stack(out)
