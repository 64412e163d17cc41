"""Slow float64 NumPy statement of the Ragenex decoder, one function per mechanism, and makers of small random models.

Shares no code with the package: the tests compare the package's modules and kernels with these functions."""
import json

import numpy as np


# ------------------------------------------------------------------------------------------ mechanisms
def layer_norm(z, gain, eps):
    """(z - mean) / sqrt(var + eps) * gain over the last axis."""
    d = z - z.mean(-1, keepdims=True)
    return d / np.sqrt((d * d).mean(-1, keepdims=True) + eps) * gain


def rms_norm(z, gain, eps):
    return z / np.sqrt((z * z).mean(-1, keepdims=True) + eps) * gain


def silu(z):
    return z / (1.0 + np.exp(-z))


def embed(tokens, positions, table, pos_table):
    return table[np.asarray(tokens)] + pos_table[np.asarray(positions)]


def read_streams(streams, weights):
    """u [tokens, width] from streams [tokens, S, width]."""
    return sum(weights[s] * streams[:, s] for s in range(streams.shape[1]))


def write_streams(streams, mix, out, y):
    """Stream t becomes sum_s mix[s, t] * stream s + out[t] * y."""
    S = streams.shape[1]
    return np.stack([sum(mix[s, t] * streams[:, s] for s in range(S)) + out[t] * y for t in range(S)], axis=1)


def temperature(position, coef, every):
    return 1.0 + coef * np.log(np.floor((position + 1) / every) + 1.0)


def queries_and_keys(h, w_q, w_k, g_q, g_k, eps, positions, temp):
    """Normed over all heads at once; queries times the temperature of their position."""
    q, k = rms_norm(h @ w_q.T, g_q, eps), rms_norm(h @ w_k.T, g_k, eps)
    if temp is not None:
        q = q * np.array([temperature(p, temp["coef"], temp["every"]) for p in positions])[:, None]
    return q, k


def causal_attention(q, k, v, heads, kv_heads, scale, first=0):
    """q [queries, heads * dim], k / v [tokens, kv_heads * dim | * vdim]; query i sits at token first + i."""
    n_q, n_k = q.shape[0], k.shape[0]
    d, dv, group = q.shape[1] // heads, v.shape[1] // kv_heads, heads // kv_heads
    out = np.zeros((n_q, heads * dv))
    for h in range(heads):
        g = h // group
        kh, vh = k[:, g * d : (g + 1) * d], v[:, g * dv : (g + 1) * dv]
        for i in range(n_q):
            n = min(first + i + 1, n_k)
            s = kh[:n] @ q[i, h * d : (h + 1) * d] * scale
            e = np.exp(s - s.max())
            out[i, h * dv : (h + 1) * dv] = (e / e.sum()) @ vh[:n]
    return out


def decayed_recurrence(q, k, v, decay, state=None):
    """q / k [tokens, heads, dim], v [tokens, heads, vdim]: state = decay * state + k v^T, out = state^T q, token by token.  Returns
    (out [tokens, heads, vdim], the last state [heads, dim, vdim])."""
    n, H, d = q.shape
    state = np.zeros((H, d, v.shape[2])) if state is None else state.copy()
    out = np.zeros((n, H, v.shape[2]))
    for t in range(n):
        for h in range(H):
            state[h] = decay[h] * state[h] + np.outer(k[t, h], v[t, h])
            out[t, h] = q[t, h] @ state[h]
    return out, state


def gated_norm(o, gain, gate, eps):
    return rms_norm(o, gain, eps) / (1.0 + np.exp(-gate))


def clamped_glu(gate, up, limit):
    g, u = np.minimum(gate, limit), np.clip(up, -limit, limit)
    return g / (1.0 + np.exp(-1.702 * g)) * (u + 1.0)


# ------------------------------------------------------------------------------------------ model
def run_order(cfg):
    loop = cfg.get("loop")
    order = list(range(len(cfg["layers"])))
    if loop:
        a, b, n = loop["start"], loop["stop"], loop["times"]
        order = order[:a] + order[a:b] * n + order[b:]
    return order


def mixer(kind, m, w, a, h, eps, positions):
    n = h.shape[0]
    if kind == "attention":
        q, k = queries_and_keys(h, w[a + "q"], w[a + "k"], w[a + "q.norm"], w[a + "k.norm"], eps, positions, m.get("q_temp"))
        o = causal_attention(q, k, h @ w[a + "v"].T, m["heads"], m["kv_heads"], m["scale"])
        return o @ w[a + "o"].T
    q, k, v = (silu(h @ w[a + x].T).reshape(n, m["heads"], -1) for x in "qkv")
    o, _ = decayed_recurrence(q, k, v, m["decay"])
    return gated_norm(o.reshape(n, -1), w[a + "norm"], h @ w[a + "g"].T, eps) @ w[a + "o"].T


def forward(cfg, w, tokens, return_layers=False):
    """Logits [tokens, vocab] of one sequence (and the sum of the streams after every layer run)."""
    w = {k: np.asarray(v, dtype=np.float64) for k, v in w.items()}
    eps, S = cfg["norm"]["eps"], cfg["streams"]
    positions = list(range(len(tokens)))
    x = np.repeat(embed(tokens, positions, w["embed"], w["pos"])[:, None], S, axis=1)
    after = []
    for i in run_order(cfg):
        layer, a = cfg["layers"][i], f"l{i}."
        h = layer_norm(read_streams(x, w[a + "hc1.in"]), w[a + "norm1"], eps)
        y = mixer(layer["type"], layer["mixer"], w, a + "mix.", h, eps, positions)
        x = write_streams(x, w[a + "hc1.mix"], w[a + "hc1.out"], w[a + "ls1"] * y)
        if layer["mlp"] is not None:
            h = layer_norm(read_streams(x, w[a + "hc2.in"]), w[a + "norm2"], eps)
            y = clamped_glu(h @ w[a + "mlp.gate"].T, h @ w[a + "mlp.up"].T, layer["mlp"]["limit"]) @ w[a + "mlp.down"].T
            x = write_streams(x, w[a + "hc2.mix"], w[a + "hc2.out"], w[a + "ls2"] * y)
        after.append(x.sum(1))
    logits = layer_norm(x.sum(1), w["final.norm"], eps) @ w["head"].T
    return (logits, after) if return_layers else logits


def greedy(cfg, w, prompt, n):
    out = list(prompt)
    for _ in range(n):
        out.append(int(forward(cfg, w, out)[-1].argmax()))
    return out


# ------------------------------------------------------------------------------------------ small models
def attention_layer(heads=6, kv_heads=2, dim=24, vdim=40, scale=None, coef=0.4, every=5, ff=72, limit=0.8):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim**-0.5 if scale is None else scale, "q_temp": {"coef": coef, "every": every}}
    return {"type": "attention", "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


def lightning_layer(decay=(0.5, 0.9, 0.995), dim=16, vdim=24, ff=72, limit=0.8):
    m = {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)}
    return {"type": "lightning", "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


def config(layers, width=88, vocab=90, eps=1e-4, streams=3, loop=None, max_positions=512):
    cfg = {"architecture": "Ragenex", "layers": layers, "width": width, "vocab": vocab, "norm": {"eps": eps}, "streams": streams, "max_positions": max_positions}
    if loop is not None:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


def shapes(cfg):
    D, V, S = cfg["width"], cfg["vocab"], cfg["streams"]
    out = {"embed": (V, D), "pos": (cfg["max_positions"], D), "final.norm": (D,), "head": (V, D)}
    for i, l in enumerate(cfg["layers"]):
        a, m = f"l{i}.", l["mixer"]
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        G = m.get("kv_heads", H)
        out.update({a + "norm1": (D,), a + "ls1": (D,), a + "mix.q": (H * d, D), a + "mix.k": (G * d, D), a + "mix.v": (G * dv, D), a + "mix.o": (D, H * dv)})
        out.update({a + "mix.q.norm": (H * d,), a + "mix.k.norm": (G * d,)} if l["type"] == "attention" else {a + "mix.g": (H * dv, D), a + "mix.norm": (H * dv,)})
        if l["mlp"] is not None:
            ff = l["mlp"]["ff"]
            out.update({a + "norm2": (D,), a + "ls2": (D,), a + "mlp.gate": (ff, D), a + "mlp.up": (ff, D), a + "mlp.down": (D, ff)})
        for q in (1, 2) if l["mlp"] is not None else (1,):
            out.update({a + f"hc{q}.in": (S,), a + f"hc{q}.out": (S,), a + f"hc{q}.mix": (S, S)})
    return out


def bf16_exact(a):
    """Rounded to values bf16 holds exactly."""
    u = np.asarray(a, dtype=np.float32).view(np.uint32)
    u = (u + 0x7FFF + ((u >> 16) & 1)) & np.uint32(0xFFFF0000)
    return u.astype(np.uint32).view(np.float32).astype(np.float64)


def weights(cfg, seed=0, sharp=2.0):
    """Random weights exact in bf16; `sharp` scales the gain of the queries so that the softmax is far from uniform."""
    rng = np.random.default_rng(seed)
    S = cfg["streams"]
    out = {}
    for name, shape in shapes(cfg).items():
        z = rng.normal(0.0, 1.0, shape)
        last = name.split(".")[-1]
        if ".hc" in name:
            z = {"in": 1.0 / S + 0.3 * z, "out": 0.6 + 0.3 * z, "mix": np.eye(S) * 0.9 + 0.1 * z if z.ndim == 2 else z}[last]
        elif z.ndim == 1:
            z = 1.0 + 0.2 * z
            z = z * (sharp if name.endswith("q.norm") else 1.0)
        elif name in ("embed", "pos"):
            z = z * (1.0 if name == "embed" else 0.5)
        else:
            z = z / np.sqrt(shape[1]) * (3.0 if name == "head" else 1.0)
        out[name] = bf16_exact(z)
    return out


def save(folder, cfg, w):
    """A checkpoint folder (config.json, model.safetensors in bf16)."""
    import torch
    from safetensors.torch import save_file

    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    save_file({k: torch.tensor(v, dtype=torch.float32).to(torch.bfloat16).contiguous() for k, v in w.items()}, str(folder / "model.safetensors"))
    return folder
