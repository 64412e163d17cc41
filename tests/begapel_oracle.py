"""Slow float64 NumPy statement of the Begapel decoder, one function per mechanism, and makers of small random models.

Shares no code with the package: the tests compare the package's modules and kernels with these functions."""
import json

import numpy as np


# ------------------------------------------------------------------------------------------ mechanisms
def rms_norm(z, gain, eps, offset):
    """z / sqrt(mean(z^2) + eps) * (offset + gain) over the last axis."""
    return z / np.sqrt(np.mean(z * z, axis=-1, keepdims=True) + eps) * (offset + gain)


def residual_step(x, y, gain, eps, mult):
    """x + mult * norm(y) with a gain stored around zero."""
    return x + mult * rms_norm(y, gain, eps, 1.0)


def rotate_pairs(z, positions, dims, base):
    """Turns the pairs (2i, 2i+1) of the first `dims` values of z [tokens, ..., n] by position * base^(-2i/dims)."""
    out = z.copy()
    for t, p in enumerate(positions):
        for i in range(dims // 2):
            a = p * base ** (-2.0 * i / dims)
            u, v = z[t, ..., 2 * i], z[t, ..., 2 * i + 1]
            out[t, ..., 2 * i] = u * np.cos(a) - v * np.sin(a)
            out[t, ..., 2 * i + 1] = v * np.cos(a) + u * np.sin(a)
    return out


def latents(h, w_dkv, gain, rank, eps, positions, dims, base):
    """The normed latent and the turned shared key part of every token."""
    d = h @ w_dkv.T
    return rms_norm(d[:, :rank], gain, eps, 0.0), rotate_pairs(d[:, rank:], positions, dims, base)


def causal_latent_attention(q, c, k_rot, w_uk, w_uv, heads, dim, vdim, scale, first=0):
    """q [queries, heads, dim + rot] (already turned) against all tokens of c / k_rot; query i sits at token first + i."""
    out = np.zeros((q.shape[0], heads, vdim))
    for h in range(heads):
        k = c @ w_uk[h * dim : (h + 1) * dim].T
        v = c @ w_uv[h * vdim : (h + 1) * vdim].T
        for i in range(q.shape[0]):
            n = first + i + 1
            s = (k[:n] @ q[i, h, :dim] + k_rot[:n] @ q[i, h, dim:]) * scale
            e = np.exp(s - s.max())
            out[i, h] = (e / e.sum()) @ v[:n]
    return out.reshape(q.shape[0], heads * vdim)


def gate(h, w_g):
    return 1.0 / (1.0 + np.exp(-(h @ w_g.T)))


def feed_forward(h, w_gate, w_up, w_down):
    g = h @ w_gate.T
    return (g / (1.0 + np.exp(-g)) * (h @ w_up.T)) @ w_down.T


def soft_cap(z, cap):
    return cap * np.tanh(z / cap)


# ------------------------------------------------------------------------------------------ model
def forward(cfg, w, tokens, return_layers=False):
    """Logits [tokens, vocab] of one sequence (and the stream after every layer)."""
    w = {k: np.asarray(v, dtype=np.float64) for k, v in w.items()}
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    pos = list(range(len(tokens)))
    x = w["embed"][np.asarray(tokens)]
    shared, streams = {}, []
    for i, layer in enumerate(cfg["layers"]):
        a, mix = f"l{i}.", layer["mixer"]
        H, d, r, dv, rank = (mix[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
        h = rms_norm(x, w[a + "norm1"], eps, 1.0)
        q = (h @ w[a + "mix.q"].T).reshape(len(tokens), H, d + r)
        q = np.concatenate([q[..., :d], rotate_pairs(q[..., d:], pos, mix["rot"]["dims"], mix["rot"]["base"])], axis=-1)
        source = mix.get("kv_from")
        if source is None:
            shared[i] = latents(h, w[a + "mix.dkv"], w[a + "mix.dkv.norm"], rank, eps, pos, mix["rot"]["dims"], mix["rot"]["base"])
        c, k_rot = shared[i if source is None else source]
        o = causal_latent_attention(q, c, k_rot, w[a + "mix.uk"], w[a + "mix.uv"], H, d, dv, mix["scale"])
        x = residual_step(x, (o * gate(h, w[a + "mix.g"])) @ w[a + "mix.o"].T, w[a + "norm1b"], eps, m)
        if layer["mlp"] is not None:
            h = rms_norm(x, w[a + "norm2"], eps, 1.0)
            x = residual_step(x, feed_forward(h, w[a + "mlp.gate"], w[a + "mlp.up"], w[a + "mlp.down"]), w[a + "norm2b"], eps, m)
        streams.append(x)
    logits = soft_cap(rms_norm(x, w["final.norm"], eps, 1.0) @ w["head"].T, cfg["logit_softcap"])
    return (logits, streams) if return_layers else logits


def greedy(cfg, w, prompt, n):
    out = list(prompt)
    for _ in range(n):
        out.append(int(forward(cfg, w, out)[-1].argmax()))
    return out


# ------------------------------------------------------------------------------------------ small models
def layer(heads=3, dim=24, rot=8, vdim=40, rank=48, ff=96, base=5000.0, scale=None, kv_from=None, rot_dims=None):
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "rot": {"base": base, "dims": rot if rot_dims is None else rot_dims},
             "scale": (dim + rot) ** -0.5 if scale is None else scale}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(layers, width=72, vocab=90, eps=1e-5, mult=0.7, cap=12.0):
    return {"architecture": "Begapel", "layers": layers, "width": width, "vocab": vocab, "norm": {"eps": eps}, "residual_mult": mult, "logit_softcap": cap}


def shapes(cfg):
    D, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, D), "final.norm": (D,), "head": (V, D)}
    for i, l in enumerate(cfg["layers"]):
        a, m = f"l{i}.", l["mixer"]
        H, d, r, dv, rank = (m[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
        out.update({a + "norm1": (D,), a + "norm1b": (D,), a + "mix.q": (H * (d + r), D), a + "mix.uk": (H * d, rank), a + "mix.uv": (H * dv, rank),
                    a + "mix.g": (H * dv, D), a + "mix.o": (D, H * dv)})
        if m.get("kv_from") is None:
            out.update({a + "mix.dkv": (rank + r, D), a + "mix.dkv.norm": (rank,)})
        if l["mlp"] is not None:
            ff = l["mlp"]["ff"]
            out.update({a + "norm2": (D,), a + "norm2b": (D,), a + "mlp.gate": (ff, D), a + "mlp.up": (ff, D), a + "mlp.down": (D, ff)})
    return out


def bf16_exact(a):
    """Rounded to values bf16 holds exactly."""
    u = np.asarray(a, dtype=np.float32).view(np.uint32)
    u = (u + 0x7FFF + ((u >> 16) & 1)) & np.uint32(0xFFFF0000)
    return u.astype(np.uint32).view(np.float32).astype(np.float64)


def weights(cfg, seed=0, sharp=2.0):
    """Random weights exact in bf16; `sharp` scales the query projections so that the softmax is far from uniform."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in shapes(cfg).items():
        if len(shape) == 1:
            a = rng.normal(0.0, 0.2, shape) + (1.0 if name.endswith("dkv.norm") else 0.0)
        else:
            a = rng.normal(0.0, 1.0, shape) / (1.0 if name == "embed" else np.sqrt(shape[1]))
            a = a * (sharp if name.endswith("mix.q") else 1.0) * (3.0 if name == "head" else 1.0)
        out[name] = bf16_exact(a)
    return out


def save(folder, cfg, w):
    """A checkpoint folder (config.json, model.safetensors in bf16)."""
    import torch
    from safetensors.torch import save_file

    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    save_file({k: torch.tensor(v, dtype=torch.float32).to(torch.bfloat16).contiguous() for k, v in w.items()}, str(folder / "model.safetensors"))
    return folder
