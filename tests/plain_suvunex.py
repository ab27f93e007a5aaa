"""Suvunex, plainly: whole sequences, no cache, no batching, one function per mechanism.

Everything here is written from the design's equations for the tests to compare the engine
with; it shares no code with the package.  ``tensors`` maps checkpoint names to tensors,
``config`` is the parsed config.json.  Arithmetic runs in ``dtype`` (float64 unless told
otherwise).

Notation: T tokens, W the model's width, H query heads, G key/value heads, d a head's
query/key size, e its value size, p_t the position of token t (0 for the first token of a
sequence).
"""

import json
import math
import os
import struct

import numpy as np
import torch


# ------------------------------------------------------------------------------- norms
def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, gain, eps):
    """``gain`` is one number for the whole row, or one per coordinate."""
    return unit_rms(x, eps) * gain


# ------------------------------------------------------------------------------- rotation
def pair_frequencies(rot, dtype=torch.float64):
    """One frequency per pair i: base^(-2i/dims), slowed down as ``rot.scaling`` says.  Only ``factor``: all divided by
    it.  With ``low``, ``high``, ``original``: a pair that makes more than ``high`` turns in ``original`` positions keeps
    its frequency, one that makes fewer than ``low`` has it divided, and between the two the weights go linearly with
    the number of turns."""
    dims = rot["dims"]
    f = float(rot["base"]) ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / max(dims, 1))
    scaling = rot.get("scaling")
    if not scaling:
        return f.to(dtype)
    factor = scaling["factor"]
    if "original" not in scaling:
        return (f / factor).to(dtype)
    out = f.clone()
    for i in range(f.numel()):
        turns = scaling["original"] * float(f[i]) / (2.0 * math.pi)
        if turns > scaling["high"]:
            continue
        if turns < scaling["low"]:
            out[i] = f[i] / factor
            continue
        s = (turns - scaling["low"]) / (scaling["high"] - scaling["low"])
        out[i] = (1.0 - s) * f[i] / factor + s * f[i]
    return out.to(dtype)


def rotate_halves(x, positions, rot):
    """x [T, heads, d]: numbers i and i + dims / 2 (i < dims / 2) turn together; what lies behind ``dims`` stays."""
    half = rot["dims"] // 2
    angle = (positions.to(x.dtype)[:, None] * pair_frequencies(rot, x.dtype)[None, :])[:, None, :]
    u, v = x[..., :half], x[..., half:2 * half]
    cos, sin = torch.cos(angle), torch.sin(angle)
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., 2 * half:]], dim=-1)


# ------------------------------------------------------------------------------- softmax
def causal_softmax(scores, extra):
    """scores [H, T, T] (query, key), keys later than the query left out; ``extra`` [H]: a score per head that takes
    part in the denominator and has no value."""
    T = scores.shape[-1]
    later = torch.ones(T, T, dtype=torch.bool).triu(1)
    s = scores.masked_fill(later[None], float("-inf"))
    sink = extra.to(s.dtype)[:, None, None].expand(-1, T, 1)
    top = torch.maximum(s.max(-1, keepdim=True).values, sink)
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))


# ------------------------------------------------------------------------------- mixers
def projection(tensors, name, h):
    """W h, plus the bias if the model has one under that name."""
    y = h @ tensors[name].to(h.dtype).T
    if name + ".b" in tensors:
        y = y + tensors[name + ".b"].to(h.dtype)
    return y


def turned_attention(tensors, prefix, m, h, positions, eps):
    """Biased projections; q and k turn, then lose their length; softmax with a one in the denominator."""
    H, G, d, e, T = m["heads"], m["kv_heads"], m["dim"], m["vdim"], h.shape[0]
    q = projection(tensors, prefix + "q", h).reshape(T, H, d)
    k = projection(tensors, prefix + "k", h).reshape(T, G, d)
    v = projection(tensors, prefix + "v", h).reshape(T, G, e)
    q = unit_rms(rotate_halves(q, positions, m["rot"]), eps)
    k = unit_rms(rotate_halves(k, positions, m["rot"]), eps)
    rows = []
    weights = None
    for head in range(H):
        group = head // (H // G)
        scores = (q[:, head] @ k[:, group].T) * m["scale"]
        weights = causal_softmax(scores[None], torch.zeros(1))[0]
        rows.append(weights @ v[:, group])
    return projection(tensors, prefix + "o", torch.cat(rows, dim=-1))


def decay_rates(tensors, prefix, m, h):
    """[T, H, d]: sigmoid(z)^(1/tau), z = W_a2 (W_a1 h) + b."""
    z = (h @ tensors[prefix + "a1"].to(h.dtype).T) @ tensors[prefix + "a2"].to(h.dtype).T
    z = z + tensors[prefix + "a2.b"].to(h.dtype)
    return torch.sigmoid(z).pow(1.0 / m["tau"]).reshape(h.shape[0], m["heads"], m["dim"])


def gated_linear_attention(tensors, prefix, m, h, eps):
    """S <- diag(alpha) S + k v^T, o = S^T q; head norm, silu gate, output projection."""
    H, d, e, T = m["heads"], m["dim"], m["vdim"], h.shape[0]
    q = (projection(tensors, prefix + "q", h) * d ** -0.5).reshape(T, H, d)
    k = projection(tensors, prefix + "k", h).reshape(T, H, d)
    v = projection(tensors, prefix + "v", h).reshape(T, H, e)
    alpha = decay_rates(tensors, prefix, m, h)
    state = torch.zeros(H, d, e, dtype=h.dtype)
    rows = []
    for t in range(T):
        state = alpha[t][:, :, None] * state + k[t][:, :, None] * v[t][:, None, :]
        rows.append(torch.einsum("hd,hde->he", q[t], state))
    o = rms_norm(torch.stack(rows), tensors[prefix + "norm"].to(h.dtype), eps).reshape(T, H * e)
    gate = projection(tensors, prefix + "g", h)
    return projection(tensors, prefix + "o", o * (gate * torch.sigmoid(gate)))


def parallel_mixer(tensors, prefix, m, h, positions, eps):
    left = turned_attention(tensors, prefix + "left.", m["left"], h, positions, eps)
    right = gated_linear_attention(tensors, prefix + "right.", m["right"], h, eps)
    return m["left_scale"] * left + m["right_scale"] * right


def talking_attention(tensors, prefix, m, h, positions, eps):
    """Values are the projected keys; head norms with gains, then the turn; a learned sink; the heads' weights are mixed
    across heads before they meet the values."""
    H, G, d, T = m["heads"], m["kv_heads"], m["dim"], h.shape[0]
    q = projection(tensors, prefix + "q", h).reshape(T, H, d)
    k = projection(tensors, prefix + "k", h).reshape(T, G, d)
    v = k
    q = rotate_halves(rms_norm(q, tensors[prefix + "q.norm"].to(h.dtype), eps), positions, m["rot"])
    k = rotate_halves(rms_norm(k, tensors[prefix + "k.norm"].to(h.dtype), eps), positions, m["rot"])
    scores = torch.stack([q[:, head] @ k[:, head // (H // G)].T for head in range(H)]) * m["scale"]
    weights = causal_softmax(scores, tensors[prefix + "sink"])
    mixed = torch.einsum("hg,gij->hij", tensors[prefix + "talk"].to(h.dtype), weights)
    rows = [mixed[head] @ v[:, head // (H // G)] for head in range(H)]
    return projection(tensors, prefix + "o", torch.cat(rows, dim=-1))


# ------------------------------------------------------------------------------- feed-forward, convolution
def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def gated_ff(tensors, prefix, h):
    return projection(tensors, prefix + "down",
                      gelu_tanh(projection(tensors, prefix + "gate", h)) * projection(tensors, prefix + "up", h))


def with_convolution(h, w):
    """Every row plus the ``taps`` newest rows (itself included, none before the first token) weighed by w, newest last."""
    taps = w.shape[1]
    out = h.clone()
    for t in range(h.shape[0]):
        for j in range(taps):
            source = t - taps + 1 + j
            if source >= 0:
                out[t] = out[t] + w[:, j] * h[source]
    return out


# ------------------------------------------------------------------------------- the model
def forward(tensors, config, tokens, dtype=torch.float64, layers_out=None):
    """Logits [T, vocab] of one whole sequence.  ``layers_out``: a list that receives the residual rows behind
    every layer."""
    eps = config["norm"]["eps"]
    t = lambda name: tensors[name].to(dtype)
    ids = torch.as_tensor(tokens, dtype=torch.long)
    positions = torch.arange(len(ids))
    x = t("embed")[ids] * config["embedding"]["scale"]
    for index, layer in enumerate(config["layers"]):
        p = f"l{index}."
        h = with_convolution(rms_norm(x, t(p + "norm1"), eps), t(p + "canon1"))
        mix = parallel_mixer if layer["type"] == "parallel" else talking_attention
        y = mix(tensors, p + "mix.", layer["mixer"], h, positions, eps)
        x = x + t(p + "ls1") * rms_norm(y, t(p + "norm1b"), eps)
        if layer.get("mlp") is not None:
            y = gated_ff(tensors, p + "mlp.", rms_norm(x, t(p + "norm2"), eps))
            x = x + t(p + "ls2") * rms_norm(y, t(p + "norm2b"), eps)
        if layers_out is not None:
            layers_out.append(x)
    return rms_norm(x, t("final.norm"), eps) @ t("head").T * config["logit_scale"]


def read_folder(folder, dtype=torch.float64):
    """(tensors, config) of a model folder; the safetensors file is read here, byte by byte."""
    with open(os.path.join(folder, "config.json")) as handle:
        config = json.load(handle)
    with open(os.path.join(folder, "model.safetensors"), "rb") as handle:
        size = struct.unpack("<Q", handle.read(8))[0]
        header = json.loads(handle.read(size))
        data = handle.read()
    tensors = {}
    for name, entry in header.items():
        if name == "__metadata__":
            continue
        lo, hi = entry["data_offsets"]
        raw = np.frombuffer(data[lo:hi], dtype=np.uint8)
        if entry["dtype"] == "BF16":
            wide = raw.view(np.uint16).astype(np.uint32) << 16
            value = torch.from_numpy(wide.view(np.float32).copy())
        elif entry["dtype"] == "F32":
            value = torch.from_numpy(raw.view(np.float32).copy())
        else:
            raise ValueError(f"{name}: dtype {entry['dtype']}")
        tensors[name] = value.reshape(entry["shape"]).to(dtype)
    return tensors, config


# ------------------------------------------------------------------------------- random models for the tests
def tensor_shapes(config):
    """{checkpoint name: shape} of a model of ``config`` (``decay_rank`` of a test's mixer, not a key of the format,
    is the inner size of the decay's two matrices)."""
    W, V, taps = config["width"], config["vocab"], config["canon"]["taps"]
    shapes = {"embed": (V, W), "head": (V, W), "final.norm": ()}
    for index, layer in enumerate(config["layers"]):
        p, m = "l%d." % index, layer["mixer"]
        shapes.update({p + "norm1": (), p + "norm1b": (), p + "ls1": (W,), p + "canon1": (W, taps)})
        if layer["type"] == "parallel":
            left, right = m["left"], m["right"]
            H, G, d, e = left["heads"], left["kv_heads"], left["dim"], left["vdim"]
            for name, rows in (("q", H * d), ("k", G * d), ("v", G * e)):
                shapes[p + "mix.left." + name] = (rows, W)
                shapes[p + "mix.left." + name + ".b"] = (rows,)
            shapes[p + "mix.left.o"] = (W, H * e)
            shapes[p + "mix.left.o.b"] = (W,)
            H, d, e, rank = right["heads"], right["dim"], right["vdim"], DECAY_RANKS.get(index, 16)
            shapes.update({p + "mix.right.q": (H * d, W), p + "mix.right.k": (H * d, W), p + "mix.right.v": (H * e, W),
                           p + "mix.right.g": (H * e, W), p + "mix.right.o": (W, H * e), p + "mix.right.norm": (e,),
                           p + "mix.right.a1": (rank, W), p + "mix.right.a2": (H * d, rank),
                           p + "mix.right.a2.b": (H * d,)})
        else:
            H, G, d = m["heads"], m["kv_heads"], m["dim"]
            for name, rows in (("q", H * d), ("k", G * d)):
                shapes[p + "mix." + name] = (rows, W)
                shapes[p + "mix." + name + ".b"] = (rows,)
                shapes[p + "mix." + name + ".norm"] = (d,)
            shapes.update({p + "mix.talk": (H, H), p + "mix.sink": (H,), p + "mix.o": (W, H * d)})
        if layer.get("mlp") is not None:
            ff = layer["mlp"]["ff"]
            shapes.update({p + "norm2": (), p + "norm2b": (), p + "ls2": (W,), p + "mlp.gate": (ff, W),
                           p + "mlp.up": (ff, W), p + "mlp.down": (W, ff)})
    return shapes


# inner sizes of the decay's two matrices, by the layer's place in a test's model (16 where none is given)
DECAY_RANKS = {0: 16, 1: 5, 2: 12, 3: 33, 4: 1}


def random_model(config, seed):
    """Random tensors (rounded to bfloat16, stored as such) that keep activations of order one."""
    g = torch.Generator().manual_seed(seed)
    tensors = {}
    for name, shape in tensor_shapes(config).items():
        leaf = name.split(".")[-1]
        if name == "embed":
            value = torch.randn(shape, generator=g) / config["embedding"]["scale"]
        elif leaf in ("norm", "norm1", "norm2", "norm1b", "norm2b"):
            value = 1.0 + 0.2 * torch.randn(shape, generator=g)
        elif leaf in ("ls1", "ls2"):
            value = 0.7 + 0.2 * torch.randn(shape, generator=g)
        elif leaf == "canon1":
            value = 0.5 * torch.randn(shape, generator=g) / math.sqrt(shape[1])
        elif leaf == "talk":
            value = torch.eye(shape[0]) + 0.4 * torch.randn(shape, generator=g)
        elif leaf == "sink":
            value = torch.randn(shape, generator=g)
        elif leaf == "b":
            value = (1.5 if name.endswith("a2.b") else 0.4) * torch.randn(shape, generator=g)
        else:
            value = torch.randn(shape, generator=g) / math.sqrt(shape[1])
        tensors[name] = value.to(torch.bfloat16)
    return tensors


def dense_mlp(ff=48):
    return {"kind": "dense", "ff": ff}


def llama_scaling(factor, low, high, original):
    return {"factor": factor, "low": low, "high": high, "original": original}


def left_side(heads=4, kv_heads=2, dim=16, vdim=16, rot_dims=None, base=10000.0, scaling=None, scale=0.25):
    rot = {"base": base, "dims": dim if rot_dims is None else rot_dims}
    if scaling is not None:
        rot["scaling"] = scaling
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": rot, "scale": scale}


def right_side(heads=3, dim=16, vdim=24, tau=8.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}


def parallel_layer(left, right, left_scale=0.7, right_scale=0.6, mlp=None):
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}}


def talking_layer(heads=4, kv_heads=2, dim=16, rot_dims=None, base=10000.0, factor=None, scale=0.25, mlp=None):
    rot = {"base": base, "dims": dim if rot_dims is None else rot_dims}
    if factor is not None:
        rot["scaling"] = {"factor": factor}
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "rot": rot, "scale": scale}}


def make_config(layers, width=64, vocab=97, eps=1e-5, taps=3, embedding_scale=4.0, logit_scale=0.5):
    return {"architecture": "Suvunex", "canon": {"taps": taps}, "embedding": {"scale": embedding_scale},
            "layers": layers, "logit_scale": logit_scale, "norm": {"eps": eps}, "vocab": vocab, "width": width}
