"""Small Nemasun configurations for the tests, and random weights for them.

They differ from each other in every size and constant: streams (1, 3, 4), widths, head
counts and groupings (several query heads a key head, one), head sizes (also one that is no
multiple of 8), windows (shorter than a cache page, longer than one, none; two of one model
different), kept first tokens (none, a few, more than a page), rows and last distances of
the bias tables, the embedding's constant, dense feed-forwards with different limits, routed
experts with and without groups, identity experts and a shared expert, a layer without a
feed-forward.
"""
import torch

_A = {"heads": 6, "kv_heads": 2, "dim": 24, "vdim": 24, "scale": 0.3, "bias_max": 40,
      "mask": {"size": 10, "keep_first": 3}}
_B = {"heads": 2, "kv_heads": 2, "dim": 16, "vdim": 16, "scale": 0.21, "bias_max": 128,
      "mask": {"size": 100, "keep_first": 70}}


def _layer(mixer, mlp):
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def _moe(ff, experts, top, identity=0, groups=None, shared=None):
    router = {"experts": experts, "top": top}
    if identity:
        router["identity"] = identity
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": router}
    if shared:
        mlp["shared"] = {"ff": shared}
    return mlp


CONFIGS = {
    "mixed": {
        "architecture": "Nemasun", "vocab": 150, "width": 80, "streams": 3,
        "norm": {"eps": 1e-5}, "embedding": {"scale": 3.0},
        "layers": [
            _layer(_A, {"kind": "dense", "ff": 104, "limit": 0.8}),
            _layer(dict(_A, heads=4, kv_heads=1, dim=40, vdim=40, bias_max=9,
                        mask={"size": 33, "keep_first": 1}),
                   _moe(56, 6, 3, identity=2, groups=(4, 2), shared=40)),
            _layer(_A, None),
            _layer(dict(_A, mask=None), _moe(24, 5, 2)),
        ],
    },
    "other": {
        "architecture": "Nemasun", "vocab": 97, "width": 64, "streams": 1,
        "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0},
        "layers": [_layer(_B, _moe(32, 7, 4, identity=5, groups=(3, 1), shared=72)),
                   _layer(_B, {"kind": "dense", "ff": 40, "limit": 7.0})],
    },
    "four": {
        "architecture": "Nemasun", "vocab": 64, "width": 36, "streams": 4,
        "norm": {"eps": 1e-5}, "embedding": {"scale": 5.0},
        "layers": [_layer({"heads": 3, "kv_heads": 1, "dim": 10, "vdim": 10, "scale": 0.4,
                           "bias_max": 70, "mask": {"size": 65}},
                          _moe(12, 4, 4, identity=4)),
                   _layer({"heads": 2, "kv_heads": 1, "dim": 32, "vdim": 32, "scale": 0.2,
                           "bias_max": 300, "mask": {"size": 64, "keep_first": 2}},
                          {"kind": "dense", "ff": 20, "limit": 1.5})],
    },
}
# of the distance tables, layer by layer (config.json does not give them)
BIAS_ROWS = {"mixed": [16, 8, 30, 12], "other": [32, 20], "four": [24, 6]}


def mixer_shapes(p, m, W, rows):
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    return {f"{p}.q": (H * d, W), f"{p}.k": (G * d, W), f"{p}.g": (H * d, W),
            f"{p}.o": (W, H * d), f"{p}.q.norm": (d,), f"{p}.k.norm": (d,), f"{p}.rel": (rows, H)}


def mlp_shapes(p, mlp, W):
    if mlp["kind"] == "dense":
        f = mlp["ff"]
        return {f"{p}.gate": (f, W), f"{p}.up": (f, W), f"{p}.down": (W, f), f"{p}.gate.b": (f,),
                f"{p}.up.b": (f,), f"{p}.down.b": (W,)}
    r = mlp["router"]
    n = r["experts"] + r.get("identity", 0)
    shapes = {f"{p}.router": (n, W), f"{p}.correction": (n,)}
    parts = [(f"{p}.e{e}", mlp["expert"]["ff"]) for e in range(r["experts"])]
    if mlp.get("shared"):
        parts.append((f"{p}.shared", mlp["shared"]["ff"]))
    for q, f in parts:
        shapes.update({f"{q}.gate": (f, W), f"{q}.up": (f, W), f"{q}.down": (W, f)})
    return shapes


def tensor_shapes(cfg, bias_rows):
    W, V, S = cfg["width"], cfg["vocab"], cfg["streams"]
    shapes = {"embed": (V, W), "head": (V, W), "final.norm": (W,)}
    for i, (layer, rows) in enumerate(zip(cfg["layers"], bias_rows)):
        p = f"l{i}"
        shapes.update(mixer_shapes(f"{p}.mix", layer["mixer"], W, rows))
        halves = ["1"]
        if layer["mlp"]:
            shapes.update(mlp_shapes(f"{p}.mlp", layer["mlp"], W))
            halves.append("2")
        for q in halves:
            shapes.update({f"{p}.norm{q}": (W,), f"{p}.hc{q}.in": (S,), f"{p}.hc{q}.out": (S,),
                           f"{p}.hc{q}.mix": (S, S)})
    return shapes


def draw(key, shape, gen):
    """One bfloat16-representable float32 tensor. Matrices are wide enough that a wrong key
    moves the logits; the streams' mixing keeps the streams apart without letting them grow."""
    t = torch.randn(shape, generator=gen)
    if key.endswith(".mix") and len(shape) == 2 and shape[0] == shape[1] and ".hc" in key:
        t = 0.75 * torch.eye(shape[0]) + 0.2 * t
    elif key.endswith(".in"):
        t = 1.0 / shape[0] + 0.15 * t
    elif key.endswith(".out"):
        t = 1.0 + 0.2 * t
    elif "norm" in key:
        t = 1.0 + 0.2 * t
    elif key.endswith(".rel"):
        t = 1.2 * t
    elif key.endswith(".correction"):
        t = 0.25 * t - 0.5  # choice scores below 0, too
    elif key.endswith(".b"):
        t = 0.3 * t
    elif key.endswith(".router"):
        t = t * 2.0 / shape[1] ** 0.5
    elif key == "embed":
        t = 0.5 * t
    else:
        t = t * 1.1 / shape[-1] ** 0.5
    return t.to(torch.bfloat16).float()


def random_weights(shapes, seed):
    gen = torch.Generator().manual_seed(seed)
    return {k: draw(k, s, gen) for k, s in shapes.items()}


def named_weights(name, seed=0):
    return random_weights(tensor_shapes(CONFIGS[name], BIAS_ROWS[name]), seed)


def write_model(folder, doc, weights):
    """A model folder as the loader reads it: config.json + model.safetensors (bfloat16)."""
    import json
    import os
    from foundry_b200.weights.safetensors_io import SINGLE_FILE, save_file
    os.makedirs(folder, exist_ok=True)
    save_file({k: v.to(torch.bfloat16) for k, v in weights.items()},
              os.path.join(folder, SINGLE_FILE), metadata={"format": "pt"})
    with open(os.path.join(folder, "config.json"), "w") as handle:
        json.dump(doc, handle)
    return folder, weights


def write_folder(folder, name, seed=0):
    return write_model(folder, CONFIGS[name], named_weights(name, seed))
