"""Small Tokovik configurations for the tests, and random weights for them.

The two differ from each other in every size and constant: widths, head counts
and groupings on both sides (several query heads a key head in one, one in the
other), key and value sizes (also sizes that are no multiple of 8), windows
(shorter than a cache page, longer than one; two layers of one model with
different ones), rotated elements (a part of the head, all of it), the
rotation's scaling (with a ramp inside the rotated elements, with none, absent),
ranks of the decays' projection, roots of the decays (also 1), a layer without
feed-forward, and the constants on the embedding and the logits (also 1).
"""
import torch


def _layer(left, right, ff):
    return {"type": "parallel", "mixer": {"left": left, "right": right},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


_A = {"heads": 6, "kv_heads": 2, "dim": 24, "vdim": 40, "scale": 0.3, "mask": {"size": 10},
      "rot": {"dims": 12, "base": 500.0,
              "scaling": {"factor": 3.0, "original": 64, "fast": 6.0, "slow": 0.5}}}
_B = {"heads": 2, "kv_heads": 2, "dim": 32, "vdim": 16, "scale": 0.2, "mask": {"size": 100},
      "rot": {"dims": 32, "base": 10000.0,
              "scaling": {"factor": 8.0, "original": 512, "fast": 32.0, "slow": 1.0}}}

CONFIGS = {
    "mixed": {
        "architecture": "Tokovik", "vocab": 150, "width": 80, "norm": {"eps": 1e-5},
        "embedding": {"scale": 3.0}, "logit_scale": 0.6,
        "layers": [
            _layer(_A, {"heads": 4, "dim": 12, "vdim": 20, "tau": 5.0}, 104),
            _layer(dict(_A, heads=2, kv_heads=1, dim=16, vdim=8, mask={"size": 33},
                        rot={"dims": 8, "base": 77.0}),
                   {"heads": 2, "dim": 40, "vdim": 24, "tau": 1.0}, None),
            _layer(_A, {"heads": 4, "dim": 12, "vdim": 20, "tau": 5.0}, 56),
        ],
    },
    "other": {
        "architecture": "Tokovik", "vocab": 97, "width": 64, "norm": {"eps": 1e-6},
        "embedding": {"scale": 1.0}, "logit_scale": 1.0,
        "layers": [_layer(_B, {"heads": 4, "dim": 32, "vdim": 16, "tau": 16.0}, 72),
                   _layer(_B, {"heads": 1, "dim": 64, "vdim": 64, "tau": 30.0}, 40)],
    },
}
# of the decays' projections, layer by layer (config.json does not give it)
RANKS = {"mixed": [5, 16, 8], "other": [3, 24]}


def mixer_shapes(p, m, W, rank):
    """The tensors of one parallel mixer under the prefix `p` (config entry `m`)."""
    a, r = m["left"], m["right"]
    H, G, d, e = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
    n, v = r["heads"] * r["dim"], r["heads"] * r["vdim"]
    return {f"{p}.left.q": (H * d, W), f"{p}.left.k": (G * d, W), f"{p}.left.v": (G * e, W),
            f"{p}.left.q.b": (H * d,), f"{p}.left.k.b": (G * d,), f"{p}.left.v.b": (G * e,),
            f"{p}.left.q.norm": (d,), f"{p}.left.k.norm": (d,), f"{p}.left.o": (W, H * e),
            f"{p}.left.out": (W,), f"{p}.right.q": (n, W), f"{p}.right.k": (n, W),
            f"{p}.right.v": (v, W), f"{p}.right.g": (v, W), f"{p}.right.a1": (rank, W),
            f"{p}.right.a2": (n, rank), f"{p}.right.a2.b": (n,),
            f"{p}.right.norm": (r["vdim"],), f"{p}.right.o": (W, v), f"{p}.right.out": (W,)}


def tensor_shapes(cfg, ranks):
    W, V = cfg["width"], cfg["vocab"]
    shapes = {"embed": (V, W), "head": (V, W), "final.norm": (W,)}
    for i, (layer, rank) in enumerate(zip(cfg["layers"], ranks)):
        p = f"l{i}"
        shapes[f"{p}.norm1"] = (W,)
        shapes.update(mixer_shapes(f"{p}.mix", layer["mixer"], W, rank))
        if layer["mlp"]:
            ff = layer["mlp"]["ff"]
            shapes.update({f"{p}.norm2": (W,), f"{p}.mlp.gate": (ff, W), f"{p}.mlp.up": (ff, W),
                           f"{p}.mlp.down": (W, ff)})
    return shapes


def draw(key, shape, gen):
    """One bfloat16-representable float32 tensor. Matrices are wide enough that a wrong key
    or state moves the logits; norms around one have weights around one, the model's own
    norms around zero; the decays' bias where a state lasts for a few dozen tokens."""
    leaf = key.split(".")[-1]
    r = torch.randn(shape, generator=gen)
    if key.endswith("a2.b"):
        t = 2.0 + r
    elif leaf == "b":
        t = 0.4 * r
    elif leaf in ("norm1", "norm2") or key == "final.norm":
        t = 0.2 * r
    elif leaf in ("norm", "out"):
        t = 1.0 + 0.2 * r
    elif leaf == "embed":
        t = 0.5 * r
    else:
        t = r / (shape[-1] ** 0.5) * 1.5
    return t.to(torch.bfloat16).to(torch.float32)


def random_tensors(shapes, seed=0):
    gen = torch.Generator().manual_seed(seed)
    return {key: draw(key, shape, gen) for key, shape in shapes.items()}


def random_weights(name, seed=0):
    """Every tensor of the configuration `name`, by file name."""
    return random_tensors(tensor_shapes(CONFIGS[name], RANKS[name]), seed)


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
    return write_model(folder, CONFIGS[name], random_weights(name, seed))
