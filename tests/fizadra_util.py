"""Helpers of the Fizadra tests: checkpoints in the file format, and weights with a pair of tokens that look for each other."""
import numpy as np


def raw_config(cfg):
    """The config.json of a normalised configuration."""
    layers = []
    for entry in cfg["layers"]:
        mix, mlp = entry["mixer"], entry["mlp"]
        if mix["type"] == "attention":
            kind, mixer = "attention", {k: mix[k] for k in ("heads", "kv_heads", "dim", "vdim", "scale")}
        else:
            kind = "latent_attention" if mix["sink"] else "latent_attention_2"
            mixer = {k: mix[k] for k in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale")}
            if mix["kv_from"] is not None:
                mixer["kv_from"] = mix["kv_from"]
        if mix["rot"]:
            mixer["rot"] = {k: mix["rot"][k] for k in ("dims", "base")}
            if mix["rot"]["scaling"]:
                mixer["rot"]["scaling"] = dict(mix["rot"]["scaling"])
        layers.append({"type": kind, "mixer": mixer, "mlp": dict(mlp) if mlp else None})
    return {"architecture": "Fizadra", "vocab": cfg["vocab_size"], "width": cfg["hidden_size"],
            "norm": {"eps": cfg["norm_eps"], "groups": cfg["norm_groups"]}, "layers": layers}


def pointed(cfg, w, query, key, strength=6.0):
    """Weights in which, in every layer, token `query` looks for token `key` through one number that does not turn: the score of
    such a pair stands out by far.  Two channels of the stream say which token a row is; nothing is added to them, and the
    depth averages keep their sign."""
    w = {n: np.array(a) for n, a in w.items()}
    q_ch, k_ch = cfg["hidden_size"] - 1, cfg["hidden_size"] - 2
    w["embed"][:, [q_ch, k_ch]] = 0
    w["embed"][query, q_ch], w["embed"][key, k_ch] = 4.0, 4.0
    for i, entry in enumerate(cfg["layers"]):
        mix, p = entry["mixer"], f"l{i}.mix."
        for name in w:
            if name.startswith(f"l{i}.") and (name.endswith(".o") or name.endswith(".down")):
                w[name][[q_ch, k_ch]] = 0
        w[f"l{i}.dwa"] = np.abs(w[f"l{i}.dwa"])
        d, H = mix["dim"], mix["heads"]
        if mix["type"] == "attention":
            for part, heads, ch in (("q", H, q_ch), ("k", mix["kv_heads"], k_ch)):
                for h in range(heads):
                    row = h * d + d - 1             # (the last dimension is beyond those that turn)
                    w[p + part][row] = 0
                    w[p + part][row, ch] = strength
                    w[p + part + ".b"][row] = 0
        else:
            w[p + "dq"][0] = 0
            w[p + "dq"][0, q_ch] = strength
            for h in range(H):
                row = h * (d + mix["rot_dim"])
                w[p + "uq"][row] = 0
                w[p + "uq"][row, 0] = 4.0
                w[p + "uk"][h * d] = 0
                w[p + "uk"][h * d, 0] = 4.0
            if mix["kv_from"] is None:
                w[p + "dkv"][0] = 0
                w[p + "dkv"][0, k_ch] = strength
    return w
