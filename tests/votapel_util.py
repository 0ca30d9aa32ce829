"""Helpers of the Votapel tests: checkpoints in the file format, and weights whose expert choices are not close calls."""
import numpy as np

from rai_b200 import synth


def raw_config(cfg):
    """The config.json of a normalised configuration."""
    layers = []
    for entry in cfg["layers"]:
        mix, mlp = entry["mixer"], entry["mlp"]
        out = {k: mix[k] for k in ("heads", "kv_heads", "dim", "vdim", "scale")}
        if mix["softcap"]:
            out["softcap"] = mix["softcap"]
        if mix["temp_every"]:
            out["q_temp"] = {"coef": mix["temp_coef"], "every": mix["temp_every"]}
        ff = None
        if mlp:
            ff = {"kind": "moe", "expert": {"ff": mlp["ff"]}, "router": {
                "experts": mlp["experts"], "top": mlp["top"], "groups": {"count": mlp["groups"], "keep": mlp["keep"]},
                "scale": mlp["router_scale"]}}
            if mlp["shared_ff"]:
                ff["shared"] = {"ff": mlp["shared_ff"]}
        layers.append({"type": "attention", "mixer": out, "mlp": ff})
    return {"architecture": "Votapel", "vocab": cfg["vocab_size"], "width": cfg["hidden_size"], "norm": {"eps": cfg["norm_eps"]},
            "max_positions": cfg["max_positions"], "residual_mult": cfg["residual_mult"], "layers": layers}


def clear_choice(values, mlp):
    """Do these channel values, at any overall size, leave every selection of the router a margin?"""
    n = mlp["experts"] // mlp["groups"]
    for size in np.linspace(0.25, 1.2, 12):
        s = 1.0 / (1.0 + np.exp(-3.0 * size * values))
        strength = np.sort(s.reshape(mlp["groups"], n), axis=1)[:, -2:].sum(1)
        order = np.sort(strength)[::-1]
        if mlp["keep"] < mlp["groups"] and order[mlp["keep"] - 1] - order[mlp["keep"]] < 0.02:
            return False
    return True


def decided_weights(cfg, seed):
    """Random weights for comparing a 16-bit model with an exact one: the first channels of the stream are set by the token
    alone (nothing later writes to them) and hold well separated values, a different order for every token; the router
    reads them through a permutation of its own, so its selections do not hang on the last bit of its input."""
    w = synth.weights(cfg, seed)
    rng = np.random.default_rng(seed)
    moe = [layer["mlp"] for layer in cfg["layers"] if layer["mlp"]]
    R = max([m["experts"] for m in moe], default=0)
    levels = np.linspace(-2.0, 2.0, R)
    perms = [rng.permutation(R)[:m["experts"]] for m in moe]
    for t in range(cfg["vocab_size"]):
        for _ in range(2000):
            x = levels[rng.permutation(R)]
            if all(clear_choice(x[p], m) for p, m in zip(perms, moe)):
                break
        else:
            raise AssertionError("no order of the levels leaves every layer a margin")
        w["embed"][t, :R] = x
    w["pos"][:, :R] = 0
    done = 0
    for i, layer in enumerate(cfg["layers"]):
        w[f"l{i}.mix.o"][:R] = 0
        w[f"l{i}.norm1"][:R] = 0
        if not layer["mlp"]:
            continue
        for name in w:
            if name.startswith(f"l{i}.mlp.") and name.endswith(".down"):
                w[name][:R] = 0
        router = rng.standard_normal(w[f"l{i}.mlp.router"].shape) * 0.02 / np.sqrt(cfg["hidden_size"])
        router[np.arange(len(perms[done])), perms[done]] = 3.0
        w[f"l{i}.mlp.router"] = router.astype(np.float32)
        done += 1
    return {n: synth.bf16_round(np.asarray(a, dtype=np.float32)).reshape(np.shape(a)) for n, a in w.items()}
