"""Helpers of the Tibelix tests: device tensors in the dtypes the engine binds (vectors and router rows float32, matrices bfloat16 or float32)."""
import numpy as np
import torch


def device_tensors(W: dict, exact: bool):
    out = {}
    for name, a in W.items():
        t = torch.from_numpy(np.ascontiguousarray(a, dtype=np.float32)).cuda()
        out[name] = t if (exact or np.ndim(a) < 2 or name.endswith(".router")) else t.to(torch.bfloat16)
    return out
