"""Redodra generation: layers normed before and after mixer and feed-forward (delta rule, attention beside Mamba-2, attention with
sinks), each reading a weighted average of all earlier results.

    python examples/models/redodra/redodra.py -n 64 --batch 8                      # random weights
    python examples/models/redodra/redodra.py --model /path/to/model -n 64         # config.json + model.safetensors
    python examples/models/redodra/redodra.py --tiny --dtype float32 -n 8          # quick functional run
"""
import argparse
import os
import sys

sys.path.insert(0, os.path.join(os.path.dirname(os.path.abspath(__file__)), "..", "..", ".."))

from nkipy_b200.models import runner  # noqa: E402
from nkipy_b200.models.config import redodra_shape  # noqa: E402


def main():
    if "--model" in sys.argv:
        return runner.main()
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    runner.add_common_args(ap)
    cfg = redodra_shape(2048, layers=15, heads=16, kv_heads=4, ff=5632, share_every=2)
    return runner.run_generation(cfg, ap.parse_args())


if __name__ == "__main__":
    sys.exit(main())
