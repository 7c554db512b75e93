"""``python -m openrlhf.cli.generate`` -> ``openrlhf_b200.cli.generate``."""
import sys

from openrlhf_b200.cli.generate import *  # noqa: F401,F403
from openrlhf_b200.cli.generate import main

if __name__ == "__main__":
    sys.exit(main())
